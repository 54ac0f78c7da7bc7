"""Fusazen without a GPU: config.json -> spec, the refusals, the tensors a configuration wants, what its runs keep between steps
(a layer's cache when another layer reads it under another mask), and the plain implementation's own consistency."""
import copy
import math

import pytest
import torch

from jllm_serve_b200.cache import CacheManager
from jllm_serve_b200.cache.manager import FixedState, PagedKeysValues, span_covering
from jllm_serve_b200.config import ConfigError, parse_config
from jllm_serve_b200.config.registry import architecture_entry
from jllm_serve_b200.config.specs import GqaAttentionSpec
from jllm_serve_b200.engine.model import DecoderModel, model_wants
from tests.fusazen_cases import FUSAZEN, fusazen_folder, random_fusazen, stored_config
from tests.plain import fusazen_plain as P


def test_the_parser_reads_every_size_and_constant():
    spec = parse_config(FUSAZEN["A"])
    assert spec.core.architecture == "Fusazen" and spec.core.dim == 56 and spec.core.vocab == 150 and spec.core.embedding_scale == 1.5
    assert all(l.arrangement == "pre_norm" and l.input_conv == "canon1" and l.input_conv_taps == 3 for l in spec.layers)
    a2 = spec.layers[0].mixer
    assert (a2.heads, a2.kv_heads, a2.head_dim, a2.value_dim, a2.chunk, a2.scale) == (6, 2, 24, 16, 20, 0.3)
    assert a2.qk_norm and a2.qk_norm_over == "all" and a2.qk_norm_eps == 2e-5 and a2.head_scale and a2.maps == 1 and a2.rope_table == -1
    d = spec.layers[1].mixer
    assert (d.kind, d.heads, d.key_dim, d.value_dim, d.norm_eps) == ("general_delta", 3, 12, 12, 2e-5)
    assert d.decay_rate == math.exp(-0.5) and d.decay_rank == 5
    att, other = spec.layers[2].mixer, spec.layers[3].mixer
    assert (att.heads, att.kv_heads, att.head_dim, att.value_dim, att.maps, att.diff, att.chunk) == (4, 2, 12, 20, 2, 0.4, 13)
    assert att.own_kv and not other.own_kv and other.chunk == 40 and other.diff == 0.3
    assert [r.cache_of for r in spec.schedule] == [None, None, None, 2, None, 2]
    assert len(spec.rope_tables) == 1 and (spec.rope_tables[0].rotary_dim, spec.rope_tables[0].theta) == (8, 100.0)
    ff = spec.layers[0].feed_forward
    assert (ff.kind, ff.hidden, ff.activation, ff.bias_names) == ("dense_mlp", 40, "relu2", ("up.b", "down.b"))
    assert spec.layers[2].feed_forward is None
    assert parse_config(FUSAZEN["C"]).core.embedding_scale == 1.0 and parse_config(FUSAZEN["C"]).layers[3].mixer.chunk == 0
    assert parse_config(stored_config(FUSAZEN["A"])).layers[1].mixer.decay_rank == -1


@pytest.mark.parametrize("change, text", [
    (lambda c: c["layers"][0].update(type="attention_3"), "unknown layer type"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "unknown feed-forward kind"),
    (lambda c: c.pop("canon"), "canon"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=14), "exceeds the head's dim"),
    (lambda c: c["layers"][2]["mixer"].pop("diff"), "diff"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=3), "divide"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "names no earlier layer"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=1), "no attention with keys and values"),
    (lambda c: c["layers"][5]["mixer"].update(kv_from=3), "no attention with keys and values"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=24), "no attention with keys and values"),
    (lambda c: c["layers"][3]["mixer"]["rot"].update(base=50.0), "no attention with keys and values"),
    (lambda c: c["layers"][1]["mixer"].update(dim=2000), "up to 1024"),
    (lambda c: c["canon"].update(taps=0), "taps"),
    (lambda c: c["layers"][0].pop("mixer"), "mixer"),
])
def test_what_the_parser_refuses(change, text):
    cfg = copy.deepcopy(FUSAZEN["A"])
    change(cfg)
    with pytest.raises(ConfigError, match=text):
        parse_config(cfg)


def test_forms_that_are_not_built_together_are_refused():
    for bad in (dict(maps=2, bias=True), dict(maps=2, gate="sigmoid"), dict(head_scale=True, qk_norm=True, sink=True),
                dict(maps=2, qk_norm=True), dict(maps=3)):
        with pytest.raises(ConfigError):
            GqaAttentionSpec(heads=2, kv_heads=1, head_dim=16, scale=1.0, **bad)


def test_the_tensors_a_configuration_wants():
    wants = model_wants(architecture_entry("Fusazen"), parse_config(FUSAZEN["A"]))
    shape = {n: w.shape for n, w in wants.items()}
    assert shape["embed"] == (150, 56) and shape["head"] == (150, 56) and shape["final.norm"] == (56,)
    assert all(shape[f"l{i}.canon1"] == (56, 3) and shape[f"l{i}.norm1"] == (56,) for i in range(6))
    assert shape["l0.mix.q"] == (144, 56) and shape["l0.mix.k"] == (48, 56) and shape["l0.mix.v"] == (32, 56)
    assert shape["l0.mix.q.norm"] == (144,) and shape["l0.mix.k.norm"] == (48,) and shape["l0.mix.temp"] == (6,)
    assert shape["l0.mix.o"] == (56, 96) and shape["l0.mlp.up.b"] == (40,) and shape["l0.mlp.down.b"] == (56,)
    assert all(shape[f"l1.mix.{n}"] == (36, 56) for n in "rkvga") and shape["l1.mix.a.b"] == shape["l1.mix.w0"] == (36,)
    assert shape["l1.mix.w1"] == (5, 56) and shape["l1.mix.w2"] == (36, 5) and shape["l1.mix.norm"] == (36,)
    assert shape["l2.mix.q"] == (4 * 2 * 12, 56) and shape["l2.mix.k"] == (2 * 2 * 12, 56) and shape["l2.mix.v"] == (40, 56)
    assert all(shape[f"l2.mix.{n}"] == (12,) for n in ("lq1", "lk1", "lq2", "lk2")) and shape["l2.mix.o"] == (56, 80)
    assert "l3.mix.k" not in shape and "l3.mix.v" not in shape and shape["l3.mix.q"] == (96, 56)
    assert "l2.norm2" not in shape and not any(n.startswith("l4.mlp") for n in shape)
    assert wants["l0.canon1"].role == "vector"


class Shell(DecoderModel):
    def __init__(self, spec):
        self.spec = spec


def test_what_the_runs_keep_between_steps():
    needs = Shell(parse_config(FUSAZEN["A"])).cache_needs()
    conv = FixedState((2, 56))
    assert needs[0] == (PagedKeysValues(2, 32, -20), conv)          # (24 values, filled up to 32)
    assert needs[1] == (FixedState((3, 12, 12)), conv)
    # layer 2 sees chunks of 13, layers 3 and 5 read its rows under chunks of 40 and 7: a window of 40 covers all of them
    assert needs[2] == (PagedKeysValues(2, 32, 40), conv)
    assert needs[3] == (conv,) and needs[5] == (conv,)
    c = Shell(parse_config(FUSAZEN["C"])).cache_needs()
    assert c[0] == (PagedKeysValues(1, 32, -33), FixedState((1, 72)))
    assert c[3] == (PagedKeysValues(2, 320, 0), FixedState((1, 72)))
    b = Shell(parse_config(FUSAZEN["B"])).cache_needs()
    assert b[1] == (PagedKeysValues(2, 128, -100), FixedState((3, 128)))      # (a reader under the same mask changes nothing)


@pytest.mark.parametrize("maps, dim, vdim, width", [(2, 64, 128, 128), (2, 50, 98, 128), (1, 52, 52, 64), (2, 32, 64, 64),
                                                    (1, 128, 128, 128), (2, 20, 16, 48), (1, 80, 80, 80), (2, 100, 30, 256),
                                                    (2, 160, 40, 320), (1, 8, 50, 64), (2, 130, 10, 264)])
def test_the_width_of_a_wide_attentions_rows(maps, dim, vdim, width):
    spec = GqaAttentionSpec(heads=2, kv_heads=1, head_dim=dim, value_dim=vdim, scale=1.0, maps=maps, head_scale=maps == 1,
                            qk_norm=maps == 1, qk_norm_over="all" if maps == 1 else "head")
    assert spec.wide and spec.row_dim == width and spec.row_dim >= max(maps * dim, vdim)
    assert GqaAttentionSpec(heads=2, kv_heads=1, head_dim=dim, value_dim=vdim, scale=1.0).row_dim == max(dim, vdim)


def test_a_span_that_covers_two_readers():
    """No page may be given back that either reader still sees, at any length; and where the spans are equal nothing changes."""
    from itertools import product

    def first(p, span):
        return 0 if span == 0 else max(0, p + 1 - span) if span > 0 else p - p % -span
    for a, b in product((0, 5, 12, -4, -9, -30), repeat=2):
        c = span_covering(a, b)
        assert all(first(p, c) <= min(first(p, a), first(p, b)) for p in range(120)), (a, b, c)
        assert a != b or c == a


def test_pages_of_a_cache_that_two_masks_read():
    """Chunks of 7 read under chunks of 20 too, pages of 4: after every step the pages that a row of either may see are there."""
    cache = CacheManager([PagedKeysValues(1, 8, span_covering(-7, -20))], 4, 60, 1)
    cache.open("a")
    at = 0
    for n in (3, 9, 1, 1, 20, 1, 7, 30, 2):
        cache.reserve("a", at, n)
        at += n
        cache.commit("a", at)
        held = [i for i, p in enumerate(cache.requests["a"].tables[0]) if p >= 0]
        need = (at - at % 20) // 4                   # the next row's chunk of 20
        assert all(i in held for i in range(need, -(-at // 4))), (at, held)
        cache.check()
    assert len(held) <= 6
    cache.close("a")
    cache.check()


@pytest.mark.parametrize("seed", range(9300, 9330))
def test_drawn_configurations_parse(seed):
    spec = parse_config(random_fusazen(seed))
    assert model_wants(architecture_entry("Fusazen"), spec) and Shell(spec).cache_needs()


def test_the_plain_recurrence_against_its_closed_form():
    """One token, and two tokens with the second's removal written out; a key that comes twice with rate 1 and no decay leaves
    only its second value behind."""
    g = torch.Generator().manual_seed(5)
    r, k, v = (torch.randn(2, 1, 6, generator=g, dtype=torch.float64) for _ in range(3))
    d, a = torch.rand(2, 1, 6, generator=g, dtype=torch.float64), torch.rand(2, 1, 6, generator=g, dtype=torch.float64)
    o = P.delta_recurrence(r, k, v, d, a)[:, 0]
    S0 = torch.outer(k[0, 0], v[0, 0])
    assert torch.allclose(o[0], S0.T @ r[0, 0])
    u = k[1, 0] / torch.sqrt((k[1, 0] ** 2).sum() + 1e-6)
    S1 = torch.diag(d[1, 0]) @ S0 - torch.outer(a[1, 0] * u, u @ S0) + torch.outer(k[1, 0], v[1, 0])
    assert torch.allclose(o[1], S1.T @ r[1, 0])
    k2 = k[:1].repeat(2, 1, 1)
    one = torch.ones(2, 1, 6, dtype=torch.float64)
    o = P.delta_recurrence(k2, k2, v, one, one)[1, 0]
    assert torch.allclose(o, v[1, 0] * (k2[0, 0] ** 2).sum(), rtol=1e-4)


def test_plain_logits_of_a_prefix_do_not_depend_on_what_follows():
    cfg, w = P.load_plain(fusazen_folder("A"))
    toks = [int(t) for t in torch.randint(0, 150, (45,), generator=torch.Generator().manual_seed(3))]
    whole = P.forward(cfg, w, toks)
    for n in (1, 13, 14, 40, 41):
        assert torch.allclose(P.forward(cfg, w, toks[:n]), whole[:n], atol=1e-9)
    moved = list(toks)
    moved[0] = (moved[0] + 1) % 150                  # a first token shows in the last logits (through the recurrences)
    assert float((P.forward(cfg, w, moved)[-1] - whole[-1]).abs().max()) > 1e-6
