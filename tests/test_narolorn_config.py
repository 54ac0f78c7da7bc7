"""Narolorn without a GPU: config.json -> spec, the refusals, the order of the layer runs, the tensors a configuration wants, what its
runs keep between steps, and what the plain implementation and the test models can tell apart."""
import copy

import pytest
import torch

from jllm_serve_b200.cache.manager import PagedKeysValues
from jllm_serve_b200.config import ConfigError, parse_config
from jllm_serve_b200.config.registry import architecture_entry
from jllm_serve_b200.config.specs import GqaAttentionSpec, LatentAttentionSpec, RoutedExpertsSpec, tile_width
from jllm_serve_b200.engine.model import DecoderModel, model_wants
from tests.narolorn_cases import NAROLORN, narolorn_folder, random_narolorn
from tests.plain import narolorn_plain as P
from tests.tiny import random_tokens


def test_the_parser_reads_every_size_and_constant():
    spec = parse_config(NAROLORN["A"])
    core = spec.core
    assert (core.architecture, core.dim, core.vocab, core.streams, core.logit_softcap, core.tied) == ("Narolorn", 56, 150, 2, 9.0, True)
    assert all(l.arrangement == "hyper_connections" and l.streams == 2 and l.norm.eps == 2e-3 for l in spec.layers)
    lat = spec.layers[0].mixer
    assert (lat.kind, lat.heads, lat.key_dim, lat.value_dim, lat.rank, lat.scale, lat.window) == ("latent_attention", 3, 12, 20, 24, 0.3, 13)
    assert lat.gated and lat.gate_full and lat.tile_rows and lat.norm_eps == 2e-3 and lat.cache_dim == 24
    keys = spec.layers[1].mixer
    assert (keys.heads, keys.kv_heads, keys.head_dim, keys.v_dim, keys.chunk, keys.scale) == (4, 2, 24, 24, 20, 0.25)
    assert keys.keys_as_values and keys.qk_norm and keys.qk_norm_over == "all" and keys.qk_norm_eps == 2e-3 and keys.rope_table == 0
    assert len(spec.rope_tables) == 1 and (spec.rope_tables[0].rotary_dim, spec.rope_tables[0].theta, spec.rope_tables[0].pairing) == (8, 100.0, "half")
    att = spec.layers[2].mixer
    assert (att.heads, att.kv_heads, att.head_dim, att.v_dim, att.softcap, att.temp_coef, att.temp_every) == (6, 2, 12, 20, 4.0, 0.4, 16)
    assert att.window == att.chunk == 0 and att.rope_table == -1 and not att.qk_norm
    ff = spec.layers[0].feed_forward
    assert (ff.experts, ff.top, ff.hidden, ff.limit, ff.shared.hidden, ff.shared.limit) == (5, 2, 16, 1.2, 24, 0.7)
    assert (ff.score, ff.normalize, ff.router_bias, ff.shared_gate, ff.weight_on) == ("softmax", True, "router.b", "shared.sg", "output")
    assert spec.layers[1].feed_forward is None
    c = parse_config(NAROLORN["C"])
    assert c.core.logit_softcap == 0.0 and c.core.streams == 1 and c.layers[1].mixer.softcap == 0.0 and c.layers[1].mixer.temp_every == 0
    assert c.layers[0].mixer.window == 0 and c.layers[2].mixer.rope_table == -1 and c.layers[0].feed_forward.shared is None


def test_the_order_of_the_layer_runs():
    order = lambda cfg: [r.layer for r in parse_config(cfg).schedule]
    assert order(NAROLORN["A"]) == [0, 1, 2, 1, 2, 1, 2, 3] == P.layer_runs(NAROLORN["A"])
    assert order(NAROLORN["C"]) == list(range(6)) and order(NAROLORN["S"]) == [0, 1, 2, 0, 1, 2]
    assert all(r.cache_of is None for r in parse_config(NAROLORN["A"]).schedule)
    one = dict(NAROLORN["A"], loop={"start": 2, "stop": 3, "times": 1})
    none = dict(NAROLORN["A"], loop={"start": 2, "stop": 2, "times": 5})
    assert order(one) == order(none) == [0, 1, 2, 3] == P.layer_runs(one) == P.layer_runs(none)


@pytest.mark.parametrize("change, text", [
    (lambda c: c["layers"][0].update(type="attention_3"), "unknown layer type"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "unknown feed-forward kind"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=26), "exceeds the head's dim"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=20), "values are the keys"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=4), "divide"),
    (lambda c: c["layers"][2]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][2]["mixer"]["q_temp"].update(every=0), "every"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "top=6"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][0]["mlp"]["shared"].update(limit=0.0), "limit"),
    (lambda c: c["layers"][0].pop("mixer"), "mixer"),
    (lambda c: c["loop"].update(stop=9), "stop=9"),
    (lambda c: c["loop"].update(start=3, stop=1), "start=3"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c.update(streams=17), "streams=17"),
    (lambda c: c.update(logit_softcap=0), "logit_softcap"),
    (lambda c: c.update(layers=[]), "at least one layer"),
])
def test_what_the_parser_refuses(change, text):
    cfg = copy.deepcopy(NAROLORN["A"])
    change(cfg)
    with pytest.raises(ConfigError, match=text):
        parse_config(cfg)


def test_forms_that_are_not_built_together_are_refused():
    for bad in (dict(keys_as_values=True, value_dim=8), dict(keys_as_values=True, gate="sigmoid"), dict(temp_every=4, bias=True), dict(softcap=-1.0)):
        with pytest.raises(ConfigError):
            GqaAttentionSpec(heads=2, kv_heads=1, head_dim=16, scale=1.0, **bad)
    for bad in (dict(gate_full=True, gated=False), dict(gate_full=True, query_rank=8), dict(tile_rows=True, own_latent=False), dict(window=-3)):
        with pytest.raises(ConfigError):
            LatentAttentionSpec(heads=2, key_dim=8, value_dim=8, rank=16, scale=1.0, **bad)
    from dataclasses import replace
    spec = parse_config(NAROLORN["A"])
    with pytest.raises(ConfigError, match="streams"):
        replace(spec, core=replace(spec.core, streams=0))
    with pytest.raises(ConfigError, match="streams"):
        replace(spec, layers=(replace(spec.layers[0], streams=3),) + spec.layers[1:])
    RoutedExpertsSpec(experts=2, top=1, hidden=8, activation="swish_clamped", limit=1.0, router_bias="b")


def test_the_tensors_a_configuration_wants():
    wants = model_wants(architecture_entry("Narolorn"), parse_config(NAROLORN["A"]))
    shape = {n: w.shape for n, w in wants.items()}
    assert shape["embed"] == (150, 56) and "head" not in shape and shape["final.norm"] == (56,)
    for i in range(4):
        assert shape[f"l{i}.norm1"] == (56,) and shape[f"l{i}.hc1.in"] == shape[f"l{i}.hc1.out"] == (2,) and shape[f"l{i}.hc1.mix"] == (2, 2)
    assert shape["l0.mix.q"] == (36, 56) and shape["l0.mix.dkv"] == (24, 56) and shape["l0.mix.dkv.norm"] == (24,)
    assert shape["l0.mix.uk"] == (36, 24) and shape["l0.mix.uv"] == (60, 24) and shape["l0.mix.g"] == (60, 56) and shape["l0.mix.o"] == (56, 60)
    assert shape["l1.mix.q"] == (96, 56) and shape["l1.mix.k"] == (48, 56) and "l1.mix.v" not in shape and shape["l1.mix.o"] == (56, 96)
    assert shape["l1.mix.q.norm"] == (96,) and shape["l1.mix.k.norm"] == (48,)
    assert not any(n.startswith(("l1.mlp", "l1.norm2", "l1.hc2")) for n in shape)
    assert shape["l2.mix.q"] == (72, 56) and shape["l2.mix.k"] == (24, 56) and shape["l2.mix.v"] == (40, 56) and shape["l2.mix.o"] == (56, 120)
    assert shape["l0.mlp.router"] == (5, 56) and shape["l0.mlp.router.b"] == (5,) and shape["l0.mlp.shared.sg"] == (1, 56)
    assert shape["l0.mlp.e4.down"] == (56, 16) and shape["l0.mlp.shared.up"] == (24, 56)
    assert wants["l0.mlp.router"].role == wants["l0.mlp.shared.sg"].role == "matrix_fp32"
    c = model_wants(architecture_entry("Narolorn"), parse_config(NAROLORN["C"]))
    assert not any(n.startswith("l0.mlp.shared") for n in c) and "l0.mlp.router.b" in c


class Shell(DecoderModel):
    def __init__(self, spec):
        self.spec = spec


def test_what_the_runs_keep_between_steps():
    """Every pass of the loop has rows of its own; windows and chunks go with the rows; rows are as wide as the tile kernels like."""
    lat, keys, att, last = PagedKeysValues(1, 24, 13, planes=1), PagedKeysValues(2, 32, -20), PagedKeysValues(2, 32, 0), PagedKeysValues(1, 40, 40, planes=1)
    assert Shell(parse_config(NAROLORN["A"])).cache_needs() == [lat, keys, att, keys, att, keys, att, last]
    b = Shell(parse_config(NAROLORN["B"])).cache_needs()
    assert b[0] == PagedKeysValues(2, 128, 0) and b[1] == b[3] == PagedKeysValues(1, 128, 100, planes=1) and b[5] == PagedKeysValues(1, 128, 64, planes=1)
    assert b[6] == PagedKeysValues(1, 64, 0)                     # (values of 48 beside keys of 64)


@pytest.mark.parametrize("width, tile", [(64, 64), (50, 64), (47, 0), (96, 128), (128, 128), (129, 0), (192, 256), (256, 256), (257, 0), (8, 0)])
def test_the_width_of_cached_rows(width, tile):
    assert tile_width(width) == tile
    spec = LatentAttentionSpec(heads=1, key_dim=8, value_dim=8, rank=width, scale=1.0, tile_rows=True)
    assert spec.cache_dim == (tile or width)
    assert LatentAttentionSpec(heads=1, key_dim=8, value_dim=8, rank=width, scale=1.0).cache_dim == width


@pytest.mark.parametrize("seed", range(9500, 9530))
def test_drawn_configurations_parse(seed):
    cfg = random_narolorn(seed)
    spec = parse_config(cfg)
    assert [r.layer for r in spec.schedule] == P.layer_runs(cfg)
    assert model_wants(architecture_entry("Narolorn"), spec) and Shell(spec).cache_needs()


# ---- the plain implementation, and what the test models can tell apart ------------------------------------------------------

def test_the_plain_temperature_cap_and_masks():
    t = P.query_temperature([0, 3, 4, 7, 8], {"coef": 0.5, "every": 4})
    ln = lambda n: float(torch.log(torch.tensor(float(n), dtype=torch.float64)))
    assert torch.allclose(t, torch.tensor([1.0, 1 + 0.5 * ln(2), 1 + 0.5 * ln(2), 1 + 0.5 * ln(3), 1 + 0.5 * ln(3)], dtype=torch.float64))
    x = torch.tensor([-1e9, -3.0, 0.0, 0.1, 1e9], dtype=torch.float64)
    c = P.capped(x, 2.0)
    assert float(c[0]) == -2.0 and float(c[4]) == 2.0 and float(c[2]) == 0.0 and abs(float(c[3]) - 0.1) < 1e-3 and P.capped(x, None) is x
    w, k = P.window_mask(6, 2), P.chunk_mask(6, 4)
    assert w.sum(dim=1).tolist() == [1, 2, 2, 2, 2, 2] and k.sum(dim=1).tolist() == [1, 2, 3, 4, 1, 2]
    assert P.window_mask(6, None).sum() == P.causal_mask(6).sum() == 21


def test_the_plain_streams_mix_from_the_old_ones():
    g = torch.Generator().manual_seed(1)
    X, y = torch.randn(3, 2, 4, generator=g, dtype=torch.float64), torch.randn(2, 4, generator=g, dtype=torch.float64)
    mix, out = torch.randn(3, 3, generator=g, dtype=torch.float64), torch.randn(3, generator=g, dtype=torch.float64)
    assert torch.allclose(P.mix_streams(X, y, mix, out), torch.einsum("st,sij->tij", mix, X) + out[:, None, None] * y)


def test_plain_logits_of_a_prefix_do_not_depend_on_what_follows():
    cfg, w = P.load_plain(narolorn_folder("A"))
    toks = random_tokens(45, 150, 3)
    whole = P.forward(cfg, w, toks)
    for n in (1, 13, 14, 20, 41):
        assert torch.allclose(P.forward(cfg, w, toks[:n]), whole[:n], atol=1e-9)


CHANGES = {
    "window one longer": lambda c: c["layers"][0]["mixer"]["mask"].update(size=14),
    "window one shorter": lambda c: c["layers"][0]["mixer"]["mask"].update(size=12),
    "chunk one longer": lambda c: c["layers"][1]["mixer"]["mask"].update(size=21),
    "another temperature step": lambda c: c["layers"][2]["mixer"]["q_temp"].update(every=17),
    "no temperature": lambda c: c["layers"][2]["mixer"].pop("q_temp"),
    "no score cap": lambda c: c["layers"][2]["mixer"].pop("softcap"),
    "an expert's limit": lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0.7),
    "the shared expert's limit": lambda c: c["layers"][0]["mlp"]["shared"].update(limit=1.2),
    "one pass fewer": lambda c: c["loop"].update(times=2),
    "another rotation": lambda c: c["layers"][1]["mixer"]["rot"].update(base=101.0),
    "fewer experts": lambda c: c["layers"][0]["mlp"]["router"].update(top=1),
    "no logit cap": lambda c: c.pop("logit_softcap"),
    "another eps": lambda c: c["norm"].update(eps=4e-3),
}


@pytest.mark.parametrize("what", list(CHANGES))
def test_a_wrong_constant_shows_in_the_test_models_logits(what):
    """What the float32 comparisons of the GPU tests could not miss: the plain logits move by far more than their tolerance."""
    cfg, w = P.load_plain(narolorn_folder("A"))
    toks = random_tokens(60, 150, 9)
    right = P.forward(cfg, w, toks)
    other = copy.deepcopy(cfg)
    CHANGES[what](other)
    moved = (P.forward(other, w, toks) - right).abs().amax(dim=1)
    assert float(moved.max()) > 2e-4 * float(right.abs().max()), float(moved.max())
    if what == "window one longer":
        assert float(moved[:13].max()) == 0.0 and float(moved[13]) > 0
    if what == "chunk one longer":
        assert float(moved[:20].max()) == 0.0 and float(moved[20]) > 0


def test_the_first_token_is_still_seen_far_back():
    """Through the layers that see every position: the first of 200 tokens moves the last logits of every test model that has one."""
    for name in ("A", "B", "S"):
        cfg, w = P.load_plain(narolorn_folder(name))
        toks = random_tokens(200, cfg["vocab"], 5)
        moved = list(toks)
        moved[0] = (moved[0] + 1) % cfg["vocab"]
        d = float((P.forward(cfg, w, moved)[-1] - P.forward(cfg, w, toks)[-1]).abs().max())
        assert d > 1e-6, (name, d)
