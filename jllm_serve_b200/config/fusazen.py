"""The Fusazen parser: config.json of `architecture: Fusazen` -> a `Decoder` spec.

Fusazen lists its layers one by one (`layers`: `type`, `mixer`, `mlp`). A layer is pre-norm: a token mixer and a feed-forward
(`mlp: null` = none), each behind an RMS norm of its own. What the mixer reads is its normed rows plus a causal convolution
of `canon.taps` taps over them (one table per layer). The embedded rows are multiplied by `embedding.scale`. The mixers:

* `general_delta`: a recurrence whose transition is a decay per key channel minus a rank-one removal (`heads`, `dim` channels
  for keys and values alike; the decay's low-rank width is read off the stored tensor).
* `attention`: differential softmax attention without biases: two maps of `dim` values per query and key head over the same
  values of `vdim`, rotary positions on the pairs (i, i + dims / 2) of the first `rot.dims` values of each map, the score
  multiplier `scale`, a chunk mask (`mask.size`), the constant `diff`. With `kv_from: j` the layer has no key and value
  projections and reads what layer j cached.
* `attention_2`: softmax attention without positions: an RMS norm over all rows of the query (key) projection at once, a stored
  factor per query head on the scores, `scale`, a chunk mask.

The feed-forward (`mlp.kind` dense): two matrices with biases around the square of relu.

Keys read: `width`, `vocab`, `norm.eps`, `canon.taps`, `embedding.scale`, `layers[i].type | mixer | mlp`. Optional: `eos`,
`max_positions` (the rotary tables' length; the engine's context), a `mask` or `rot` that is left out (no mask, no rotation).
"""
from __future__ import annotations

import math

from .reader import ConfigReader
from .specs import (AttentionNames, ConfigError, Core, Decoder, DenseMlpSpec, GeneralDeltaSpec, GqaAttentionSpec, LayerNames,
                    LayerRun, LayerSpec, ModelNames, NormSpec, RopeTableSpec)

FUSAZEN_NAMES = ModelNames(embedding="embed", layer="l{}.", final_norm="final.norm", head="head")
FUSAZEN_LAYER_NAMES = LayerNames(mixer="mix.", feed_forward="mlp.", mixer_norm="norm1", feed_forward_norm="norm2")
FUSAZEN_ATTENTION_NAMES = AttentionNames(q="q", k="k", v="v", o="o", q_norm="q.norm", k_norm="k.norm", head_scale="temp",
                                         lambdas=("lq1", "lk1", "lq2", "lk2"))
INPUT_CONV = "canon1"
DEFAULT_POSITIONS = 1 << 17


class _Tables:
    """The model's rotary tables: mixers with the same rotation share one."""

    def __init__(self):
        self.specs = []

    def index(self, spec: RopeTableSpec) -> int:
        if spec not in self.specs:
            self.specs.append(spec)
        return self.specs.index(spec)


def _chunk(m: ConfigReader) -> int:
    mask = m.mapping("mask")
    return mask.positive("size") if mask is not None else 0


def _differential(m: ConfigReader, eps: float, tables: _Tables) -> GqaAttentionSpec:
    rot, dim, table = m.mapping("rot"), m.positive("dim"), -1
    if rot is not None:
        if rot.positive("dims") > dim:
            raise ConfigError(f"{rot.where}: dims={rot.positive('dims')} exceeds the head's dim={dim}")
        table = tables.index(RopeTableSpec(rotary_dim=rot.positive("dims"), theta=rot.number("base"), pairing="half"))
    return GqaAttentionSpec(heads=m.positive("heads"), kv_heads=m.positive("kv_heads"), head_dim=dim, value_dim=m.positive("vdim"),
                            rope_table=table, scale=m.number("scale"), chunk=_chunk(m), maps=2, diff=m.number("diff"),
                            diff_norm_eps=eps, own_kv=not m.has("kv_from"), names=FUSAZEN_ATTENTION_NAMES)


def _whole_norm(m: ConfigReader, eps: float) -> GqaAttentionSpec:
    return GqaAttentionSpec(heads=m.positive("heads"), kv_heads=m.positive("kv_heads"), head_dim=m.positive("dim"),
                            value_dim=m.positive("vdim"), rope_table=-1, qk_norm=True, qk_norm_over="all", qk_norm_eps=eps,
                            scale=m.number("scale"), head_scale=True, chunk=_chunk(m), names=FUSAZEN_ATTENTION_NAMES)


def _mixer(kind: str, m: ConfigReader, eps: float, tables: _Tables):
    if kind == "general_delta":
        dim = m.positive("dim")
        return GeneralDeltaSpec(heads=m.positive("heads"), key_dim=dim, value_dim=dim, decay_rate=math.exp(-0.5),
                                decay_rank=m.positive("decay_rank", -1) if m.has("decay_rank") else -1, norm_eps=eps)
    if kind == "attention":
        return _differential(m, eps, tables)
    if kind == "attention_2":
        return _whole_norm(m, eps)
    raise ConfigError(f"{m.where}: unknown layer type {kind!r} (built: general_delta, attention, attention_2)")


def _feed_forward(f: ConfigReader | None):
    if f is None:
        return None
    kind = f.string("kind", "dense")
    if kind != "dense":
        raise ConfigError(f"{f.where}: unknown feed-forward kind {kind!r} (built: dense)")
    return DenseMlpSpec(hidden=f.positive("ff"), activation="relu2", names=("up", "down"), bias_names=("up.b", "down.b"))


def parse_fusazen(values: dict) -> Decoder:
    c = ConfigReader(values)
    dim, vocab = c.positive("width"), c.positive("vocab")
    norm, canon, emb = c.mapping("norm"), c.mapping("canon"), c.mapping("embedding")
    eps = norm.number("eps", 1e-6) if norm is not None else 1e-6
    if canon is None:
        raise ConfigError("config.json: required key 'canon' is missing")
    taps = canon.positive("taps")
    entries = values.get("layers")
    if not isinstance(entries, list) or not entries:
        raise ConfigError("config.json: 'layers' must be a list with at least one layer")
    norm_spec = NormSpec("rmsnorm", eps, gain_name="")
    tables = _Tables()
    specs, schedule = [], []
    for i, e in enumerate(entries):
        r = ConfigReader(e, f"config.json:layers[{i}]")
        m = r.mapping("mixer")
        if m is None:
            raise ConfigError(f"{r.where}: required key 'mixer' is missing")
        mixer = _mixer(r.string("type"), m, eps, tables)
        source = None
        if mixer.kind == "gqa_attention" and not mixer.own_kv:
            source = m.integer("kv_from")
            if not 0 <= source < i:
                raise ConfigError(f"{m.where}: kv_from={source} names no earlier layer")
            own = specs[source].mixer
            shape = ("kv_heads", "head_dim", "v_dim", "maps", "rope_table")
            if own.kind != "gqa_attention" or not own.own_kv or any(getattr(own, k) != getattr(mixer, k) for k in shape):
                raise ConfigError(f"{m.where}: kv_from={source} is no attention with keys and values of this layer's sizes")
        specs.append(LayerSpec(mixer, _feed_forward(r.mapping("mlp")), norm_spec, "pre_norm", FUSAZEN_LAYER_NAMES,
                               input_conv=INPUT_CONV, input_conv_taps=taps))
        schedule.append(LayerRun(i, source))
    kinds = [s.mixer.kind for s in specs]
    twos = sum(getattr(s.mixer, "maps", 1) == 2 for s in specs)
    description = (f"Fusazen width={dim} vocab={vocab} layers={len(specs)} (delta rule {kinds.count('general_delta')}, differential "
                   f"attention {twos}, attention {kinds.count('gqa_attention') - twos})")
    core = Core(architecture="Fusazen", model_type="Fusazen", dim=dim, layers=len(specs), vocab=vocab, norm_eps=eps, tied=False,
                bos=-1, eos=c.int_list("eos"), max_positions=c.positive("max_positions", DEFAULT_POSITIONS),
                description=description, embedding_scale=emb.number("scale", 1.0) if emb is not None else 1.0)
    return Decoder(core, tuple(specs), tuple(tables.specs), norm_spec, tuple(schedule), FUSAZEN_NAMES)
