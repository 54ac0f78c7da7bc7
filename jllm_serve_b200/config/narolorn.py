"""The Narolorn parser: config.json of `architecture: Narolorn` -> a `Decoder` spec.

Narolorn lists its layers one by one (`layers`: `type`, `mixer`, `mlp`); `loop` passes layers start .. stop - 1 `times` times in a
row with the same weights, each pass with a cache of its own. The residual is `streams` streams that are mixed behind every part
(`hyper_connections`: the tensors `<layer>.hc1.*` and `<layer>.hc2.*`). The mixers:

* `attention`: grouped-query softmax attention without positions; queries grow with their position (`q_temp.coef | every`), scores
  are multiplied by `scale` and capped (`softcap`).
* `latent_attention`: attention over a cached latent of `kv_rank` values under a sliding window (`mask.size`), with a sigmoid gate
  per value of the concatenated heads.
* `attention_2`: RMS norms over all rows of the query (key) projection at once, rotary positions on the pairs (i, i + dims / 2) of the
  first `rot.dims` values of each head, a chunk mask (`mask.size`); the values are the keys as projected.

The feed-forward (`mlp.kind` moe): clamped gated units, of which a token uses `router.top` by a softmax over the chosen logits (with a
bias per expert), beside a shared one with a gate per token. The head is the embedding, its result capped (`logit_softcap`).

Keys read: `width`, `vocab`, `streams`, `logit_softcap`, `norm.eps`, `loop.start | stop | times`, `layers[i].type | mixer | mlp`; of a
mixer `heads`, `kv_heads`, `dim`, `vdim`, `kv_rank`, `scale`, `softcap`, `q_temp.coef | every`, `mask.size`, `rot.dims | base`; of an
`mlp` `kind`, `expert.ff | limit`, `router.experts | top`, `shared.ff | limit`. Optional: `eos`, `max_positions` (the rotary tables'
length; the engine's context), and whatever is left out means without: a `mask`, `rot`, `q_temp`, `softcap`, `logit_softcap`, `loop`, `mlp`
or `shared`.
"""
from __future__ import annotations

from .reader import ConfigReader
from .specs import (AttentionNames, ConfigError, Core, Decoder, DenseGluSpec, GqaAttentionSpec, LatentAttentionSpec, LayerNames,
                    LayerRun, LayerSpec, ModelNames, NormSpec, RopeTableSpec, RoutedExpertsSpec)

NAROLORN_NAMES = ModelNames(embedding="embed", layer="l{}.", final_norm="final.norm", head="embed")
NAROLORN_LAYER_NAMES = LayerNames(mixer="mix.", feed_forward="mlp.", mixer_norm="norm1", feed_forward_norm="norm2")
NAROLORN_ATTENTION_NAMES = AttentionNames(q="q", k="k", v="v", o="o", q_norm="q.norm", k_norm="k.norm")
GLU_NAMES = ("gate", "up", "down")
DEFAULT_POSITIONS = 1 << 17


def _span(m: ConfigReader) -> int:
    mask = m.mapping("mask")
    return mask.positive("size") if mask is not None else 0


def _optional_number(c: ConfigReader, key: str) -> float:
    if not c.has(key):
        return 0.0
    value = c.number(key)
    if not value > 0:
        raise ConfigError(f"{c.where}: {key}={value} must be positive")
    return value


def _capped(m: ConfigReader) -> GqaAttentionSpec:
    temp = m.mapping("q_temp")
    return GqaAttentionSpec(heads=m.positive("heads"), kv_heads=m.positive("kv_heads"), head_dim=m.positive("dim"),
                            value_dim=m.positive("vdim"), rope_table=-1, scale=m.number("scale"), softcap=_optional_number(m, "softcap"),
                            temp_every=temp.positive("every") if temp is not None else 0,
                            temp_coef=temp.number("coef") if temp is not None else 0.0, names=NAROLORN_ATTENTION_NAMES)


def _latent(m: ConfigReader, eps: float) -> LatentAttentionSpec:
    return LatentAttentionSpec(heads=m.positive("heads"), key_dim=m.positive("dim"), value_dim=m.positive("vdim"),
                               rank=m.positive("kv_rank"), scale=m.number("scale"), norm_eps=eps, window=_span(m), gated=True,
                               gate_full=True, tile_rows=True)


def _keys_as_values(m: ConfigReader, eps: float, tables: list) -> GqaAttentionSpec:
    dim, rot, table = m.positive("dim"), m.mapping("rot"), -1
    if m.has("vdim") and m.positive("vdim") != dim:
        raise ConfigError(f"{m.where}: vdim={m.positive('vdim')} must equal dim={dim}: the values are the keys")
    if rot is not None:
        if rot.positive("dims") > dim:
            raise ConfigError(f"{rot.where}: dims={rot.positive('dims')} exceeds the head's dim={dim}")
        spec = RopeTableSpec(rotary_dim=rot.positive("dims"), theta=rot.number("base"), pairing="half")
        if spec not in tables:
            tables.append(spec)
        table = tables.index(spec)
    return GqaAttentionSpec(heads=m.positive("heads"), kv_heads=m.positive("kv_heads"), head_dim=dim, value_dim=dim, rope_table=table,
                            qk_norm=True, qk_norm_over="all", qk_norm_eps=eps, scale=m.number("scale"), chunk=_span(m),
                            keys_as_values=True, names=NAROLORN_ATTENTION_NAMES)


def _mixer(kind: str, m: ConfigReader, eps: float, tables: list):
    if kind == "attention":
        return _capped(m)
    if kind == "latent_attention":
        return _latent(m, eps)
    if kind == "attention_2":
        return _keys_as_values(m, eps, tables)
    raise ConfigError(f"{m.where}: unknown layer type {kind!r} (built: attention, latent_attention, attention_2)")


def _feed_forward(f: ConfigReader | None):
    if f is None:
        return None
    kind = f.string("kind", "moe")
    if kind != "moe":
        raise ConfigError(f"{f.where}: unknown feed-forward kind {kind!r} (built: moe)")
    expert, router, shared = f.mapping("expert"), f.mapping("router"), f.mapping("shared")
    if expert is None or router is None:
        raise ConfigError(f"{f.where}: a mixture of experts needs 'expert' and 'router'")
    unit = DenseGluSpec(hidden=shared.positive("ff"), activation="swish_clamped", names=GLU_NAMES,
                        limit=shared.number("limit")) if shared is not None else None
    return RoutedExpertsSpec(experts=router.positive("experts"), top=router.positive("top"), hidden=expert.positive("ff"), scale=1.0,
                             correction=False, normalize=True, score="softmax", activation="swish_clamped", limit=expert.number("limit"),
                             weight_on="output", router_bias="router.b", shared=unit,
                             shared_gate="shared.sg" if unit is not None else "")


def _schedule(loop: ConfigReader | None, layers: int) -> tuple:
    """Layers [start, stop) `times` times in a row, the others once."""
    if loop is None:
        return tuple(LayerRun(i) for i in range(layers))
    start, stop, times = loop.integer("start"), loop.integer("stop"), loop.positive("times")
    if not 0 <= start <= stop <= layers:
        raise ConfigError(f"{loop.where}: start={start} and stop={stop} must lie in order in [0, {layers}]")
    order = list(range(start)) + list(range(start, stop)) * times + list(range(stop, layers))
    return tuple(LayerRun(i) for i in order)


def parse_narolorn(values: dict) -> Decoder:
    c = ConfigReader(values)
    dim, vocab, streams = c.positive("width"), c.positive("vocab"), c.positive("streams", 1)
    if streams > 16:
        raise ConfigError(f"config.json: streams={streams} (built: up to 16)")
    norm = c.mapping("norm")
    eps = norm.number("eps", 1e-6) if norm is not None else 1e-6
    entries = values.get("layers")
    if not isinstance(entries, list) or not entries:
        raise ConfigError("config.json: 'layers' must be a list with at least one layer")
    norm_spec = NormSpec("rmsnorm", eps, gain_name="")
    tables, specs = [], []
    for i, e in enumerate(entries):
        r = ConfigReader(e, f"config.json:layers[{i}]")
        m = r.mapping("mixer")
        if m is None:
            raise ConfigError(f"{r.where}: required key 'mixer' is missing")
        specs.append(LayerSpec(_mixer(r.string("type"), m, eps, tables), _feed_forward(r.mapping("mlp")), norm_spec,
                               "hyper_connections", NAROLORN_LAYER_NAMES, streams=streams))
    schedule = _schedule(c.mapping("loop"), len(specs))
    latent = sum(s.mixer.kind == "latent_attention" for s in specs)
    tied = sum(getattr(s.mixer, "keys_as_values", False) for s in specs)
    description = (f"Narolorn width={dim} vocab={vocab} layers={len(specs)} runs={len(schedule)} streams={streams} (latent attention "
                   f"{latent}, keys as values {tied}, attention {len(specs) - latent - tied})")
    core = Core(architecture="Narolorn", model_type="Narolorn", dim=dim, layers=len(specs), vocab=vocab, norm_eps=eps, tied=True,
                bos=-1, eos=c.int_list("eos"), max_positions=c.positive("max_positions", DEFAULT_POSITIONS), description=description,
                logit_softcap=_optional_number(c, "logit_softcap"), streams=streams)
    return Decoder(core, tuple(specs), tuple(tables), norm_spec, schedule, NAROLORN_NAMES)
