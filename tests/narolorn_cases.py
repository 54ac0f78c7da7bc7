"""Tiny Narolorn configurations and model folders for the tests: every size differs between them, and values that one model may
happen to make equal or 1 (key and value widths, heads and kv heads, rotated and whole head widths, an expert's and the shared
expert's size and limit, experts and experts used, one stream, a window or chunk that is a multiple of the page size, a loop of one
pass, a layer without a feed-forward) are taken apart."""
from __future__ import annotations

import functools
import json
import tempfile
from pathlib import Path

import torch


def _att(heads, kv_heads, dim, vdim, scale, cap, temp, mlp):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if cap:
        m["softcap"] = cap
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def _latent(heads, dim, vdim, rank, scale, size, mlp):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": scale}
    if size:
        m["mask"] = {"size": size}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def _keys(heads, kv_heads, dim, scale, size, rot, mlp):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if size:
        m["mask"] = {"size": size}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "attention_2", "mixer": m, "mlp": mlp}


def _moe(experts, top, ff, limit, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


def _model(width, vocab, eps, streams, cap, layers, loop=None):
    cfg = {"architecture": "Narolorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "streams": streams, "layers": layers}
    if cap:
        cfg["logit_softcap"] = cap
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# A: small sizes, most of them no multiples of 16; values narrower and wider than keys; part of a head rotated; a layer without a
# feed-forward inside the loop, three passes
NAROLORN_A = _model(56, 150, 2e-3, 2, 9.0, [
    _latent(3, 12, 20, 24, 0.3, 13, _moe(5, 2, 16, 1.2, (24, 0.7))),
    _keys(4, 2, 24, 0.25, 20, (8, 100.0), None),
    _att(6, 2, 12, 20, 0.35, 4.0, (0.4, 16), _moe(4, 3, 24, 0.8, (8, 1.5))),
    _latent(2, 20, 12, 40, 0.25, 40, _moe(3, 1, 40, 2.0, (16, 1.0)))], loop=(1, 3, 3))
# B: the widths the tile kernels take: heads of 128 and 64, cached rows of 128 and (96 filled up to) 128 values; spans whose edges
# fall inside pages and tiles; four streams
NAROLORN_B = _model(128, 300, 1e-6, 4, 20.0, [
    _att(4, 2, 128, 128, 0.09, 6.0, (0.3, 50), _moe(3, 2, 32, 1.5, (64, 2.5))),
    _latent(4, 64, 64, 128, 0.125, 100, _moe(5, 5, 24, 1.0, (40, 1.5))),
    _keys(4, 2, 64, 0.12, 70, (64, 10000.0), _moe(4, 4, 32, 2.0, (32, 0.9))),
    _latent(3, 32, 48, 96, 0.17, 64, _moe(4, 2, 16, 1.2, (32, 2.0))),
    _att(2, 1, 64, 48, 0.125, 10.0, (0.5, 128), None)], loop=(1, 3, 2))
# C: what one model may make equal is apart: one stream; as many kv heads as heads; 20 query heads of a latent; one expert used, and
# all of them; no masks, no rotation, no caps, no temperature, no loop, no shared expert; cached rows wider than the tile kernels take
NAROLORN_C = _model(72, 97, 1e-5, 1, None, [
    _latent(20, 16, 24, 50, 0.25, None, _moe(4, 1, 12, 1.0)),
    _att(3, 3, 32, 32, 0.2, None, None, _moe(3, 3, 20, 1.5, (28, 1.5))),
    _keys(2, 2, 40, 0.2, None, None, _moe(1, 1, 30, 0.6, (10, 3.0))),
    _latent(2, 24, 8, 280, 0.2, 1, None),
    _keys(5, 1, 256, 0.06, 1, (128, 500.0), _moe(6, 5, 16, 1.1, (16, 0.5))),
    _att(20, 1, 16, 40, 0.3, 2.5, (1.0, 1), _moe(2, 1, 36, 1.0, (12, 1.0)))])
# D: nothing is a multiple of 4 or 8 (the products fall to the CUDA-core kernel in both precisions, no access is a vector's); five streams
NAROLORN_D = _model(50, 61, 1e-2, 5, 5.0, [
    _latent(3, 10, 6, 21, 0.4, 9, _moe(3, 2, 13, 0.9, (7, 1.4))),
    _att(3, 1, 10, 7, 0.5, 3.0, (0.6, 7), _moe(5, 2, 9, 1.3, (11, 0.8))),
    _keys(3, 1, 10, 0.4, 11, (6, 20.0), _moe(2, 1, 15, 1.0, (5, 2.0)))], loop=(0, 2, 2))
# S: like B, with every expert used: no router has a call to make, so every row is held to the tolerance in bfloat16 too
NAROLORN_S = _model(136, 210, 1e-6, 3, 15.0, [
    _latent(4, 64, 32, 64, 0.125, 48, _moe(4, 4, 32, 1.0, (48, 2.0))),
    _keys(6, 2, 96, 0.1, 64, (32, 1000.0), _moe(3, 3, 40, 1.5, (16, 1.0))),
    _att(8, 2, 64, 64, 0.125, 5.0, (0.4, 32), _moe(2, 2, 24, 2.0, (32, 0.8)))], loop=(0, 3, 2))

NAROLORN = {"A": NAROLORN_A, "B": NAROLORN_B, "C": NAROLORN_C, "D": NAROLORN_D, "S": NAROLORN_S}


def sharpen(tensors: dict, config: dict, q_gain: float = 1.7) -> dict:
    """Random weights of N(0, 0.02) leave every attention nearly uniform, every gated unit far inside its limits, every gate at a half
    and the caps without effect; a lost key, an edge that is one position off or a limit on the wrong side would not show. Here every
    matrix is rescaled so that unit inputs give unit outputs and the embedding to N(0, 1); the queries are scaled up further so that
    single keys stand out and scores reach their cap; the routers' biases so that most calls are clear; the streams' weights are spread (an
    error of a part's input is multiplied from sublayer to sublayer: with sharper queries and wilder mixes than these, bfloat16
    rounding would hide what is looked for; single keys that stand out among hundreds are the kernels' own tests)."""
    out = dict(tensors)
    g = torch.Generator().manual_seed(7)
    S = int(config["streams"])
    for name, t in tensors.items():
        f = t.float()
        if name == "embed":
            f = f * 50.0
        elif name.endswith((".hc1.in", ".hc2.in")):
            f = (1.0 + 0.3 * torch.randn(t.shape, generator=g)) / S
        elif name.endswith((".hc1.out", ".hc2.out")):
            f = 0.6 + 0.2 * torch.randn(t.shape, generator=g)
        elif name.endswith((".hc1.mix", ".hc2.mix")):
            f = 0.9 * torch.eye(S) + 0.1 * torch.randn(t.shape, generator=g)
        elif name.endswith("router.b"):
            f = torch.randn(t.shape, generator=g)
        elif t.dim() == 2:
            gain = q_gain if name.endswith("mix.q") else 1.2 if name.endswith("router") else 1.0
            f = f * (gain / (0.02 * t.shape[1] ** 0.5))
        elif name.endswith("mix.q.norm"):
            f = f * q_gain
        else:
            continue
        out[name] = f.to(t.dtype)
    return out


def random_narolorn(seed: int) -> dict:
    """A configuration drawn (seeded) from everything the design's keys allow at small sizes: any order of the three kinds of layers,
    any loop, one to six streams, layers without a feed-forward, spans of 1 to 130 positions or none, caps, temperatures, widths from
    4 to 128."""
    import random
    rng = random.Random(seed)
    widths = [4, 8, 12, 16, 24, 32, 48, 64, 96, 128]

    def mlp():
        if rng.random() < 0.15:
            return None
        experts = rng.randint(1, 8)
        shared = None if rng.random() < 0.15 else (rng.choice([4, 8, 20, 40]), rng.choice([0.5, 1.0, 2.5]))
        return _moe(experts, rng.randint(1, experts), rng.choice([8, 12, 16, 24, 40]), rng.choice([0.6, 1.0, 1.7]), shared)

    def size():
        return rng.choice([None, 1, 3, 16, 31, 64, 100, 130])

    layers = []
    for _ in range(rng.randint(2, 5)):
        r, kv = rng.random(), rng.choice([1, 1, 2, 3])
        dim = rng.choice(widths)
        scale = round(rng.uniform(0.6, 1.4) / dim ** 0.5, 4)
        vdim = dim if rng.random() < 0.5 else rng.choice(widths)
        if r < 0.35:
            layers.append(_latent(rng.choice([1, 2, 3, 5, 18]), dim, vdim, rng.choice([6, 16, 24, 48, 64, 96, 128, 200]), scale, size(), mlp()))
        elif r < 0.7:
            temp = None if rng.random() < 0.2 else (round(rng.uniform(0.1, 0.8), 3), rng.choice([1, 5, 16, 100]))
            layers.append(_att(kv * rng.choice([1, 2, 3, 8]), kv, dim, vdim, scale, rng.choice([None, 1.5, 4.0, 30.0]), temp, mlp()))
        else:
            rot = None if rng.random() < 0.2 else (dim if rng.random() < 0.4 else 2 * rng.randint(1, dim // 2), rng.choice([30.0, 10000.0]))
            layers.append(_keys(kv * rng.choice([1, 2, 3, 8]), kv, dim, scale, size(), rot, mlp()))
    n = len(layers)
    start = rng.randint(0, n - 1)
    loop = None if rng.random() < 0.3 else (start, rng.randint(start, n), rng.randint(1, 3))
    return _model(rng.choice([24, 40, 64, 72, 128]), rng.choice([53, 128, 300]), rng.choice([1e-6, 1e-5, 1e-4]), rng.randint(1, 6),
                  rng.choice([None, 4.0, 30.0]), layers, loop)


def narolorn_folder_of(config: dict, seed: int = 3, sharp: bool = True, q_gain: float = 1.7) -> Path:
    """A temporary model folder for any configuration (random, by default sharpened weights); never inside the repository."""
    from jllm_serve_b200.config import parse_config
    from jllm_serve_b200.config.registry import architecture_entry, model_type_of
    from jllm_serve_b200.engine.model import model_wants
    from jllm_serve_b200.weights import random_tensors, write_safetensors
    wants = model_wants(architecture_entry(model_type_of(config)), parse_config(config))
    tensors = random_tensors(wants, seed, "cpu", torch.bfloat16)
    if sharp:
        tensors = sharpen(tensors, config, q_gain)
    d = Path(tempfile.mkdtemp(prefix="jllm_narolorn_"))
    (d / "config.json").write_text(json.dumps(config, indent=1))
    write_safetensors(d / "model.safetensors", tensors, {"format": "pt"})
    return d


@functools.lru_cache(maxsize=None)
def narolorn_folder(name: str, seed: int = 3, sharp: bool = True) -> Path:
    return narolorn_folder_of(NAROLORN[name], seed, sharp)
