"""Tiny Fusazen configurations and model folders for the tests: every size differs between them, and values that one model may
happen to make equal or 1 (key and value widths, two maps and the value's width, heads and kv heads, rotated and whole map widths,
the masks of a layer and of the layer whose keys it reads, the decay's rank and a head's width, a chunk that is a multiple of the
page size, a layer without a feed-forward) are taken apart."""
from __future__ import annotations

import copy
import functools
import json
import tempfile
from pathlib import Path

import torch


def _delta(heads, dim, rank, mlp):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim, "decay_rank": rank}, "mlp": mlp}


def _diff(heads, kv_heads, dim, vdim, scale, diff, size, rot, mlp, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if size:
        m["mask"] = {"size": size}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def _whole(heads, kv_heads, dim, vdim, scale, size, mlp):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size:
        m["mask"] = {"size": size}
    return {"type": "attention_2", "mixer": m, "mlp": mlp}


def _ff(n):
    return {"kind": "dense", "ff": n}


def _model(width, vocab, eps, taps, scale, layers):
    cfg = {"architecture": "Fusazen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "canon": {"taps": taps}, "layers": layers}
    if scale is not None:
        cfg["embedding"] = {"scale": scale}
    return cfg


# A: small sizes, most of them no multiples of 16; values narrower and wider than two maps; part of a map rotated; a layer that
# reads the keys of the layer in front of it under a LARGER mask, and one under a smaller; a layer without a feed-forward
FUSAZEN_A = _model(56, 150, 2e-5, 3, 1.5, [
    _whole(6, 2, 24, 16, 0.3, 20, _ff(40)),
    _delta(3, 12, 5, _ff(72)),
    _diff(4, 2, 12, 20, 0.35, 0.4, 13, (8, 100.0), None),
    _diff(4, 2, 12, 20, 0.3, 0.3, 40, (8, 100.0), _ff(24), kv_from=2),
    _delta(2, 20, 8, None),
    _diff(4, 2, 12, 20, 0.4, 0.5, 7, (8, 100.0), _ff(32), kv_from=2)])
# B: the widths the tile and chunk kernels take: maps of 64 under values of 128, maps of 32 under values of 64, heads of 128 and 64;
# recurrences of 64 and 128 channels; chunks whose edges fall inside pages and tiles
FUSAZEN_B = _model(128, 300, 1e-6, 4, 0.25, [
    _delta(4, 64, 16, _ff(192)),
    _diff(4, 2, 64, 128, 0.125, 0.55, 100, (32, 10000.0), _ff(160)),
    _whole(4, 1, 128, 128, 0.09, 70, _ff(96)),
    _diff(4, 2, 64, 128, 0.125, 0.35, 100, (32, 10000.0), _ff(128), kv_from=1),
    _delta(1, 128, 24, None),
    _diff(2, 1, 32, 64, 0.2, 0.2, 128, (32, 500.0), _ff(64))])
# C: what one model may make equal is apart: 20 query heads to a kv head; a convolution of 1 tap; chunks of 1 position (a row sees
# itself alone); no mask, no rotation; maps whose rows are wider than the tile kernels take; values of one channel group;
# recurrences that the chunk kernels do not take; no embedding scale key
FUSAZEN_C = _model(72, 97, 1e-5, 1, None, [
    _diff(20, 1, 16, 16, 0.25, 0.45, 33, None, _ff(30)),
    _delta(2, 50, 12, _ff(44)),
    _whole(3, 3, 32, 8, 0.2, 1, _ff(20)),
    _diff(2, 2, 160, 40, 0.08, 0.25, None, (160, 10000.0), None),
    _whole(2, 1, 256, 256, 0.06, None, _ff(36)),
    _diff(2, 2, 160, 40, 0.08, 0.5, 21, (160, 10000.0), _ff(28), kv_from=3)])
# D: nothing is a multiple of 4 or 8 (the products fall to the CUDA-core kernel in both precisions, no access is a vector's); seven taps
FUSAZEN_D = _model(50, 61, 1e-4, 7, 2.0, [
    _diff(3, 1, 10, 6, 0.4, 0.4, 9, (6, 20.0), _ff(21)),
    _delta(3, 7, 3, _ff(13)),
    _whole(3, 3, 5, 9, 0.5, 11, _ff(10)),
    _diff(3, 1, 10, 6, 0.35, 0.6, 30, (6, 20.0), _ff(15), kv_from=0)])

FUSAZEN = {"A": FUSAZEN_A, "B": FUSAZEN_B, "C": FUSAZEN_C, "D": FUSAZEN_D}


def stored_config(config: dict) -> dict:
    """The configuration as a model folder has it: the decay's rank is the stored tensor's own and in no key."""
    out = copy.deepcopy(config)
    for layer in out["layers"]:
        layer["mixer"].pop("decay_rank", None)
    return out


def sharpen(tensors: dict, config: dict, q_gain: float = 4.0) -> dict:
    """Random weights of N(0, 0.02) leave every activation tiny: every attention nearly uniform, both maps alike, every decay the
    same; a lost key, a chunk's edge that is one position off or a stale state would not show. Here every matrix is rescaled so
    that unit inputs give unit outputs and the embedding to N(0, 1) behind its scale; the queries of the differential attentions are
    scaled up further so that single keys stand out (the other attention's are normed: its factors per head are scaled instead); the
    small vectors (biases, the four vectors of lambda, the convolution) to sizes that matter."""
    out = dict(tensors)
    emb = float(config.get("embedding", {}).get("scale", 1.0))
    kinds = [l["type"] for l in config["layers"]]
    for name, t in tensors.items():
        f = t.float()
        layer = int(name[1:name.index(".")]) if name[0] == "l" and name[1].isdigit() else -1
        if name == "embed":
            f = f * (50.0 / emb)
        elif name.endswith("canon1"):
            f = f * 20.0
        elif t.dim() == 2:
            gain = q_gain if name.endswith("mix.q") and kinds[layer] == "attention" else 1.0
            f = f * (gain / (0.02 * t.shape[1] ** 0.5))
        elif name.endswith(("lq1", "lk1", "lq2", "lk2")):
            f = f * (50.0 * 0.4 ** 0.5 / t.shape[0] ** 0.25)
        elif name.endswith(".temp"):
            f = f * q_gain * 0.6
        elif name.endswith((".w0", ".a.b")):
            f = f * 60.0
        elif name.endswith((".up.b", ".down.b")):
            f = f * 20.0
        else:
            continue
        out[name] = f.to(t.dtype)
    return out


def random_fusazen(seed: int) -> dict:
    """A configuration drawn (seeded) from everything the design's keys allow at small sizes: any order of the three kinds of
    layers, layers that read any earlier differential layer's keys under a mask of their own, layers without a feed-forward, map
    and value widths from 4 to 128, rotations of a part or all of a map or none, chunks of 1 to 130 positions or none, 1 to 5 taps."""
    import random
    rng = random.Random(seed)
    widths = [4, 8, 12, 16, 24, 32, 48, 64, 96, 128]

    def ff():
        return None if rng.random() < 0.15 else _ff(rng.choice([8, 24, 40, 64, 100]))

    def size():
        return rng.choice([None, 1, 3, 16, 31, 64, 100, 130])

    layers, sources = [], {}
    for i in range(rng.randint(3, 6)):
        r = rng.random()
        if r < 0.3:
            layers.append(_delta(rng.choice([1, 2, 3, 5]), rng.choice([6, 8, 12, 16, 32, 64, 72, 128]), rng.choice([2, 6, 8, 16]), ff()))
        elif r < 0.55:
            kv = rng.choice([1, 1, 2, 3])
            dim = rng.choice(widths)
            vdim = dim if rng.random() < 0.5 else rng.choice(widths)
            layers.append(_whole(kv * rng.choice([1, 2, 3, 8]), kv, dim, vdim, round(rng.uniform(0.6, 1.4) / dim ** 0.5, 4), size(), ff()))
        elif r < 0.8 or not sources:
            kv = rng.choice([1, 2, 3])
            dim = rng.choice(widths)
            vdim = 2 * dim if rng.random() < 0.5 else rng.choice(widths)
            rot = None if rng.random() < 0.2 else (dim if rng.random() < 0.4 else 2 * rng.randint(1, dim // 2), rng.choice([30.0, 10000.0]))
            args = (kv * rng.choice([1, 2, 3, 9]), kv, dim, vdim, round(rng.uniform(0.6, 1.4) / dim ** 0.5, 4))
            sources[i] = (args, rot)
            layers.append(_diff(*args, round(rng.uniform(0.1, 0.5), 3), size(), rot, ff()))
        else:
            j = rng.choice(list(sources))
            args, rot = sources[j]
            layers.append(_diff(*args, round(rng.uniform(0.1, 0.5), 3), size(), rot, ff(), kv_from=j))
    return _model(rng.choice([24, 40, 64, 72, 128]), rng.choice([53, 128, 300]), rng.choice([1e-6, 1e-5, 1e-4]), rng.randint(1, 5),
                  rng.choice([0.5, 1.0, 3.0]), layers)


def fusazen_folder_of(config: dict, seed: int = 3, sharp: bool = True, q_gain: float = 4.0) -> Path:
    """A temporary model folder for any configuration (random, by default sharpened weights); never inside the repository."""
    from jllm_serve_b200.config import parse_config
    from jllm_serve_b200.config.registry import architecture_entry, model_type_of
    from jllm_serve_b200.engine.model import model_wants
    from jllm_serve_b200.weights import random_tensors, write_safetensors
    wants = model_wants(architecture_entry(model_type_of(config)), parse_config(config))
    tensors = random_tensors(wants, seed, "cpu", torch.bfloat16)
    if sharp:
        tensors = sharpen(tensors, config, q_gain)
    d = Path(tempfile.mkdtemp(prefix="jllm_fusazen_"))
    (d / "config.json").write_text(json.dumps(stored_config(config), indent=1))
    write_safetensors(d / "model.safetensors", tensors, {"format": "pt"})
    return d


@functools.lru_cache(maxsize=None)
def fusazen_folder(name: str, seed: int = 3, sharp: bool = True) -> Path:
    return fusazen_folder_of(FUSAZEN[name], seed, sharp)
