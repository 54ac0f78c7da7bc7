"""Plain, slow implementation of the Narolorn decoder: the oracle of its tests.

Narolorn is a small decoder-only design: an embedding that is also the head, a list of layers of which a run in the middle may be
passed several times with the same weights (each pass with a cache of its own), a final RMS norm, capped logits. There is no one
residual stream: `streams` copies travel side by side, every part reads a weighted sum of them, and behind every part the copies
are mixed among each other and each takes the part's result with a weight of its own. A mixer is an attention whose queries grow
with the position and whose scores are capped (`attention`), an attention over a cached latent under a sliding window with a gate
on its result (`latent_attention`), or an attention under a chunk mask whose values are its unrotated, unnormed keys
(`attention_2`). The feed-forward is a mixture of clamped gated units beside a shared one with a gate per token.

Whole sequences, one function per mechanism, tensors on the CPU in float64 unless the caller says otherwise. It shares no code with
the product: it reads config.json and model.safetensors with its own few lines and writes every sum as a loop or a plain torch
expression.

Notation (h: the rows a part reads [T, width]; Wn: the tensor named n, stored [out, in]; p: position):
  rms(x)       = x / sqrt(mean(x^2) + eps);  norm(x, n) = rms(x) * n
  temperature  q <- q (1 + coef ln(floor((p + 1) / every) + 1))
  cap          s <- c tanh(s / c)
  latent       c_t = norm(Wdkv h_t, n); per head k = Wuk c, v = Wuv c; y = Wo (concat_heads(o) * sigmoid(Wg h))
  window       row t sees j with 0 <= t - j < size;   chunk  row t sees j <= t with j // size = t // size
  attention_2  q <- norm(Wq h, nq), k <- norm(Wk h, nk) over ALL rows of the projection, then rotated; values Wk h as it is
  rotary       f_i = base^(-2i / dims), i < dims / 2; the pair (a, b) = values (i, i + dims / 2) at position p ->
               (a cos(p f_i) - b sin(p f_i), b cos(p f_i) + a sin(p f_i)); values from `dims` on do not rotate
  unit         g = min(Wgate h, L), u = clamp(Wup h, -L, L);  Wdown (g sigmoid(1.702 g) (u + 1))
  experts      z = Wr h + b; the `top` largest z, weights softmax over those; + sigmoid(Wsg h) * shared unit(h)
  sublayer     u = sum_s in[s] X_s;  y = part(norm(u));  X_t <- sum_s mix[s, t] X_s + out[t] y
"""
from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import numpy as np
import torch


def read_tensors(path) -> dict:
    """safetensors: u64 little-endian header length, JSON header, raw data."""
    raw = Path(path).read_bytes()
    (hlen,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8:8 + hlen])
    data = raw[8 + hlen:]
    kinds = {"F32": np.float32, "F64": np.float64, "I32": np.int32, "I64": np.int64, "F16": np.float16}
    out = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        lo, hi = meta["data_offsets"]
        if meta["dtype"] == "BF16":
            arr = (np.frombuffer(data[lo:hi], dtype=np.uint16).astype(np.uint32) << 16).view(np.float32)
        else:
            arr = np.frombuffer(data[lo:hi], dtype=kinds[meta["dtype"]])
        out[name] = torch.from_numpy(arr.reshape(meta["shape"]).copy())
    return out


def load_plain(folder, dtype=torch.float64):
    folder = Path(folder)
    cfg = json.loads((folder / "config.json").read_text())
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in read_tensors(folder / "model.safetensors").items()}
    return cfg, w


# ---- mechanisms, one function each --------------------------------------------------------------------------------

def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm(x, gain, eps):
    return rms(x, eps) * gain


def capped(x, cap):
    """x itself where nothing caps it (None)."""
    return x if cap is None else cap * torch.tanh(x / cap)


def query_temperature(positions, temp):
    """[T] factors on the queries; `temp` None: ones."""
    out = torch.ones(len(positions), dtype=torch.float64)
    if temp is not None:
        coef, every = float(temp["coef"]), int(temp["every"])
        for i, p in enumerate(positions):
            out[i] = 1.0 + coef * math.log((int(p) + 1) // every + 1)
    return out


def rotate_half(x, positions, rot):
    """x [T, heads, dim]: the first rot.dims values of every head rotated by the position's angles, value i with i + dims / 2."""
    if rot is None:
        return x
    dims, base = int(rot["dims"]), float(rot["base"])
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    angle = positions.to(torch.float64)[:, None] * f[None, :]
    c, s = torch.cos(angle).to(x.dtype)[:, None, :], torch.sin(angle).to(x.dtype)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def causal_mask(T):
    """[T, T] bool: which keys a row sees."""
    t = torch.arange(T)
    return t[None, :] <= t[:, None]


def window_mask(T, size):
    t = torch.arange(T)
    return causal_mask(T) if size is None else causal_mask(T) & (t[:, None] - t[None, :] < size)


def chunk_mask(T, size):
    t = torch.arange(T)
    return causal_mask(T) if size is None else causal_mask(T) & (t[None, :] // size == t[:, None] // size)


def softmax_attention(q, k, v, scale, seen, cap=None):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] -> [T, H, vdim]; query head h reads key head h // (H / G)."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = torch.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        s = capped((q[:, h] @ k[:, h // per].T) * scale, cap).masked_fill(~seen, float("-inf"))
        out[:, h] = torch.softmax(s, dim=-1) @ v[:, h // per]
    return out


def size_of(m):
    return int(m["mask"]["size"]) if m.get("mask") is not None else None


def capped_attention(h, w, p, m):
    T, H, G, dim, vdim = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    factor = query_temperature(range(T), m.get("q_temp")).to(h.dtype)
    q = (h @ w[p + "q"].T).view(T, H, dim) * factor[:, None, None]
    k, v = (h @ w[p + "k"].T).view(T, G, dim), (h @ w[p + "v"].T).view(T, G, vdim)
    o = softmax_attention(q, k, v, float(m["scale"]), causal_mask(T), m.get("softcap"))
    return o.reshape(T, H * vdim) @ w[p + "o"].T


def latent_attention(h, w, p, m, eps):
    T, H, dim, vdim = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    c = norm(h @ w[p + "dkv"].T, w[p + "dkv.norm"], eps)
    q = (h @ w[p + "q"].T).view(T, H, dim)
    k, v = (c @ w[p + "uk"].T).view(T, H, dim), (c @ w[p + "uv"].T).view(T, H, vdim)
    o = softmax_attention(q, k, v, float(m["scale"]), window_mask(T, size_of(m))).reshape(T, H * vdim)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def keys_as_values_attention(h, w, p, m, eps):
    T, H, G, dim = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    pos = torch.arange(T)
    raw = h @ w[p + "k"].T
    q = rotate_half(norm(h @ w[p + "q"].T, w[p + "q.norm"], eps).view(T, H, dim), pos, m.get("rot"))
    k = rotate_half(norm(raw, w[p + "k.norm"], eps).view(T, G, dim), pos, m.get("rot"))
    o = softmax_attention(q, k, raw.view(T, G, dim), float(m["scale"]), chunk_mask(T, size_of(m)))
    return o.reshape(T, H * dim) @ w[p + "o"].T


def clamped_unit(h, gate, up, down, limit):
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ down.T


def router_weights(h, w, p, top, gaps_out=None):
    """[T, experts]: the chosen experts' weights, 0 elsewhere. `gaps_out` (a list) gets [T]: how far the last chosen logit lies above
    the first that is not chosen."""
    z = h @ w[p + "router"].T + w[p + "router.b"]
    out = torch.zeros_like(z)
    gap = torch.full((z.shape[0],), float("inf"), dtype=z.dtype)
    for t in range(z.shape[0]):
        order = sorted(range(z.shape[1]), key=lambda e: (-float(z[t, e]), e))
        chosen = order[:top]
        out[t, chosen] = torch.softmax(z[t, chosen], dim=0)
        if top < z.shape[1]:
            gap[t] = z[t, order[top - 1]] - z[t, order[top]]
    if gaps_out is not None:
        gaps_out.append(gap)
    return out


def mixture(h, w, p, f, gaps_out=None):
    weights = router_weights(h, w, p, int(f["router"]["top"]), gaps_out)
    y = torch.zeros_like(h)
    for e in range(int(f["router"]["experts"])):
        names = [w[f"{p}e{e}.{n}"] for n in ("gate", "up", "down")]
        y += weights[:, e:e + 1] * clamped_unit(h, *names, float(f["expert"]["limit"]))
    if f.get("shared") is not None:
        names = [w[f"{p}shared.{n}"] for n in ("gate", "up", "down")]
        y += torch.sigmoid(h @ w[p + "shared.sg"].T) * clamped_unit(h, *names, float(f["shared"]["limit"]))
    return y


def read_streams(streams, weights):
    """streams [S, T, width], weights [S] -> sum_s weights[s] streams[s]."""
    return sum(weights[s] * streams[s] for s in range(streams.shape[0]))


def mix_streams(streams, y, mix, out):
    """All streams anew from the old ones: X_t <- sum_s mix[s, t] X_s + out[t] y."""
    S = streams.shape[0]
    return torch.stack([sum(mix[s, t] * streams[s] for s in range(S)) + out[t] * y for t in range(S)])


def layer_runs(cfg):
    """The layers in the order they run: start .. stop - 1 `times` times in a row."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if loop is None:
        return list(range(n))
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))


# ---- the model ------------------------------------------------------------------------------------------------------

def forward(cfg, w, tokens, layers_out=None, gaps_out=None):
    """Logits [T, vocab] of one whole sequence; `layers_out` (a list) gets the sum of the streams after every layer run, `gaps_out`
    (a list) one tensor [T] per routed feed-forward: how close the router's call was."""
    x = w["embed"][torch.tensor(tokens)]
    eps = float(cfg["norm"]["eps"])
    streams = torch.stack([x] * int(cfg["streams"]))
    for i in layer_runs(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        m = layer["mixer"]
        h = norm(read_streams(streams, w[p + "hc1.in"]), w[p + "norm1"], eps)
        if layer["type"] == "attention":
            y = capped_attention(h, w, p + "mix.", m)
        elif layer["type"] == "latent_attention":
            y = latent_attention(h, w, p + "mix.", m, eps)
        elif layer["type"] == "attention_2":
            y = keys_as_values_attention(h, w, p + "mix.", m, eps)
        else:
            raise ValueError(layer["type"])
        streams = mix_streams(streams, y, w[p + "hc1.mix"], w[p + "hc1.out"])
        if layer.get("mlp") is not None:
            h = norm(read_streams(streams, w[p + "hc2.in"]), w[p + "norm2"], eps)
            y = mixture(h, w, p + "mlp.", layer["mlp"], gaps_out)
            streams = mix_streams(streams, y, w[p + "hc2.mix"], w[p + "hc2.out"])
        if layers_out is not None:
            layers_out.append(streams.sum(dim=0))
    x = norm(streams.sum(dim=0), w["final.norm"], eps)
    return capped(x @ w["embed"].T, cfg.get("logit_softcap"))


def greedy_generate(cfg, w, prompt, n):
    """`n` tokens chosen greedily (the lowest index wins a tie), the whole sequence run anew for every token."""
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(forward(cfg, w, tokens)[-1].argmax()))
    return tokens[len(prompt):]
