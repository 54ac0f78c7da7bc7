"""Plain, slow implementation of the Fusazen decoder: the oracle of its tests.

Fusazen is a small decoder-only design: a scaled embedding, a list of pre-norm layers, a final RMS norm and a head. What a
layer's mixer reads is its normed rows plus a short causal convolution over them. A mixer is a recurrence with a matrix state
per request whose transition is a diagonal decay minus a rank-one removal (`general_delta`), a differential attention (two
attention maps per head over the same values, the second subtracted with a learned factor; `attention`), possibly over the keys
and values that an earlier layer cached, or an attention with a norm over all heads of the queries (keys) together and a factor
per head on its scores (`attention_2`). Both attentions see the earlier positions of their own chunk of the sequence only. The
feed-forward is two matrices with biases around the square of relu.

Whole sequences, token by token where a mechanism is recurrent, one function per mechanism, tensors on the CPU in float64
unless the caller says otherwise. It shares no code with the product: it reads config.json and model.safetensors with its own
few lines and writes every sum as a loop or a plain torch expression.

Notation (h: the rows a part reads [T, width]; Wn: the tensor named n, stored [out, in]; p: position):
  rms(x)      = x / sqrt(mean(x^2) + eps);  norm(x, n) = rms(x) * n
  input conv  h_t <- h_t + sum_j c[:, j] h_(t - taps + 1 + j), zeros in front of the sequence
  delta       r, k, v = Wr h, Wk h, Wv h (heads x dim); d = exp(-exp(-1/2) sigmoid(Ww2 tanh(Ww1 h) + w0)); a = sigmoid(Wa h + ba);
              per head u = k / sqrt(sum(k^2) + 1e-6);  S_t = diag(d_t) S_(t-1) - outer(a_t u_t, S_(t-1)^T u_t) + outer(k_t, v_t);
              o_t = S_t^T r_t;  y = Wo (concat_heads(rms(o_t)) * n * sigmoid(Wg h))
  rotary      f_i = base^(-2i / dims), i < dims / 2; the pair (a, b) = values (i, i + dims / 2) at position p ->
              (a cos(p f_i) - b sin(p f_i), b cos(p f_i) + a sin(p f_i)); values from `dims` on do not rotate
  chunk mask  row t sees j <= t with j // size = t // size
  diff. att.  a head's q and k are two maps [q1, q2], [k1, k2] (each rotated); m_x = softmax(scale q_x . k_x) v;
              lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff;  o = rms(m_1 - lambda m_2) (1 - diff);  y = Wo concat_heads(o)
  attention_2 q <- norm(Wq h, nq), k <- norm(Wk h, nk) over ALL rows of the projection; scores scale temp_head q . k
  ff          y = Wdown relu(Wup h + bup)^2 + bdown
  layer       x += mixer(input conv(norm(x, n1)));  x += ff(norm(x, n2))
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


def input_convolution(h, conv):
    """h [T, width], conv [width, taps] -> h + the causal convolution of every channel over time."""
    taps = conv.shape[1]
    out = h.clone()
    for t in range(h.shape[0]):
        for j in range(taps):
            at = t - taps + 1 + j
            if at >= 0:
                out[t] += conv[:, j] * h[at]
    return out


def delta_recurrence(r, k, v, d, a, turns_out=None):
    """r, k, v, d, a [T, heads, dim] -> o [T, heads, dim]; the state starts at zero. `turns_out` (a list) gets one tensor [T]: the
    least |o| / (|S| |r|) of a token's heads. Near 0 the direction of o, all that the norm behind it keeps, hangs on the last bits
    of its inputs: a sequence's first token has S = k v^T and o = (k . r) v, whose SIGN is that of k . r."""
    near = torch.ones(k.shape[0], dtype=k.dtype)
    T, H, n = k.shape
    S = torch.zeros((H, n, v.shape[2]), dtype=k.dtype)
    o = torch.zeros_like(v)
    for t in range(T):
        u = k[t] / torch.sqrt((k[t] * k[t]).sum(dim=-1, keepdim=True) + 1e-6)
        read = torch.einsum("hi,hij->hj", u, S)
        S = d[t][:, :, None] * S - (a[t] * u)[:, :, None] * read[:, None, :] + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hij,hi->hj", S, r[t])
        near[t] = (o[t].norm(dim=-1) / (S.flatten(1).norm(dim=-1) * r[t].norm(dim=-1) + 1e-300)).min()
    if turns_out is not None:
        turns_out.append(near)
    return o


def general_delta(h, w, p, m, eps, turns_out=None):
    T, H, n = h.shape[0], int(m["heads"]), int(m["dim"])
    r, k, v = ((h @ w[p + x].T).view(T, H, n) for x in ("r", "k", "v"))
    decay = torch.sigmoid(torch.tanh(h @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])
    d = torch.exp(-math.exp(-0.5) * decay).view(T, H, n)
    a = torch.sigmoid(h @ w[p + "a"].T + w[p + "a.b"]).view(T, H, n)
    o = rms(delta_recurrence(r, k, v, d, a, turns_out), eps).reshape(T, H * n)
    return (o * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def rotate_half(x, positions, rot):
    """x [T, heads, dim]: the first rot.dims values of every head rotated by the position's angles, value i with i + dims / 2."""
    if rot is None:
        return x
    dims, base = int(rot["dims"]), float(rot["base"])
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    angle = (positions.to(torch.float64)[:, None] * f[None, :]).to(x.dtype)
    c, s = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def chunk_mask(T, mask):
    """[T, T] bool: which keys a row sees."""
    t = torch.arange(T)
    seen = t[None, :] <= t[:, None]
    if mask is not None:
        c = int(mask["size"])
        seen = seen & (t[None, :] // c == t[:, None] // c)
    return seen


def softmax_attention(q, k, v, scores_scale, seen):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim], scores_scale [H] -> [T, H, vdim]; query head h reads head h // (H / G)."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = torch.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T) * scores_scale[h]
        s = s.masked_fill(~seen, float("-inf"))
        out[:, h] = torch.softmax(s, dim=-1) @ v[:, h // per]
    return out


def differential_lambda(w, p, diff):
    return float(torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + diff)


def differential_keys_values(h, w, p, m):
    """What a layer caches: its two rotated key maps and its values."""
    T, G, dim, vdim = h.shape[0], int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(T)
    k = (h @ w[p + "k"].T).view(T, G, 2, dim)
    return [rotate_half(k[:, :, x], pos, m.get("rot")) for x in (0, 1)], (h @ w[p + "v"].T).view(T, G, vdim)


def differential_attention(h, w, p, m, eps, keys_values):
    T, H, dim, vdim = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    pos, seen = torch.arange(T), chunk_mask(T, m.get("mask"))
    (k1, k2), v = keys_values
    q = (h @ w[p + "q"].T).view(T, H, 2, dim)
    scale = torch.full((H,), float(m["scale"]), dtype=h.dtype)
    a1 = softmax_attention(rotate_half(q[:, :, 0], pos, m.get("rot")), k1, v, scale, seen)
    a2 = softmax_attention(rotate_half(q[:, :, 1], pos, m.get("rot")), k2, v, scale, seen)
    diff = float(m["diff"])
    o = rms(a1 - differential_lambda(w, p, diff) * a2, eps) * (1 - diff)
    return o.reshape(T, H * vdim) @ w[p + "o"].T


def whole_norm_attention(h, w, p, m, eps):
    T, H, G, dim, vdim = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = norm(h @ w[p + "q"].T, w[p + "q.norm"], eps).view(T, H, dim)
    k = norm(h @ w[p + "k"].T, w[p + "k.norm"], eps).view(T, G, dim)
    v = (h @ w[p + "v"].T).view(T, G, vdim)
    o = softmax_attention(q, k, v, float(m["scale"]) * w[p + "temp"], chunk_mask(T, m.get("mask")))
    return o.reshape(T, H * vdim) @ w[p + "o"].T


def feed_forward(h, w, p):
    z = torch.relu(h @ w[p + "up"].T + w[p + "up.b"])
    return (z * z) @ w[p + "down"].T + w[p + "down.b"]


# ---- the model ------------------------------------------------------------------------------------------------------

def forward(cfg, w, tokens, layers_out=None, turns_out=None):
    """Logits [T, vocab] of one whole sequence; `layers_out` (a list) gets the residual stream after every layer, `turns_out` (a
    list) one tensor [T] per delta layer: how near a head's result is to turning its sign (see `delta_recurrence`)."""
    x = w["embed"][torch.tensor(tokens)] * float(cfg.get("embedding", {}).get("scale", 1.0))
    eps = float(cfg["norm"]["eps"])
    kept = {}                                     # layer -> the keys and values it would cache
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = input_convolution(norm(x, w[p + "norm1"], eps), w[p + "canon1"])
        if layer["type"] == "general_delta":
            y = general_delta(h, w, p + "mix.", m, eps, turns_out)
        elif layer["type"] == "attention":
            if m.get("kv_from") is None:
                kept[i] = differential_keys_values(h, w, p + "mix.", m)
            y = differential_attention(h, w, p + "mix.", m, eps, kept[i if m.get("kv_from") is None else int(m["kv_from"])])
        elif layer["type"] == "attention_2":
            y = whole_norm_attention(h, w, p + "mix.", m, eps)
        else:
            raise ValueError(layer["type"])
        x = x + y
        if layer.get("mlp") is not None:
            x = x + feed_forward(norm(x, w[p + "norm2"], eps), w, p + "mlp.")
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm(x, w["final.norm"], eps) @ w["head"].T


def greedy_generate(cfg, w, prompt, n):
    """`n` tokens chosen greedily (the lowest index wins a tie), the whole sequence run anew for every token."""
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(forward(cfg, w, tokens)[-1].argmax()))
    return tokens[len(prompt):]
