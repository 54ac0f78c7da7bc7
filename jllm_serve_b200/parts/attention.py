"""Grouped-query causal attention over the paged cache, with optional per-head q/k RMSNorm and RoPE.

Order of operations from the reference (src/main/java/org/robomiri/jllm/cpu/CpuBackend.java:
422-458,595-615): q, k, v projections (biases if configured); RMSNorm of every query and key
head with the shared gains `q_norm` / `k_norm`; rotation; keys and values into the cache;
attention of every row over its request's keys [first, position]; `x += att @ Wo^T`.
Query head h reads kv head h // (heads / kv_heads) (cpu/KvCache.java:82,527). q, k and v
are one stacked [Q + 2 KV, dim] matrix, as the reference's fused `matmul3`.

A run that reads another run's cache (`cache.writes == False`) projects queries only.

What a spec may ask for beyond that: value heads of another width than key heads (a cache row is as wide as the wider of
the two); rotation of interleaved pairs; q and k divided by their root mean square behind the rotation; a chunk mask (a row
sees the earlier rows of its own chunk of the sequence only); a sigmoid gate per head, read from the mixer's input by rows
that ride at the end of the stacked projection. These run through the general per-head kernel (`ops.head_prepare`) and
the gate kernel; the attention itself is `ops.attention` for every form.

Further: a window that keeps the sequence's first `keep_first` positions visible to every later row (they keep their true
positions; the cache never gives their pages back); a learned sink per query head, a number whose exponential joins the
softmax's denominator without a key or a value; a sigmoid gate of FULL width (one gate value per value of the concatenated
heads, `gate = "sigmoid"`), whose rows also ride at the end of the stacked projection; and `out_scale`, a factor on the
mixer's result that a mixer of mixers sets (applied together with the gate, in front of the output projection).

And the WIDE forms (`spec.wide`), whose rows another kernel prepares (`ops.map_prepare`): an RMS norm over all query (key) columns
of a row at once; a stored factor per query head on the scores (folded into the query gains, which multiply the same values, when
the part is built); and a differential attention of two maps per head over the same values. The two maps cost one pass and one
copy of the values: a cached key row holds [map 1, map 2], a query head becomes two rows [q1, 0] and [0, q2] of that width, so the
attention kernels see heads x 2 query heads over kv_heads plain heads; `ops.map_difference` then subtracts the second map's
result (times lambda, a number of the layer made from four stored vectors), norms the difference per head and scales it. Rows are
filled up with zeros to a width the tile kernels take where that costs little (`spec.row_dim`). With `own_kv` False there are no
key and value projections: the run reads what another run cached, under its own mask. The same preparation multiplies queries that
grow with their position (`temp_every`) and, with `keys_as_values`, caches the keys' raw columns as the values (one projection). A cap
on the scores (`softcap`) is the attention kernels' own, in every form.
"""
from __future__ import annotations

import torch

from ..cache.manager import PagedKeysValues
from ..csrc import ops
from ..weights.loader import TensorWant
from .base import Mixer, register_mixer
from .linear import Linear


def _up8(n: int) -> int:
    return -(-n // 8) * 8


class GqaAttention(Mixer):
    can_overwrite = True           # a block that norms the result before adding it asks for x = ... instead of x += ...
    takes_out_scale = True         # `out_scale` multiplies the result (applied in front of the output product)

    def __init__(self, spec, dim: int, tensors: dict, prefix: str, runtime, rope=None):
        self.spec, self.dim, self.rt, self.rope = spec, dim, runtime, rope
        self.overwrite, self.out_scale = False, 1.0
        # what the attention kernels are told about the keys a row sees: 0 all, w > 0 a window, -c < 0 chunks of c positions
        self.span = -spec.chunk if spec.chunk else spec.window
        self.keep_first = int(getattr(spec, "keep_first", 0))
        self.wide = spec.wide
        if rope is not None and rope.rotary_dim > spec.head_dim:
            raise ValueError(f"rotary_dim={rope.rotary_dim} exceeds head_dim={spec.head_dim}")
        if self.wide:
            self._build_wide(tensors, prefix)
            return
        H, Hkv, hd, vd, names = spec.heads, spec.kv_heads, spec.head_dim, spec.v_dim, spec.names
        self.q_width, self.k_width, self.v_width = H * hd, Hkv * hd, Hkv * vd
        self.gated = spec.gate in ("head_sigmoid", "sigmoid")
        self.gate_width = H if spec.gate == "head_sigmoid" else H * vd      # gate values per row
        # the classic form (one head width, pairs (i, i + half), nothing behind the rotation) runs on the fused kernels that
        # were built for it; everything else on the general per-head kernel
        self.classic = (vd == hd and not spec.unit_qk and (rope is None or rope.pairing == "half"))
        if self.classic and spec.gate == "sigmoid" and rope is not None and rope.rotary_dim != hd and hd in (64, 128, 256):
            # a rotation of part of such a head: the general kernel's register form is the faster one (2,048 rows of 16 + 8
            # heads of 128: 14 us against 70)
            self.classic = False
        w = [tensors.pop(prefix + n) for n in (names.q, names.k, names.v)]
        b = [tensors.pop(prefix + n) for n in (names.q_bias, names.k_bias, names.v_bias)] if spec.bias else None
        self.k_off, self.v_off = self.q_width, self.q_width + self.k_width
        self.width = self.q_width + self.k_width + self.v_width
        self.g_off = -1
        if self.gated:
            # the gate's rows ride at the end of the stacked product, from a multiple of 8 columns on
            self.g_off = _up8(self.width)
            g = tensors.pop(prefix + names.gate)
            pad = self.g_off - self.width
            if pad:
                w.append(torch.zeros((pad, dim), dtype=g.dtype, device=g.device))
            w.append(g)
            # (and the row's width stays a multiple of 8 values: the tile kernels read queries by 16-byte pieces)
            tail = _up8(self.gate_width) - self.gate_width
            if tail:
                w.append(torch.zeros((tail, dim), dtype=g.dtype, device=g.device))
            if b:
                b.append(torch.zeros((pad + self.gate_width + tail,), dtype=b[0].dtype, device=b[0].device))
            self.width = self.g_off + self.gate_width + tail
        self.qkv = Linear(torch.cat(w, dim=0).contiguous(), torch.cat(b).contiguous() if b else None)
        self._q_only = None          # the query rows alone, made when a run first reads another run's cache
        del w, b
        self.out = Linear(tensors.pop(prefix + names.o), tensors.pop(prefix + names.o_bias) if spec.out_bias else None)
        self.sink = tensors.pop(prefix + names.sink) if spec.sink else None
        self.q_gain = tensors.pop(prefix + names.q_norm) if spec.qk_norm else None
        self.k_gain = tensors.pop(prefix + names.k_norm) if spec.qk_norm else None

    def _build_wide(self, tensors: dict, prefix: str) -> None:
        s, names = self.spec, self.spec.names
        q_width, k_width, v_width = s.heads * s.maps * s.head_dim, s.kv_heads * s.maps * s.head_dim, s.kv_heads * s.v_dim
        w = [tensors.pop(prefix + names.q)]
        self.k_off, self.v_off, self.width = 0, 0, q_width
        if s.own_kv:
            rows, at = [], 0
            pieces = [(w[0], q_width), (tensors.pop(prefix + names.k), k_width)]
            if not s.keys_as_values:
                pieces.append((tensors.pop(prefix + names.v), v_width))
            for t, n in pieces:
                if at != _up8(at):       # every piece starts at a multiple of 8 columns
                    rows.append(torch.zeros((_up8(at) - at, self.dim), dtype=t.dtype, device=t.device))
                    at = _up8(at)
                rows.append(t)
                self.k_off, self.v_off = self.v_off, at
                at += n
            if s.keys_as_values:
                self.k_off = self.v_off
            w, self.width = rows, at
        self.qkv = Linear(torch.cat(w, dim=0).contiguous())
        del w
        W, vd = s.row_dim, s.v_dim
        out = tensors.pop(prefix + names.o)
        if s.maps == 1 and W != vd:
            # the attention's result keeps the rows' width; its tail (zeros) meets columns of zeros
            wide = torch.zeros((self.dim, s.heads, W), dtype=out.dtype, device=out.device)
            wide[:, :, :vd] = out.view(self.dim, s.heads, vd)
            out = wide.view(self.dim, s.heads * W).contiguous()
        self.out = Linear(out)
        self.q_gain = self.k_gain = None
        if s.qk_norm:
            self.q_gain = tensors.pop(prefix + names.q_norm).float()
            self.k_gain = tensors.pop(prefix + names.k_norm).float().contiguous() if s.own_kv else None
        if s.head_scale:
            factor = tensors.pop(prefix + names.head_scale).float().repeat_interleave(s.maps * s.head_dim)
            if self.q_gain is None:
                raise ValueError("a factor per head on the scores is built together with a norm over all heads")
            self.q_gain = self.q_gain * factor
        self.q_gain = self.q_gain.contiguous() if self.q_gain is not None else None
        self.lam = 0.0
        if s.maps == 2:
            q1, k1, q2, k2 = (tensors.pop(prefix + n).double() for n in names.lambdas)
            self.lam = float((torch.exp((q1 * k1).sum()) - torch.exp((q2 * k2).sum())).item()) + s.diff

    @classmethod
    def _wide_wants(cls, s, dim: int, prefix: str) -> dict:
        names = s.names
        q_width, k_width = s.heads * s.maps * s.head_dim, s.kv_heads * s.maps * s.head_dim
        out = {prefix + names.q: TensorWant((q_width, dim)), prefix + names.o: TensorWant((dim, s.heads * s.v_dim))}
        if s.own_kv:
            out[prefix + names.k] = TensorWant((k_width, dim))
            if not s.keys_as_values:
                out[prefix + names.v] = TensorWant((s.kv_heads * s.v_dim, dim))
        if s.qk_norm:
            out[prefix + names.q_norm] = TensorWant((q_width,), "vector", init="gain")
            if s.own_kv:
                out[prefix + names.k_norm] = TensorWant((k_width,), "vector", init="gain")
        if s.head_scale:
            out[prefix + names.head_scale] = TensorWant((s.heads,), "vector", init="gain")
        if s.maps == 2:
            out.update({prefix + n: TensorWant((s.head_dim,), "vector") for n in names.lambdas})
        return out

    @classmethod
    def wants(cls, spec, dim: int, prefix: str) -> dict:
        if spec.wide:
            return cls._wide_wants(spec, dim, prefix)
        H, Hkv, hd, vd, names = spec.heads, spec.kv_heads, spec.head_dim, spec.v_dim, spec.names
        out = {prefix + names.q: TensorWant((H * hd, dim)),
               prefix + names.k: TensorWant((Hkv * hd, dim)),
               prefix + names.v: TensorWant((Hkv * vd, dim)),
               prefix + names.o: TensorWant((dim, H * vd))}
        if spec.bias:
            out.update({prefix + names.q_bias: TensorWant((H * hd,), "vector"),
                        prefix + names.k_bias: TensorWant((Hkv * hd,), "vector"),
                        prefix + names.v_bias: TensorWant((Hkv * vd,), "vector")})
        if spec.out_bias:
            out[prefix + names.o_bias] = TensorWant((dim,), "vector")
        if spec.qk_norm:
            out[prefix + names.q_norm] = TensorWant((hd,), "vector", init="gain")
            out[prefix + names.k_norm] = TensorWant((hd,), "vector", init="gain")
        if spec.gate == "head_sigmoid":
            out[prefix + names.gate] = TensorWant((H, dim))
        elif spec.gate == "sigmoid":
            out[prefix + names.gate] = TensorWant((H * vd, dim))
        if getattr(spec, "sink", False):
            out[prefix + names.sink] = TensorWant((H,), "vector")
        return out

    @classmethod
    def cache_need(cls, spec):
        # a cache row holds a key in its first head_dim values and a value in its first value_dim; under a chunk mask the
        # pages of chunks that have passed are given back as under a window (the need's window is then -chunk)
        return PagedKeysValues(spec.kv_heads, spec.row_dim, -spec.chunk if spec.chunk else spec.window,
                               keep_first=int(getattr(spec, "keep_first", 0)))

    def _tiles_fit(self) -> bool:
        s = self.spec
        if self.wide:
            return ops.attention_decode_fits(self.rt.dtype, s.heads * s.maps, s.kv_heads, s.row_dim)
        return (s.v_dim == s.head_dim and ops.attention_decode_fits(self.rt.dtype, s.heads, s.kv_heads, s.head_dim)
                and ops.attention_tiles_take(self.keep_first, self.sink))

    def decode_bucket_cap(self, rows: int) -> int:
        s = self.spec
        if not self._tiles_fit():
            return 1                   # the plain attention's launches do not depend on the context
        scratch = self.rt.buffer("attention_scratch", 2 << 20, torch.float32, rows=1)[0]
        heads, width = (s.heads * s.maps, s.row_dim) if self.wide else (s.heads, s.head_dim)
        return ops.decode_bucket_cap(rows, s.kv_heads, heads, width, self.span, scratch)

    def _forward_wide(self, xb, x, batch, cache) -> None:
        s, rows, rope, W = self.spec, xb.shape[0], self.rope, self.spec.row_dim
        if cache.writes != s.own_kv:
            raise ops.KernelError("an attention without key and value projections reads another run's cache, one with them its own")
        qkv = self.rt.buffer("qkv", self.width)[:rows]
        self.qkv.forward(xb, qkv)
        heads = s.heads * s.maps
        q = self.rt.buffer("map_queries", heads * W)[:rows]
        ops.map_prepare(qkv, self.k_off, self.v_off, self.q_gain, self.k_gain, s.qk_norm_eps, rope.cos if rope else None,
                        rope.sin if rope else None, rope.rotary_dim if rope else 0, rope.pairing if rope else "half",
                        batch.positions, batch.slots[cache.group] if cache.writes else None, q, cache.keys, cache.values, s.heads,
                        s.kv_heads, s.maps, s.head_dim, s.v_dim, W, self.rt.page_size, write_kv=cache.writes,
                        temp_every=s.temp_every, temp_coef=s.temp_coef)
        att = self.rt.buffer("attention_out", heads * W)[:rows]
        scratch = self.rt.buffer("attention_scratch", 2 << 20, torch.float32, rows=1)[0]
        ops.attention(q, cache.keys, cache.values, att, batch, cache.group, heads, s.kv_heads, W, self.rt.page_size, self.span,
                      s.scale, scratch, keep_first=self.keep_first, softcap=s.softcap)
        if s.maps == 2:
            y = self.rt.buffer("map_difference", s.heads * s.v_dim)[:rows]
            ops.map_difference(att, W, self.lam, s.diff_norm_eps, 1.0 - s.diff, y, s.heads, s.v_dim)
            att = y
        self.out.forward(att, x, accumulate=not self.overwrite)

    def forward(self, xb, x, batch, cache) -> None:
        if self.wide:
            return self._forward_wide(xb, x, batch, cache)
        s, rows = self.spec, xb.shape[0]
        if cache.writes or not self.classic or self.gated:
            qkv = self.rt.buffer("qkv", self.width)[:rows]
            self.qkv.forward(xb, qkv)
        else:
            qkv = self.rt.buffer("q_only", self.q_width)[:rows]
            if self._q_only is None:
                self._q_only = self.qkv.rows(0, self.q_width)
            self._q_only.forward(xb, qkv)
        rope = self.rope
        att = self.rt.buffer("attention_out", s.heads * s.v_dim)[:rows]
        scratch = self.rt.buffer("attention_scratch", 2 << 20, torch.float32, rows=1)[0]
        if (self.classic and not self.gated and cache.writes and batch.decode_only and rope is not None
                and self.sink is None and not self.keep_first and self.out_scale == 1.0 and not s.softcap
                and ops.attention_decode_fits(qkv.dtype, s.heads, s.kv_heads, s.head_dim)
                and ops.attention_decode_fresh_fits(qkv.dtype, s.heads, s.kv_heads, s.head_dim, rope.rotary_dim)):
            # a step of single rows: the attention kernel norms and rotates its own rows and writes their keys and values
            # (where that pays: it says whether it ran)
            if ops.attention_decode_fresh(qkv, self.q_gain, self.k_gain, s.qk_norm_eps, rope.cos, rope.sin, cache.keys,
                                          cache.values, att, batch.row_seg, batch.positions,
                                          batch.block_tables[cache.group], rows, s.heads, s.kv_heads, s.head_dim,
                                          self.rt.page_size, self.span, s.scale, batch.kv_bucket, scratch):
                return self.out.forward(att, x, accumulate=not self.overwrite)
        slots = batch.slots[cache.group] if cache.writes else None
        if self.classic:
            ops.qk_norm_rope_store(qkv, self.q_gain, self.k_gain, s.qk_norm_eps,
                                   rope.cos if rope else None, rope.sin if rope else None,
                                   rope.rotary_dim if rope else 0, batch.positions, slots, cache.keys, cache.values,
                                   s.heads, s.kv_heads, s.head_dim, self.rt.page_size, write_kv=cache.writes)
        else:
            ops.head_prepare(qkv, 0, self.k_off, self.v_off, self.q_gain, self.k_gain, s.qk_norm_eps,
                             rope.cos if rope else None, rope.sin if rope else None, rope.rotary_dim if rope else 0,
                             rope.pairing if rope else "half", s.unit_qk, batch.positions, slots, cache.keys, cache.values,
                             s.heads, s.kv_heads, s.head_dim, s.v_dim, self.rt.page_size, write_kv=cache.writes)
        ops.attention(qkv, cache.keys, cache.values, att, batch, cache.group, s.heads, s.kv_heads, s.head_dim,
                      self.rt.page_size, self.span, s.scale, scratch, value_dim=s.v_dim, keep_first=self.keep_first,
                      sink=self.sink, softcap=s.softcap)
        if s.gate == "sigmoid":
            ops.sigmoid_gate(att, qkv[:, self.g_off:self.g_off + self.gate_width], self.out_scale)
        else:
            if self.gated:
                ops.head_gate(att, qkv[:, self.g_off:self.g_off + s.heads], s.heads, s.v_dim)
            if self.out_scale != 1.0:
                raise ops.KernelError("a factor on the attention's result is built together with the gate of full width")
        self.out.forward(att, x, accumulate=not self.overwrite)


register_mixer("gqa_attention", GqaAttention, replace=True)
