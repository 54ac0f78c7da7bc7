"""A generalized delta rule as a mixer: a recurrent state per request and head whose transition decays and removes.

With h the normed rows, per head (dk key channels, dv value channels):

    r = Wr h,  k = Wk h,  v = Wv h
    d = exp(-rate sigmoid(W2 tanh(W1 h) + w0)),   a = sigmoid(Wa h + ba)         per key channel
    u = k / sqrt(sum(k^2) + 1e-6)
    S_t = diag(d_t) S_(t-1) - (a_t u_t) (u_t^T S_(t-1)) + k_t v_t^T,   o_t = S_t^T r_t
    x  += Wo ( rms(o_t) per head * n * sigmoid(Wg h) )                           n: a gain over all heads

One stacked input product (r, k, v, the gate, a's rows and W1) leaves in float32, so that everything that enters the recurrence
besides the projections (decays, removal rates, unit keys) is 32-bit in both precisions; the low-rank decay projection's second
product leaves in float32 too. The state S [heads, dk, dv] is float32 and lives in the cache manager's state slots (zero when a
request is opened). Single rows run token by token (`ops.delta_recurrent`), prompt portions in chunks of 32 tokens
(`ops.delta_chunked`: within a chunk the removals are the solution of a triangular system that is linear in the state in front
of it); a step of both runs each on its own rows. The norm and gate behind the recurrence ride in its last launch (single rows:
for heads of up to 64 values, else in a launch of their own).
"""
from __future__ import annotations

import torch

from ..cache.manager import FixedState
from ..csrc import ops
from ..weights.loader import TensorWant
from .base import Mixer, register_mixer
from .linear import Linear


def _up8(n: int) -> int:
    return -(-n // 8) * 8


class GeneralDelta(Mixer):
    can_overwrite = True
    EXTRA_CHUNKS = 128         # prompt portions in one step that the chunk scratch has room for beyond its rows' own chunks

    def __init__(self, spec, dim: int, tensors: dict, prefix: str, runtime):
        self.spec, self.dim, self.rt = spec, dim, runtime
        self.overwrite = False
        parts = [tensors.pop(prefix + n) for n in ("r", "k", "v", "g", "a", "w1")]
        self.rank = parts[5].shape[0]
        self.offsets, rows, at = [], [], 0
        for w in parts:            # every piece starts at a multiple of 8 columns
            self.offsets.append(at)
            pad = _up8(w.shape[0]) - w.shape[0]
            rows.append(w)
            if pad:
                rows.append(torch.zeros((pad, dim), dtype=w.dtype, device=w.device))
            at += w.shape[0] + pad
        self.width = at
        self.inp = Linear(torch.cat(rows, dim=0).contiguous())
        del parts, rows
        self.decay = Linear(tensors.pop(prefix + "w2"), tensors.pop(prefix + "w0"))
        self.a_bias = tensors.pop(prefix + "a.b")
        self.gain = tensors.pop(prefix + "norm")
        self.out = Linear(tensors.pop(prefix + "o"))

    @classmethod
    def wants(cls, spec, dim: int, prefix: str) -> dict:
        H, dk, dv, rank = spec.heads, spec.key_dim, spec.value_dim, spec.decay_rank
        return {prefix + "r": TensorWant((H * dk, dim)), prefix + "k": TensorWant((H * dk, dim)),
                prefix + "v": TensorWant((H * dv, dim)), prefix + "g": TensorWant((H * dv, dim)),
                prefix + "a": TensorWant((H * dk, dim)), prefix + "a.b": TensorWant((H * dk,), "vector"),
                prefix + "w1": TensorWant((rank, dim)), prefix + "w2": TensorWant((H * dk, rank)),
                prefix + "w0": TensorWant((H * dk,), "vector"), prefix + "norm": TensorWant((H * dv,), "vector", init="gain"),
                prefix + "o": TensorWant((dim, H * dv))}

    @classmethod
    def cache_need(cls, spec):
        return FixedState((spec.heads, spec.key_dim, spec.value_dim), "float32")

    def decode_bucket_cap(self, rows: int) -> int:
        return 1                       # nothing here looks at the context's length

    def _chunks(self, proj, z, batch, state, o, segments: int, rows: int, gate, y) -> bool:
        """Rows [0, rows), segments [0, segments) in chunks, their norm and gate included; False where the sizes are not taken."""
        s = self.spec
        H, dk, dv = s.heads, s.key_dim, s.value_dim
        r_off, k_off, v_off, _, a_off, _ = self.offsets
        room = self.rt.max_rows // ops.DELTA_CHUNK + self.EXTRA_CHUNKS
        qp = self.rt.buffer("delta_chunk_queries", H * dk, torch.float32)[:rows]
        transition = self.rt.buffer("delta_chunk_transition", H * dk * dk, torch.float32, rows=room)
        added = self.rt.buffer("delta_chunk_added", H * dk * dv, torch.float32, rows=room)
        return ops.delta_chunked(proj[:rows], r_off, k_off, v_off, a_off, z[:rows], self.a_bias, s.decay_rate, state,
                                 batch.seg_start[:segments], batch.seg_len[:segments], batch.state_slots[:segments], o[:rows], H, dk,
                                 dv, batch.max_q_len, qp, transition, added, norm=(gate[:rows], self.gain, s.norm_eps, y[:rows]))

    def forward(self, xb, x, batch, cache) -> None:
        s, rows = self.spec, xb.shape[0]
        if not cache.writes or cache.state is None:
            raise ops.KernelError("a delta rule keeps its own state: a run cannot read another run's")
        H, dk, dv = s.heads, s.key_dim, s.value_dim
        r_off, k_off, v_off, g_off, a_off, w_off = self.offsets
        proj = self.rt.buffer("delta_proj", self.width, torch.float32)[:rows]
        self.inp.forward(xb, proj)
        t = self.rt.buffer("delta_decay_in", self.rank)[:rows]
        ops.delta_tanh(proj[:, w_off:w_off + self.rank], t)
        z = self.rt.buffer("delta_decay_logits", H * dk, torch.float32)[:rows]
        self.decay.forward(t, z)
        o = self.rt.buffer("delta_out", H * dv, torch.float32)[:rows]
        y = self.rt.buffer("delta_gated", H * dv)[:rows]
        gate = proj[:, g_off:g_off + H * dv]
        segments, done, done_rows = batch.seg_start.numel(), 0, 0         # segments (rows) that have run
        if not batch.decode_only:
            # prompt portions in chunks; the single rows beside them (the scheduler puts them last) token by token
            ms, mr = (batch.multi_segments, batch.multi_rows) if batch.multi_segments >= 0 else (segments, rows)
            if ms > 0 and self._chunks(proj, z, batch, cache.state, o, ms, mr, gate, y):
                done, done_rows = ms, mr
        if done < segments:
            args = (proj, r_off, k_off, v_off, a_off, z, self.a_bias, s.decay_rate, cache.state, batch.seg_start[done:],
                    batch.seg_len[done:], batch.state_slots[done:], o, H, dk, dv)
            if not ops.delta_recurrent(*args, norm=(gate, self.gain, s.norm_eps, y)):
                ops.delta_recurrent(*args)
                ops.gated_head_norm(o[done_rows:], gate[done_rows:], self.gain, s.norm_eps, 1.0, y[done_rows:], H, dv, "sigmoid",
                                    gain_per_column=True)
        self.out.forward(y, x, accumulate=not self.overwrite)


register_mixer("general_delta", GeneralDelta, replace=True)
