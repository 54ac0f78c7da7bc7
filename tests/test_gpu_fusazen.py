"""Fusazen on the GPU against the plain implementation: every mechanism alone, then whole models through the step function
under every way of cutting the same requests, then generation, the command line and the trace program."""
import functools
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from tests import traces
from tests.fusazen_cases import FUSAZEN, fusazen_folder, fusazen_folder_of, random_fusazen
from tests.helpers import ARGMAX_SHARE, RMS_TOL, TOL
from tests.plain import fusazen_plain as P
from tests.tiny import random_tokens

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
DEV = "cuda:0"


def ops():
    from jllm_serve_b200.csrc import ops as o
    o.require_device()
    return o


def close(got, want, dtype, what, loose=1.0):
    tol = (2e-5 if dtype == torch.float32 else 1.6e-2) * float(want.abs().max()) * loose
    assert torch.isfinite(got).all(), f"{what}: non-finite values"
    diff = float((got.double().cpu() - want.double()).abs().max())
    assert diff <= tol, f"{what}: largest difference {diff:.3e} exceeds {tol:.3e}"


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


class FakeBatch:
    """The tables of a step that the kernels read: segments of consecutive rows, each with a state slot."""

    def __init__(self, lens, slots):
        starts = [sum(lens[:i]) for i in range(len(lens))]
        self.seg_start, self.seg_len, self.state_slots = i32(starts), i32(lens), i32(slots)
        self.row_seg = i32([s for s, n in enumerate(lens) for _ in range(n)])
        self.decode_only = max(lens) == 1
        self.max_q_len = max(lens)
        self.rows = sum(lens)


# ---- the input convolution ------------------------------------------------------------------------------------------

@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
@pytest.mark.parametrize("dim", [56, 50, 1030, 2048])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_norm_and_convolution_over_portions_and_slots(dtype, dim, taps):
    """Three requests in slots 2, 0 and 3 (slot 1 is another's and stays as it is), cut into steps of portions, of single rows and
    of both; each row against the convolution over the whole sequence; the state at the end is the last taps - 1 normed rows."""
    o = ops()
    g = torch.Generator().manual_seed(taps * 100 + dim)
    lens, slots, eps = [40, 23, 9], [2, 0, 3], 1e-5
    xs = [torch.randn(n, dim, generator=g) * (1 + s) for s, n in enumerate(lens)]
    gain = torch.randn(dim, generator=g).to(dtype)
    conv = (torch.randn(dim, taps, generator=g) * 0.5).to(dtype)
    hs = [P.norm(x.double(), gain.double(), eps) for x in xs]
    want = [P.input_convolution(h, conv.double()) for h in hs]
    state = torch.zeros(4, max(taps - 1, 1), dim, device=DEV)
    state[1] = 7.0
    fed = [0, 0, 0]
    got = [[], [], []]
    for step in ([17, 1, 3], [1, 1, 1], [2, 13, 0], [1, 1, 0], [0, 5, 5], [19, 2, 0]):
        who = [i for i in range(3) if step[i]]
        batch = FakeBatch([step[i] for i in who], [slots[i] for i in who])
        x = torch.cat([xs[i][fed[i]:fed[i] + step[i]] for i in who]).to(DEV)
        out = torch.empty(batch.rows, dim, dtype=dtype, device=DEV)
        o.norm_conv(x, gain.to(DEV), eps, conv.to(DEV), state, batch, out)
        at = 0
        for i in who:
            got[i].append(out[at:at + step[i]].float().cpu())
            at += step[i]
            fed[i] += step[i]
    assert fed == lens
    for i in range(3):
        close(torch.cat(got[i]), want[i], dtype, f"request {i}")
        if taps > 1:
            close(state[slots[i]], hs[i][-(taps - 1):], torch.float32, f"state of request {i}")
    assert bool((state[1] == 7.0).all())


# ---- the delta rule ----------------------------------------------------------------------------------------------------

def delta_case(H, dk, dv, lens, seed, strong=False):
    """Per request: r, k, v, the decay's and the removal's raw values. `strong`: few directions of keys (so that a token removes
    what an earlier one wrote), rates near 1, decays from almost none to the strongest the design has."""
    g = torch.Generator().manual_seed(seed)
    reqs = []
    for n in lens:
        r, v = torch.randn(n, H, dk, generator=g), torch.randn(n, H, dv, generator=g)
        k = torch.randn(n, H, dk, generator=g)
        z, a = torch.randn(n, H, dk, generator=g) * 2, torch.randn(n, H, dk, generator=g)
        if strong:
            few = torch.randn(3, H, dk, generator=g)
            k = few[torch.randint(0, 3, (n,), generator=g)] + 0.05 * k
            a = a * 0.3 + 5.0
            z = torch.where(torch.rand(n, H, dk, generator=g) < 0.5, torch.full_like(z, 9.0), torch.full_like(z, -9.0))
        reqs.append((r, k, v, z, a))
    return reqs


RATE = math.exp(-0.5)


def delta_plain(req, a_bias):
    r, k, v, z, a = (t.double() for t in req)
    H, dk = k.shape[1:]
    d = torch.exp(-RATE * torch.sigmoid(z))
    return P.delta_recurrence(r, k, v, d, torch.sigmoid(a + a_bias.double().view(H, dk)))


def delta_rows(reqs, cuts):
    """The stacked product's rows of the given (request, from, to) portions: [r | k | pad | v | a | gate] and z."""
    rows, zs = [], []
    for i, lo, hi in cuts:
        r, k, v, z, a = (t[lo:hi].flatten(1) for t in reqs[i])
        n = hi - lo
        pad = torch.full((n, (-(r.shape[1] + k.shape[1])) % 8), 1e30)
        more = torch.full((n, (-v.shape[1]) % 8), 1e30)
        rows.append(torch.cat([r, k, pad, v, more, a], dim=1))
        zs.append(z)
    R = reqs[0][0].flatten(1).shape[1]
    V = reqs[0][2].flatten(1).shape[1]
    k_off, v_off = R, R + R + (-2 * R) % 8
    a_off = v_off + V + (-V) % 8
    proj = torch.cat(rows)
    tail = (-proj.shape[1]) % 8
    if tail:
        proj = torch.cat([proj, torch.full((proj.shape[0], tail), 1e30)], dim=1)
    return proj.to(DEV), torch.cat(zs).to(DEV).contiguous(), (0, k_off, v_off, a_off)


SIZES = [(3, 12, 12), (2, 64, 64), (1, 128, 128), (2, 50, 34), (1, 100, 100), (2, 32, 64), (1, 256, 48), (1, 300, 20), (1, 700, 16),
         (5, 8, 24)]


@pytest.mark.parametrize("strong", [False, True])
@pytest.mark.parametrize("H, dk, dv", SIZES)
def test_delta_rule_token_by_token_and_in_chunks(H, dk, dv, strong):
    """Portions that begin and end inside and at the edges of chunks of 32, single rows, two requests in slots 2 and 0: both forms
    against the float64 recurrence over the whole sequence, the states they leave behind included."""
    o = ops()
    lens, slots = [150, 71], [2, 0]
    reqs = delta_case(H, dk, dv, lens, H * 1000 + dk, strong)
    a_bias = torch.randn(H * dk, generator=torch.Generator().manual_seed(9)) * 0.5
    want = [delta_plain(r, a_bias) for r in reqs]
    finals = {}
    for form in ("tokens", "chunks"):
        state = torch.zeros(3, H, dk, dv, device=DEV)
        state[1] = 3.0
        fed, got = [0, 0], [[], []]
        for step in ([33, 2], [1, 1], [32, 31], [2, 0], [64, 5], [1, 32], [17, 0]):
            who = [i for i in (0, 1) if step[i]]
            cuts = [(i, fed[i], fed[i] + step[i]) for i in who]
            proj, z, (r_off, k_off, v_off, a_off) = delta_rows(reqs, cuts)
            b = FakeBatch([step[i] for i in who], [slots[i] for i in who])
            out = torch.full((b.rows, H * dv), float("nan"), device=DEV)
            args = (proj, r_off, k_off, v_off, a_off, z, a_bias.to(DEV), RATE, state, b.seg_start, b.seg_len, b.state_slots, out, H, dk, dv)
            done = False
            if form == "chunks":
                room = b.rows // 32 + len(who)
                done = o.delta_chunked(*args, b.max_q_len, torch.empty(b.rows, H * dk, device=DEV),
                                       torch.full((room, H * dk * dk), float("nan"), device=DEV),
                                       torch.full((room, H * dk * dv), float("nan"), device=DEV))
                assert done == (dk % 4 == 0 and dv % 4 == 0 and max(dk, dv) <= 128), (dk, dv, done)
            if not done:
                assert o.delta_recurrent(*args)
            at = 0
            for i in who:
                got[i].append(out[at:at + step[i]].cpu())
                at += step[i]
                fed[i] += step[i]
        assert fed == lens
        for i in (0, 1):
            close(torch.cat(got[i]), want[i].flatten(1), torch.float32, f"{form}, request {i}")
        assert bool((state[1] == 3.0).all())
        finals[form] = state
    close(finals["chunks"], finals["tokens"].double().cpu(), torch.float32, "the states of both forms")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, dk, dv", [(2, 64, 64), (3, 12, 12), (1, 128, 128), (4, 20, 32), (2, 8, 40)])
def test_delta_rule_with_the_norm_and_gate_in_its_last_launch(dtype, H, dk, dv):
    """The same rows with and without: rms per head, a gain over all heads, a sigmoid gate; the chunked form for portions, the
    token form for single rows (heads of up to 64 values)."""
    o = ops()
    reqs = delta_case(H, dk, dv, [77, 5], 3)
    a_bias = torch.zeros(H * dk)
    g = torch.Generator().manual_seed(4)
    wide = torch.randn(82, H * dv + 8, generator=g)
    gain = torch.randn(H * dv, generator=g).to(dtype)
    eps = 1e-5
    for single in (False, True):
        lens = [1, 1] if single else [77, 5]
        proj, z, (r_off, k_off, v_off, a_off) = delta_rows(reqs, [(0, 0, lens[0]), (1, 0, lens[1])])
        b = FakeBatch(lens, [0, 1])
        state = torch.zeros(2, H, dk, dv, device=DEV)
        out = torch.full((b.rows, H * dv), float("nan"), device=DEV)
        gate = wide[:b.rows].to(DEV)[:, 4:4 + H * dv]
        y = torch.full((b.rows, H * dv), float("nan"), dtype=dtype, device=DEV)
        args = (proj, r_off, k_off, v_off, a_off, z, a_bias.to(DEV), RATE, state, b.seg_start, b.seg_len, b.state_slots, out, H, dk, dv)
        norm = (gate, gain.to(DEV), eps, y)
        if single:
            ran = o.delta_recurrent(*args, norm=norm)
            assert ran == (max(dk, dv) <= 64)
        else:
            ran = o.delta_chunked(*args, 77, torch.empty(b.rows, H * dk, device=DEV), torch.empty(6, H * dk * dk, device=DEV),
                                  torch.empty(6, H * dk * dv, device=DEV), norm=norm)
            assert ran
        if not ran:
            continue
        plain = torch.cat([delta_plain([t[:n] for t in reqs[i]], a_bias) for i, n in enumerate(lens)])
        want = P.rms(plain, eps).flatten(1) * gain.double() * torch.sigmoid(gate.double().cpu())
        close(y, want, dtype, f"single={single}", loose=3.0)


def test_delta_rule_over_many_short_portions_in_one_step():
    """40 requests of 2 to 41 rows in one step: every segment's chunks have numbers of their own."""
    o = ops()
    H, dk, dv = 2, 16, 16
    lens = [2 + i for i in range(40)]
    reqs = delta_case(H, dk, dv, lens, 11)
    a_bias = torch.zeros(H * dk)
    proj, z, (r_off, k_off, v_off, a_off) = delta_rows(reqs, [(i, 0, n) for i, n in enumerate(lens)])
    b = FakeBatch(lens, list(range(39, -1, -1)))
    state = torch.zeros(40, H, dk, dv, device=DEV)
    out = torch.full((b.rows, H * dv), float("nan"), device=DEV)
    room = b.rows // 32 + 40
    scratch = (torch.empty(b.rows, H * dk, device=DEV), torch.full((room, H * dk * dk), float("nan"), device=DEV),
               torch.full((room, H * dk * dv), float("nan"), device=DEV))
    args = (proj, r_off, k_off, v_off, a_off, z, a_bias.to(DEV), RATE, state, b.seg_start, b.seg_len, b.state_slots, out, H, dk, dv, 41)
    assert o.delta_chunked(*args, *scratch)
    want = torch.cat([delta_plain(r, a_bias) for r in reqs]).flatten(1)
    close(out, want, torch.float32, "forty portions")
    assert not o.delta_chunked(*args, scratch[0], scratch[1][:room - 1], scratch[2][:room - 1])     # too little room: refused


def test_tanh_of_a_view():
    o = ops()
    for dtype in (torch.float32, torch.bfloat16):
        x = torch.randn(9, 40, generator=torch.Generator().manual_seed(1)) * 2
        out = torch.empty(9, 13, dtype=dtype, device=DEV)
        o.delta_tanh(x.to(DEV)[:, 5:18], out)
        close(out, torch.tanh(x[:, 5:18].double()), dtype, "tanh")


# ---- wide attention --------------------------------------------------------------------------------------------------

def rot_tables(dims, base, n):
    ang = torch.outer(torch.arange(n, dtype=torch.float64), torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)],
                                                                          dtype=torch.float64))
    return ang.cos().float().to(DEV), ang.sin().float().to(DEV)


class WideCase:
    """Requests of the given lengths whose stacked projections [q | k | v] are random; every position's keys and values go into
    a paged cache (pages in a shuffled order, NaN wherever nothing was written) through the kernel under test."""

    def __init__(self, dtype, heads, kv_heads, maps, dim, vdim, lens, rot=None, page=16, seed=0, normed=False, edit=None):
        from jllm_serve_b200.config.specs import GqaAttentionSpec
        self.o, self.dtype, self.H, self.G, self.maps, self.dim, self.vdim, self.page = ops(), dtype, heads, kv_heads, maps, dim, vdim, page
        spec = GqaAttentionSpec(heads=heads, kv_heads=kv_heads, head_dim=dim, value_dim=vdim, scale=1.0, maps=maps, head_scale=maps == 1,
                                qk_norm=maps == 1, qk_norm_over="all" if maps == 1 else "head")
        self.W, self.lens, self.rot = spec.row_dim, lens, rot
        g = torch.Generator().manual_seed(seed)
        self.q = [torch.randn(n, heads, maps, dim, generator=g) for n in lens]
        self.k = [torch.randn(n, kv_heads, maps, dim, generator=g) for n in lens]
        self.v = [torch.randn(n, kv_heads, vdim, generator=g) for n in lens]
        if edit is not None:
            edit(self)
        self.q, self.k, self.v = ([t.to(dtype).float() for t in ts] for ts in (self.q, self.k, self.v))
        self.q_gain = self.k_gain = None
        if normed:
            self.q_gain = torch.randn(heads * maps * dim, generator=g)
            self.k_gain = torch.randn(kv_heads * maps * dim, generator=g)
        self.eps = 1e-5
        per = [-(-n // page) for n in lens]
        order = torch.randperm(sum(per) + 2, generator=g).tolist()
        tables = torch.full((len(lens), max(per)), -1, dtype=torch.int32)
        at = 0
        for s, b in enumerate(per):
            tables[s, :b] = torch.tensor(order[at:at + b], dtype=torch.int32)
            at += b
        self.tables = tables
        self.kc = torch.full((sum(per) + 2, kv_heads, page, self.W), float("nan"), dtype=dtype, device=DEV)
        self.vc = torch.full_like(self.kc, float("nan"))

    def prepare(self, cuts, write=True):
        """The rows of the (request, from, to) portions: their queries, with their keys and values written (or left alone)."""
        qw, kw, vw = self.H * self.maps * self.dim, self.G * self.maps * self.dim, self.G * self.vdim
        k_off = -(-qw // 8) * 8
        v_off = k_off + -(-kw // 8) * 8
        rows = []
        for s, lo, hi in cuts:
            row = torch.full((hi - lo, v_off + vw), float("nan"))
            row[:, :qw], row[:, k_off:k_off + kw] = self.q[s][lo:hi].flatten(1), self.k[s][lo:hi].flatten(1)
            row[:, v_off:] = self.v[s][lo:hi].flatten(1)
            rows.append(row)
        src = torch.cat(rows).to(self.dtype).to(DEV)
        pos = [p for s, lo, hi in cuts for p in range(lo, hi)]
        slots = [int(self.tables[s, p // self.page]) * self.page + p % self.page for s, lo, hi in cuts for p in range(lo, hi)]
        cos = sin = None
        if self.rot:
            cos, sin = rot_tables(self.rot[0], self.rot[1], max(self.lens))
        q = torch.full((src.shape[0], self.H * self.maps * self.W), float("nan"), dtype=self.dtype, device=DEV)
        gains = [x.to(DEV) if x is not None else None for x in (self.q_gain, self.k_gain)]
        self.o.map_prepare(src, k_off, v_off, *gains, self.eps, cos, sin, self.rot[0] if self.rot else 0, "half", i32(pos),
                           i32(slots), q, self.kc, self.vc, self.H, self.G, self.maps, self.dim, self.vdim, self.W, self.page, write_kv=write)
        return q

    def attend(self, q, cuts, span, scale):
        class B:
            pass
        b = B()
        b.row_seg = i32([s for s, lo, hi in cuts for _ in range(lo, hi)])
        b.positions = i32([p for s, lo, hi in cuts for p in range(lo, hi)])
        order = [s for s, _, _ in cuts]
        b.block_tables = [self.tables.to(DEV)]
        lens = [hi - lo for _, lo, hi in cuts]
        b.rows, b.decode_only = sum(lens), max(lens) == 1
        # (the tables hold one row per segment of the step: the step's segments are the case's requests, in order)
        assert order == list(range(len(self.lens)))
        b.seg_start, b.seg_len = i32([sum(lens[:i]) for i in range(len(lens))]), i32(lens)
        b.seg_kv_len = i32([hi for _, _, hi in cuts])
        b.multi_segments, b.multi_rows, b.kv_bucket = -1, 0, max(1, max(self.lens) // 256)
        out = torch.full((b.rows, self.H * self.maps * self.W), float("nan"), dtype=self.dtype, device=DEV)
        scratch = torch.empty(1 << 21, device=DEV)
        self.o.attention(q, self.kc, self.vc, out, b, 0, self.H * self.maps, self.G, self.W, self.page, span, scale, scratch)
        return out

    def plain(self, s, lo, hi, chunk, scale, factors=None):
        """[rows, H, maps, vdim] in float64."""
        n = self.lens[s]
        q, k = self.q[s].double(), self.k[s].double()
        if self.q_gain is not None:
            q = P.norm(q.flatten(1), self.q_gain.double(), self.eps).view(q.shape)
            k = P.norm(k.flatten(1), self.k_gain.double(), self.eps).view(k.shape)
        pos, rot = torch.arange(n), {"dims": self.rot[0], "base": self.rot[1]} if self.rot else None
        seen = P.chunk_mask(n, {"size": chunk} if chunk else None)
        sc = torch.full((self.H,), scale, dtype=torch.float64)
        out = [P.softmax_attention(P.rotate_half(q[:, :, m], pos, rot), P.rotate_half(k[:, :, m], pos, rot), self.v[s].double(), sc, seen)
               for m in range(self.maps)]
        return torch.stack(out, dim=2)[lo:hi]


SHAPES = [  # heads, kv_heads, maps, dim, vdim, rotated
    (4, 2, 2, 64, 128, 32), (4, 2, 2, 64, 128, 64), (2, 1, 2, 32, 64, 8), (4, 2, 2, 12, 20, 8), (3, 1, 2, 50, 88, 24), (2, 2, 2, 10, 6, 6),
    (2, 1, 2, 160, 40, 160), (20, 1, 2, 16, 16, 0), (4, 1, 1, 128, 128, 0), (6, 2, 1, 24, 16, 0), (3, 3, 1, 5, 9, 0), (2, 1, 1, 256, 256, 0)]


@pytest.mark.parametrize("H, G, maps, dim, vdim, dims", SHAPES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_maps_side_by_side_through_every_attention_kernel(dtype, H, G, maps, dim, vdim, dims):
    """Whole prompts, portions and single rows of three requests under chunks of 50 and without a mask: both maps' results of
    every row against float64, whatever kernel takes the width; filled-up columns of queries and cached rows are zeros."""
    lens = [130, 61, 17]
    case = WideCase(dtype, H, G, maps, dim, vdim, lens, rot=(dims, 500.0) if dims else None, seed=dim + vdim, normed=maps == 1)
    scale = (1.0 if maps == 2 else 0.5) / dim ** 0.5
    whole = [(s, 0, n) for s, n in enumerate(lens)]
    q = case.prepare(whole)
    held = [int(p) for row in case.tables for p in row if p >= 0]
    flat = case.kc.permute(0, 2, 1, 3).reshape(-1, G, case.W)
    vflat = case.vc.permute(0, 2, 1, 3).reshape(-1, G, case.W)
    rows = [int(case.tables[s, p // 16]) * 16 + p % 16 for s, n in enumerate(lens) for p in range(n)]
    assert not flat[rows][:, :, maps * dim:].float().abs().any() and not vflat[rows][:, :, vdim:].float().abs().any()
    assert torch.isnan(flat).any() and len(held) == len(set(held))
    qv = q.view(-1, H, maps, case.W)
    for m in range(maps):
        keep = torch.ones(case.W, dtype=torch.bool)
        keep[m * dim:(m + 1) * dim] = False
        assert not qv[:, :, m][:, :, keep.to(DEV)].float().abs().any()
    for chunk in (50, 0):
        out = case.attend(q, whole, -chunk, scale).view(-1, H, maps, case.W)[..., :vdim]
        want = torch.cat([case.plain(s, 0, n, chunk, scale) for s, n in enumerate(lens)])
        close(out, want, dtype, f"whole, chunk {chunk}", loose=2.0 if dtype == torch.float32 else 1.0)
        for cuts in ([(0, 120, 130), (1, 40, 61), (2, 15, 17)], [(0, 129, 130), (1, 60, 61), (2, 16, 17)],
                     [(0, 99, 103), (1, 49, 50), (2, 0, 17)]):
            got = case.attend(case.prepare(cuts, write=False), cuts, -chunk, scale).view(-1, H, maps, case.W)[..., :vdim]
            want = torch.cat([case.plain(s, lo, hi, chunk, scale) for s, lo, hi in cuts])
            close(got, want, dtype, f"{cuts}, chunk {chunk}", loose=2.0 if dtype == torch.float32 else 1.0)


@pytest.mark.parametrize("H, G, maps, dim, vdim", [(2, 1, 2, 64, 128), (2, 1, 2, 12, 20), (2, 2, 1, 128, 128), (2, 1, 2, 32, 64)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("row, key, chunk", [(99, 96, 48), (99, 95, 48), (96, 95, 48), (95, 48, 48), (95, 47, 48), (111, 0, 0), (63, 32, 32),
                                             (64, 63, 64), (129, 128, 64), (129, 127, 64), (47, 16, 16), (31, 16, 16), (32, 16, 16)])
def test_a_single_key_that_stands_out_at_a_chunks_edge(dtype, row, key, chunk, H, G, maps, dim, vdim):
    """One query points at one key (of the second map, where there are two) far back, at a page's border, just inside or just
    outside the row's chunk: inside, the row's result is that key's value; outside, it is as if the key were not there. In a prompt
    and in a single row."""
    n = row + 1

    def edit(c):
        c.k[0][key, :, maps - 1] *= 8.0
        c.q[0][row, :, maps - 1] = c.k[0][key, :, maps - 1].repeat_interleave(H // G, dim=0) / 8.0 * 4.0

    case = WideCase(dtype, H, G, maps, dim, vdim, [n], seed=row + key, edit=edit)
    scale = 1.0 / dim ** 0.5
    q = case.prepare([(0, 0, n)])
    inside = chunk == 0 or key // chunk == row // chunk
    want = case.plain(0, row, n, chunk, scale)
    near = (want[0, :, maps - 1] - case.v[0][key].double().repeat_interleave(H // G, dim=0)).abs().max()
    assert (float(near) < 0.05) == inside
    for rows, cut in ((q, (0, 0, n)), (case.prepare([(0, row, n)], write=False), (0, row, n))):
        got = case.attend(rows, [cut], -chunk, scale).view(-1, H, maps, case.W)[-1:, ..., :vdim]
        close(got, want, dtype, f"row {row} key {key} chunk {chunk}", loose=2.0)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, width, vdim", [(4, 128, 128), (3, 48, 20), (2, 16, 6), (5, 64, 50)])
def test_difference_of_two_maps(dtype, H, width, vdim):
    o = ops()
    g = torch.Generator().manual_seed(vdim)
    att = torch.randn(11, H * 2 * width, generator=g).to(dtype)
    if width > vdim:
        att.view(11, H, 2, width)[..., vdim:] = float("nan")       # (never read)
    out = torch.full((11, H * vdim), float("nan"), dtype=dtype, device=DEV)
    o.map_difference(att.to(DEV), width, 0.37, 1e-5, 0.6, out, H, vdim)
    a = att.double().view(11, H, 2, width)[..., :vdim]
    close(out, (P.rms(a[:, :, 0] - 0.37 * a[:, :, 1], 1e-5) * 0.6).flatten(1), dtype, "difference")


# ---- products and the small kernels ----------------------------------------------------------------------------------

@pytest.mark.parametrize("rows, K, N", [(1, 64, 96), (8, 256, 512), (40, 512, 384), (64, 2048, 2048), (100, 1024, 1280), (150, 512, 768),
                                        (300, 512, 16384), (513, 1024, 8192), (5, 50, 21), (33, 56, 40), (200, 72, 44)])
@pytest.mark.parametrize("with_bias", [True, False])
def test_relu_squared_in_every_products_epilogue(rows, K, N, with_bias):
    from jllm_serve_b200.parts.linear import Linear
    ops()
    g = torch.Generator().manual_seed(rows + N)
    a = torch.randn(rows, K, generator=g)
    w = torch.randn(N, K, generator=g) / K ** 0.5
    bias = torch.randn(N, generator=g) if with_bias else None
    for dtype in (torch.bfloat16, torch.float32):
        if dtype == torch.float32 and rows * K * N > 2 ** 30:
            continue
        at, wt = a.to(dtype).to(DEV), w.to(dtype).to(DEV)
        bt = bias.to(dtype).to(DEV) if with_bias else None
        z = at.double() @ wt.double().T + (bt.double() if with_bias else 0.0)
        want = torch.relu(z).square().cpu()
        out = torch.full((rows, N), float("nan"), dtype=dtype, device=DEV)
        Linear(wt, bt).forward(at, out, relu2=True)
        close(out, want, dtype, f"{dtype} relu squared")
        if dtype == torch.bfloat16:            # float32 results (the other path through the epilogues), and the bias on a sum
            out = torch.full((rows, N), float("nan"), device=DEV)
            Linear(wt, bt).forward(at, out, relu2=True)
            close(out, want, torch.float32, "float32 result", loose=3.0)
            acc = torch.randn(rows, N, generator=g)
            out = acc.to(DEV)
            Linear(wt, bt).forward(at, out, accumulate=True)
            close(out, z.cpu() + acc.double(), torch.float32, "added", loose=3.0)


def test_embedding_rows_with_a_scale():
    o = ops()
    for dtype, dim in ((torch.float32, 24), (torch.bfloat16, 24), (torch.bfloat16, 50), (torch.float32, 7), (torch.bfloat16, 2048)):
        table = torch.randn(30, dim, generator=torch.Generator().manual_seed(dim)).to(dtype)
        out = torch.empty(5, dim, device=DEV)
        o.embed_rows(i32([3, 0, 29, 7, 7]), table.to(DEV), out, 1.7)
        close(out, table.double()[[3, 0, 29, 7, 7]] * 1.7, torch.float32, "embedding")
        o.embed_rows(i32([3, 0, 29, 7, 7]), table.to(DEV), out)
        assert torch.equal(out.cpu(), table.float()[[3, 0, 29, 7, 7]])


# ---- whole models through the step function ---------------------------------------------------------------------------

@functools.lru_cache(maxsize=None)
def plain_model(folder):
    return P.load_plain(folder)


@functools.lru_cache(maxsize=256)
def plain_rows(folder, tokens):
    """(logits, [T]: how near the row's delta heads are to turning their sign)."""
    turns = []
    logits = P.forward(*plain_model(folder), list(tokens), turns_out=turns)
    return logits, torch.stack(turns).min(dim=0).values if turns else torch.ones(len(tokens))


class Checker:
    """Rows against the plain implementation's float64 logits. float32: every row within the tolerance; bfloat16: nearly every row
    (a few in a hundred may lie up to four times beyond it: heads whose two maps nearly cancel), and the sums over all rows. A row
    at which a delta head is about to turn its sign (nearly always a sequence's first row, whose head results are sign(k . r)
    times a direction) only has to be finite; such rows are few, or the test fails."""

    NEAR_TURN = {"float32": 5e-4, "bfloat16": 2e-2}

    def __init__(self, folder, sequences, dtype, what, slack=1.0):
        self.folder = folder
        self.sequences, self.dtype, self.what, self.slack = sequences, dtype, what, slack
        self.plain, self.errors, self.flips, self.err2, self.ref2, self.scale, self.seen = {}, [], 0, 0.0, 0.0, 0.0, set()
        self.skipped = 0

    def row(self, rid, position, got):
        if rid not in self.plain:
            self.plain[rid] = plain_rows(self.folder, tuple(self.sequences[rid]))
        want = self.plain[rid][0][position]
        assert torch.isfinite(got).all(), f"{self.what}: non-finite logits for {rid} position {position}"
        self.seen.add((rid, position))
        if float(self.plain[rid][1][position]) < self.NEAR_TURN[self.dtype]:
            self.skipped += 1
            return
        d = got.double() - want
        self.errors.append((float(d.abs().max()), rid, position))
        self.err2 += float((d * d).sum())
        self.ref2 += float((want * want).sum())
        self.scale = max(self.scale, float(want.abs().max()))
        self.flips += int(got.argmax()) != int(want.argmax())

    def finish(self):
        for rid, toks in self.sequences.items():
            missing = [p for p in range(len(toks)) if (rid, p) not in self.seen]
            assert not missing, f"{self.what}: no logits for {rid} positions {missing[:5]}"
        assert self.skipped <= max(2, len(self.sequences), 3 * len(self.seen) // 100), f"{self.what}: {self.skipped} rows skipped"
        assert self.errors, f"{self.what}: no row to compare"
        tol = 2 * TOL[self.dtype] * self.scale * self.slack
        worst = max(self.errors)
        over = [e for e in self.errors if e[0] > tol]
        rms = (self.err2 / max(self.ref2, 1e-300)) ** 0.5
        print(f"{self.what} [{self.dtype}] rows {len(self.errors)} (+{self.skipped}): largest difference {worst[0]:.3e} at {worst[1:]} "
              f"({worst[0] / self.scale:.2e} of the largest |logit|), {len(over)} rows over, rms {rms:.2e}, flips {self.flips}")
        first = min(over, key=lambda e: (e[1], e[2])) if over else None
        allowed = 0 if self.dtype == "float32" else max(2, 3 * len(self.errors) // 100)
        assert len(over) <= allowed and worst[0] <= 4 * tol, \
            f"{self.what}: {len(over)} rows beyond {tol:.3e}, the first at {first}, the largest {worst}"
        assert rms <= 3 * self.slack * RMS_TOL[self.dtype]
        assert 1 - self.flips / len(self.errors) >= ARGMAX_SHARE[self.dtype] - 0.04 * self.slack


def run_trace(name, dtype, steps, sequences, what, **kw):
    from jllm_serve_b200.csrc import ops as o
    from jllm_serve_b200.engine import ModelRunner, Segment
    args = dict(dtype=dtype, page_size=16, max_tokens=traces.peak_tokens(steps, 16), max_batch_tokens=512, max_requests=4,
                ctx=1024, poison_freed_pages=True)
    slack = kw.pop("slack", 1.0)
    args.update(kw)
    folder = name if isinstance(name, Path) else fusazen_folder(name)
    runner = ModelRunner(folder, **args)
    checker = Checker(folder, sequences, dtype, f"{name if not isinstance(name, Path) else ''} {what}", slack)
    fed = {}
    for st in steps:
        segs = [Segment(e["id"], e["tokens"], fed.get(e["id"], 0), e["want"]) for e in st["entries"]]
        rows = runner.step(segs).float().cpu()
        r = 0
        for e in st["entries"]:
            base = fed.get(e["id"], 0)
            for w in e["want"]:
                checker.row(e["id"], base + w, rows[r])
                r += 1
            fed[e["id"]] = base + len(e["tokens"])
        for rid in st["end"]:
            runner.finish(rid)
            fed.pop(rid, None)
    runner.cache.check()
    o.check_kernel_errors()
    checker.finish()
    runner.close()


def sequences_for(name, lengths, seed=21):
    return {f"r{i}": random_tokens(n, FUSAZEN[name]["vocab"], seed + i) for i, n in enumerate(lengths)}


LENGTHS = (1, 2, 37, 150, 16, 333, 65, 129)
WAYS = {
    "whole": traces.whole,
    "prompt, then token by token": lambda r: traces.prompt_then_decode(r, tail=24),
    "portions down to two tokens": traces.changing_portions,
    "all requests side by side": lambda r: traces.all_together(dict(list(r.items())[:4]), tail=6),
    "mixed, slots and pages used again": lambda r: traces.mixed(r, max_live=4, portion=40, prefill_share=0.7),
    "as the scheduler forms them": lambda r: traces.scheduled(r, {k: max(1, len(t) - 9) for k, t in r.items()}, portions=(70, 33, 128, 40)),
}


@pytest.mark.parametrize("way", list(WAYS))
@pytest.mark.parametrize("name", ["A", "B", "C"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_every_cut_of_the_same_requests_gives_the_plain_logits(name, dtype, way):
    seqs = sequences_for(name, LENGTHS)
    steps = WAYS[way](seqs)
    used = {e["id"] for st in steps for e in st["entries"]}
    run_trace(name, dtype, steps, {r: t for r, t in seqs.items() if r in used}, way)


@pytest.mark.parametrize("way", ["prompt, then token by token", "portions down to two tokens", "mixed, slots and pages used again"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_model_whose_sizes_are_multiples_of_nothing(dtype, way):
    seqs = sequences_for("D", (3, 70, 1, 141, 18), seed=31)
    run_trace("D", dtype, WAYS[way](seqs), seqs, way)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_while_chunks_pass_and_pages_go_back(dtype):
    """300 tokens one by one with pages of 8: the chunks (7, 13, 20, 40; in B 70, 100, 128) pass over decoded tokens, the pages
    behind them go back to the pool, and the layer that is read under a larger mask keeps what its readers still see."""
    for name in ("A", "B"):
        seqs = sequences_for(name, (420,), seed=5)
        run_trace(name, dtype, traces.prompt_then_decode(seqs, tail=300), seqs, "300 tokens one by one", page_size=8)


def test_a_state_slot_and_pages_that_are_used_again_start_clean():
    """One state slot and few pages: every request gets the slot and the pages the one before it left."""
    seqs = sequences_for("A", (90, 3, 61, 1, 40), seed=8)
    run_trace("A", "float32", traces.whole(seqs), seqs, "one slot", max_requests=1, max_tokens=96)
    run_trace("A", "float32", traces.changing_portions(seqs, sizes=(2, 9, 2, 31)), seqs, "one slot, portions", max_requests=1,
              max_tokens=96)


def test_more_rows_than_a_batch_holds_run_as_several_batches():
    seqs = sequences_for("C", (300, 77), seed=12)
    run_trace("C", "float32", traces.all_together(seqs, tail=2), seqs, "a step in parts", max_batch_tokens=64)


def test_a_captured_decode_step_equals_a_launched_one():
    """Decode steps of one shape are replayed from a graph: the same rows as launch by launch, bit for bit."""
    from jllm_serve_b200.engine import ModelRunner, Segment
    seqs = sequences_for("B", (40, 9, 77), seed=14)
    rows = {}
    for graphs in (False, True):
        runner = ModelRunner(fusazen_folder("B"), dtype="bfloat16", page_size=16, max_tokens=512, max_batch_tokens=256, max_requests=4,
                             ctx=512, cuda_graphs=graphs)
        runner.step([Segment(r, t[:-8], 0, []) for r, t in seqs.items()])
        out = []
        for k in range(8):
            out.append(runner.step([Segment(r, t[len(t) - 8 + k:len(t) - 7 + k], len(t) - 8 + k, [0]) for r, t in seqs.items()]).float().cpu())
        rows[graphs] = torch.stack(out)
        runner.close()
    assert torch.equal(rows[False], rows[True])


@pytest.mark.parametrize("seed", [9301, 9302, 9303, 9304, 9305, 9306, 9307, 9308, 9309, 9310])
def test_a_random_configuration_mixed_and_decoded(seed):
    """Configurations drawn at random: sizes, layer orders, masks, borrowed keys and constants in combinations that the fixed test
    models do not hold; requests mixed in steps with slots and pages used again, and a tail decoded token by token."""
    import random
    cfg = random_fusazen(seed)
    folder = fusazen_folder_of(cfg, seed, q_gain=2.0)
    rng = random.Random(seed)
    lengths = [rng.randint(1, 30), rng.randint(40, 140), rng.randint(150, 300), rng.randint(2, 70), rng.randint(100, 200)]
    seqs = {f"r{i}": random_tokens(n, cfg["vocab"], seed + i) for i, n in enumerate(lengths)}
    shape = "; ".join(l["type"] for l in cfg["layers"])
    for dtype in ("float32", "bfloat16"):
        run_trace(folder, dtype, traces.mixed(seqs, max_live=4, portion=50, prefill_share=0.7), seqs, f"seed {seed} ({shape}) mixed", slack=2.0)
        run_trace(folder, dtype, traces.prompt_then_decode(seqs, tail=40), seqs, f"seed {seed} ({shape}) decoded tail", slack=2.0)


def test_a_run_without_keys_of_its_own_reads_only_anothers():
    """The schedule and the layer must agree: a layer with key projections cannot borrow, one without cannot run alone."""
    from jllm_serve_b200.csrc.ops import KernelError
    from jllm_serve_b200.engine import ModelRunner, Segment
    runs = [(i, None) for i in range(3)] + [(2, 2)]                  # layer 2 has keys of its own and is told to borrow
    runner = ModelRunner(config=FUSAZEN["A"], seed=1, schedule=runs, dtype="float32", max_tokens=64, max_batch_tokens=64, max_requests=1,
                         ctx=64)
    with pytest.raises(KernelError, match="reads another run's cache"):
        runner.step([Segment("a", [1, 2, 3], 0, [2])])
    runner.close()


# ---- generation and the trace program -----------------------------------------------------------------------------------

def engine_for(name, dtype, **kw):
    from jllm_serve_b200.engine import Engine
    args = dict(dtype=dtype, page_size=8, max_tokens_cached=1024, max_batch_tokens=64, chunk=32, min_chunk=4, max_running=4,
                ctx=256)
    args.update(kw)
    return Engine(fusazen_folder(name), **args)


@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_float32_equals_plain(name):
    from jllm_serve_b200.sampling import SamplingParams
    cfg, w = P.load_plain(fusazen_folder(name))
    prompts = [random_tokens(n, FUSAZEN[name]["vocab"], 40 + n) for n in (5, 17, 41, 2, 33, 9)]
    got = engine_for(name, "float32").generate(prompts, SamplingParams.greedy_params(12, ignore_eos=True))
    for p, r in zip(prompts, got):
        assert r.tokens == P.greedy_generate(cfg, w, p, 12) and r.finish_reason == "length"


def test_greedy_generation_bfloat16_follows_plain():
    from jllm_serve_b200.sampling import SamplingParams
    cfg, w = P.load_plain(fusazen_folder("B"))
    prompts = [random_tokens(n, FUSAZEN["B"]["vocab"], 60 + n) for n in (9, 40, 70)]
    got = engine_for("B", "bfloat16").generate(prompts, SamplingParams.greedy_params(10, ignore_eos=True))
    for p, r in zip(prompts, got):
        logits = P.forward(cfg, w, p + r.tokens[:-1])
        for i, t in enumerate(r.tokens):
            row = logits[len(p) - 1 + i]
            assert float(row.max() - row[t]) <= 6 * TOL["bfloat16"] * float(logits.abs().max()), (i, t)


def test_generation_with_preemption_in_a_small_pool_equals_plain():
    from jllm_serve_b200.sampling import SamplingParams
    cfg, w = P.load_plain(fusazen_folder("A"))
    prompts = [random_tokens(n, FUSAZEN["A"]["vocab"], 80 + n) for n in (60, 1, 33, 64, 100, 20)]
    params = SamplingParams.greedy_params(16, ignore_eos=True)
    got = engine_for("A", "float32", max_tokens_cached=200, max_batch_tokens=48).generate(prompts, params)
    for i, (p, r) in enumerate(zip(prompts, got)):
        assert r.tokens == P.greedy_generate(cfg, w, p, 16), f"request {i}"


def test_command_line_run_and_bench_on_a_fusazen_model(tmp_path):
    folder = fusazen_folder("D")
    prompt = random_tokens(11, FUSAZEN["D"]["vocab"], 5)
    cmd = [sys.executable, str(ROOT / "bin" / "jllm"), "run", "--model", str(folder), "--dtype", "fp32", "--temp", "0",
           "--max-tokens", "7", "--ctx", "64", "--ignore-eos", "--tokens", ",".join(map(str, prompt))]
    proc = subprocess.run(cmd, capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    cfg, w = P.load_plain(folder)
    assert [int(t) for t in proc.stdout.strip().split(",")] == P.greedy_generate(cfg, w, prompt, 7)
    cfg_file = tmp_path / "config.json"
    cfg_file.write_text(json.dumps(FUSAZEN["B"]))
    proc = subprocess.run([sys.executable, str(ROOT / "bin" / "jllm"), "bench", "--random-weights", "3", "--model-config",
                           str(cfg_file), "--ctx", "256", "--bench.prompt-tokens", "50", "--bench.max-tokens", "8",
                           "--bench.rounds", "2"], capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert proc.stdout.startswith("prefill 50 tok in") and "decode 8 tok in" in proc.stdout


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_program_on_a_fusazen_folder(dtype, tmp_path):
    seqs = sequences_for("A", (50, 7, 1, 90, 33), seed=30)
    steps = traces.mixed(seqs, max_live=4, portion=24)
    text = "".join(json.dumps(s) + "\n" for s in steps)
    proc = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(fusazen_folder("A")), "--dtype", dtype,
                           "--out", str(tmp_path), "--max-tokens", str(traces.peak_tokens(steps)), "--poison"],
                          input=text, capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == [f"done {s['step']}" for s in steps]
    import numpy as np
    vocab = FUSAZEN["A"]["vocab"]
    checker = Checker(fusazen_folder("A"), seqs, dtype, "trace program")
    fed = {}
    for st in steps:
        rows = torch.from_numpy(np.fromfile(tmp_path / f"{st['step']}.f32", dtype="<f4").reshape(-1, vocab))
        r = 0
        for e in st["entries"]:
            base = fed.get(e["id"], 0)
            for w in e["want"]:
                checker.row(e["id"], base + w, rows[r])
                r += 1
            fed[e["id"]] = base + len(e["tokens"])
    checker.finish()
