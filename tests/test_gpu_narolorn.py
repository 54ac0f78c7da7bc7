"""Narolorn on the GPU against the plain implementation: every mechanism alone, then whole models through the step function under
every way of cutting the same requests, then generation, the command line and the trace program."""
import functools
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from tests import traces
from tests.helpers import ARGMAX_SHARE, RMS_TOL, TOL
from tests.narolorn_cases import NAROLORN, narolorn_folder, narolorn_folder_of, random_narolorn
from tests.plain import narolorn_plain as P
from tests.tiny import random_tokens

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]


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


# ---- the streams --------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dim", [56, 50, 1030, 2048, 4096, 8192, 8200])
@pytest.mark.parametrize("S", [1, 2, 3, 4, 5, 16])
@pytest.mark.parametrize("dtype", DTYPES)
def test_streams_opened_mixed_and_read(dtype, S, dim):
    """The three uses of the launch in a row: open and read; mix, store and read; mix and read picked rows (nothing stored); mix and
    store alone. Against the plain functions, streams and normed rows both."""
    o = ops()
    g = torch.Generator().manual_seed(S * 10000 + dim)
    rows, eps = 5, 1e-4
    x0, y = torch.randn(rows, dim, generator=g), torch.randn(rows, dim, generator=g) * 2
    mix, out = torch.randn(S, S, generator=g) * 0.6, torch.randn(S, generator=g)
    read, read2 = torch.randn(S, generator=g), torch.randn(S, generator=g)
    gain = torch.randn(dim, generator=g).to(dtype)
    X = torch.full((rows, S, dim), float("nan"), device=DEV)
    h = torch.full((rows, dim), float("nan"), dtype=dtype, device=DEV)
    both = torch.cat([mix.reshape(-1), out]).to(DEV)
    o.stream_mix(X, start=x0.to(DEV), read=read.to(DEV), gain=gain.to(DEV), eps=eps, out=h)
    plain = torch.stack([x0.double()] * S)
    assert torch.equal(X.cpu(), torch.stack([x0] * S, dim=1))
    close(h, P.norm(P.read_streams(plain, read.double()), gain.double(), eps), dtype, "opened")
    o.stream_mix(X, result=y.to(DEV), mix=both, read=read2.to(DEV), gain=gain.to(DEV), eps=eps, out=h)
    plain = P.mix_streams(plain, y.double(), mix.double(), out.double())
    close(X, plain.transpose(0, 1), torch.float32, "mixed")
    close(h, P.norm(P.read_streams(plain, read2.double()), gain.double(), eps), dtype, "mixed and read")
    before = X.clone()
    picked = i32([3, 0, 3])
    few = torch.full((3, dim), float("nan"), dtype=dtype, device=DEV)
    ones = torch.ones(S, device=DEV)
    o.stream_mix(X, result=y.to(DEV), mix=both, read=ones, gain=gain.to(DEV), eps=eps, out=few, row_index=picked, write=False)
    after = P.mix_streams(plain, y.double(), mix.double(), out.double())
    assert torch.equal(X, before)
    close(few, P.norm(after.sum(dim=0), gain.double(), eps)[[3, 0, 3]], dtype, "picked rows")
    o.stream_mix(X, result=y.to(DEV), mix=both)
    close(X, after.transpose(0, 1), torch.float32, "mixed alone", loose=2.0)


def test_a_rows_streams_do_not_depend_on_the_other_rows():
    o = ops()
    g = torch.Generator().manual_seed(5)
    X, y = torch.randn(9, 3, 128, generator=g).to(DEV), torch.randn(9, 128, generator=g).to(DEV)
    both, read, gain = torch.randn(12, generator=g).to(DEV), torch.randn(3, generator=g).to(DEV), torch.randn(128, generator=g).to(DEV)
    h = torch.empty(9, 128, device=DEV)
    one = X[4:5].clone()
    o.stream_mix(X, result=y, mix=both, read=read, gain=gain, eps=1e-6, out=h)
    h1 = torch.empty(1, 128, device=DEV)
    o.stream_mix(one, result=y[4:5].contiguous(), mix=both, read=read, gain=gain, eps=1e-6, out=h1)
    assert torch.equal(one[0], X[4]) and torch.equal(h1[0], h[4])


# ---- attention: caps, windows, chunks -------------------------------------------------------------------------------------

class Paged:
    """Requests of the given lengths with random queries, keys and values; keys and values in a paged cache (pages in a shuffled
    order, NaN wherever nothing was written)."""

    def __init__(self, dtype, heads, kv_heads, dim, lens, page=16, seed=0, spread=1.0, edit=None):
        self.o, self.dtype, self.H, self.G, self.dim, self.lens, self.page = ops(), dtype, heads, kv_heads, dim, lens, page
        g = torch.Generator().manual_seed(seed)
        self.q = [torch.randn(n, heads, dim, generator=g) * spread for n in lens]
        self.k = [torch.randn(n, kv_heads, dim, generator=g) for n in lens]
        self.v = [torch.randn(n, kv_heads, dim, generator=g) for n in lens]
        if edit is not None:
            edit(self)
        self.q, self.k, self.v = ([t.to(dtype).float() for t in ts] for ts in (self.q, self.k, self.v))
        per = [-(-n // page) for n in lens]
        order = torch.randperm(sum(per) + 2, generator=g).tolist()
        tables = torch.full((len(lens), max(per)), -1, dtype=torch.int32)
        at = 0
        for s, b in enumerate(per):
            tables[s, :b] = torch.tensor(order[at:at + b], dtype=torch.int32)
            at += b
        self.tables = tables
        kc = torch.full((sum(per) + 2, kv_heads, page, dim), float("nan"))
        vc = torch.full_like(kc, float("nan"))
        for s, n in enumerate(lens):
            for p in range(n):
                kc[tables[s, p // page], :, p % page], vc[tables[s, p // page], :, p % page] = self.k[s][p], self.v[s][p]
        self.kc, self.vc = kc.to(DEV, dtype), vc.to(DEV, dtype)

    def attend(self, cuts, span, scale, cap, scratch=True):
        class B:
            pass
        b = B()
        lens = [hi - lo for _, lo, hi in cuts]
        assert [s for s, _, _ in cuts] == list(range(len(self.lens)))
        b.row_seg = i32([s for s, lo, hi in cuts for _ in range(lo, hi)])
        b.positions = i32([p for s, lo, hi in cuts for p in range(lo, hi)])
        b.block_tables = [self.tables.to(DEV)]
        b.rows, b.decode_only = sum(lens), max(lens) == 1
        b.seg_start, b.seg_len = i32([sum(lens[:i]) for i in range(len(lens))]), i32(lens)
        b.seg_kv_len = i32([hi for _, _, hi in cuts])
        b.multi_segments, b.multi_rows, b.kv_bucket = -1, 0, max(1, max(self.lens) // 256)
        q = torch.cat([self.q[s][lo:hi] for s, lo, hi in cuts]).flatten(1).to(DEV, self.dtype).contiguous()
        out = torch.full((b.rows, self.H * self.dim), float("nan"), dtype=self.dtype, device=DEV)
        self.o.attention(q, self.kc, self.vc, out, b, 0, self.H, self.G, self.dim, self.page, span, scale,
                         torch.empty(1 << 21, device=DEV) if scratch else None, softcap=cap or 0.0)
        return out.view(-1, self.H, self.dim)

    def plain(self, s, lo, hi, span, scale, cap):
        n = self.lens[s]
        seen = P.window_mask(n, span) if span > 0 else P.chunk_mask(n, -span) if span < 0 else P.causal_mask(n)
        return P.softmax_attention(self.q[s].double(), self.k[s].double(), self.v[s].double(), scale, seen, cap)[lo:hi]


HEADS = [(4, 2, 64), (4, 2, 128), (3, 1, 256), (16, 1, 128), (4, 2, 48), (2, 1, 96), (20, 1, 64), (2, 2, 10)]


@pytest.mark.parametrize("cap, spread", [(5.0, 4.0), (20.0, 1.0), (0.5, 1.0), (50.0, 30.0)])
@pytest.mark.parametrize("H, G, dim", HEADS)
@pytest.mark.parametrize("dtype", DTYPES)
def test_capped_scores_through_every_attention_kernel(dtype, H, G, dim, cap, spread):
    """Whole prompts, portions and single rows of three requests; scores far inside the cap, around it and far beyond it (a spread of
    30: most of them sit at the cap itself), without a mask, under a window and under chunks."""
    case = Paged(dtype, H, G, dim, [140, 61, 18], seed=dim, spread=spread)
    scale = 1.0 / dim ** 0.5
    for span in (0, 37, -50):
        for cuts in ([(0, 0, 140), (1, 0, 61), (2, 0, 18)], [(0, 120, 140), (1, 40, 61), (2, 15, 18)], [(0, 139, 140), (1, 60, 61), (2, 17, 18)],
                     [(0, 138, 140), (1, 60, 61), (2, 16, 18)]):
            got = case.attend(cuts, span, scale, cap)
            want = torch.cat([case.plain(s, lo, hi, span, scale, cap) for s, lo, hi in cuts])
            close(got, want, dtype, f"{cuts} span {span}", loose=1.5)


@pytest.mark.parametrize("kernel", ["pair", "tc", "mma"])
def test_capped_scores_in_each_prompt_kernel(kernel):
    """Prompt tiles of which some warps' scores stay inside the cap and some do not (the polynomial and the exponential side by side)."""
    o = ops()
    n, H, G, dim, cap, scale = 700, 4, 2, 128, 8.0, 128 ** -0.5

    def edit(c):
        c.q[0][64:96] *= 12.0                   # (one warp of rows far beyond the cap)
        c.q[0][300] *= 12.0
    case = Paged(torch.bfloat16, H, G, dim, [n], seed=3, edit=edit)
    q = case.q[0].flatten(1).to(DEV, torch.bfloat16)
    for span in (0, -256, 200):
        out = torch.full((n, H * dim), float("nan"), dtype=torch.bfloat16, device=DEV)
        o.attention_prefill(q, case.kc, case.vc, out, i32([0]), i32([n]), i32([n]), case.tables.to(DEV), n, H, G, dim, 16, span, scale,
                            kernel=kernel, softcap=cap)
        close(out.view(n, H, dim), case.plain(0, 0, n, span, scale, cap), torch.bfloat16, f"{kernel} span {span}")
    o.check_kernel_errors()


@pytest.mark.parametrize("dim", [64, 128, 256])
def test_capped_scores_with_split_and_dealt_out_keys(dim):
    """Single rows whose keys are split over many blocks, and pairs dealt out evenly over fewer blocks than pairs."""
    o = ops()
    lens = [900, 333, 64, 1, 512]
    case = Paged(torch.bfloat16, 4, 2, dim, lens, seed=8, spread=3.0)
    scale, cap = 1.0 / dim ** 0.5, 4.0
    q = torch.stack([case.q[s][n - 1] for s, n in enumerate(lens)]).flatten(1).to(DEV, torch.bfloat16)
    args = (q, case.kc, case.vc)
    tail = (i32(list(range(5))), i32([n - 1 for n in lens]), case.tables.to(DEV), 5, 4, 2, dim, 16, 0, scale)
    want = torch.stack([case.plain(s, n - 1, n, 0, scale, cap)[0] for s, n in enumerate(lens)])
    scratch = torch.empty(1 << 21, device=DEV)
    for splits in (1, 3, 8, 17):
        out = torch.full((5, 4 * dim), float("nan"), dtype=torch.bfloat16, device=DEV)
        o.attention_decode_extras(*args, out, *tail, splits, scratch, softcap=cap)
        close(out.view(5, 4, dim), want, torch.bfloat16, f"{splits} splits")
    for blocks in (1, 7, 40):
        out = torch.full((5, 4 * dim), float("nan"), dtype=torch.bfloat16, device=DEV)
        o.attention_decode_flat(*args, out, *tail, blocks, scratch, softcap=cap)
        close(out.view(5, 4, dim), want, torch.bfloat16, f"dealt out over {blocks}")


@pytest.mark.parametrize("H, G, dim", [(2, 1, 128), (2, 1, 64), (3, 1, 96), (2, 2, 20)])
@pytest.mark.parametrize("row, key, span", [(99, 63, 37), (99, 62, 37), (100, 0, 101), (100, 0, 100), (64, 64, 1), (64, 63, 1), (64, 63, 2),
                                            (160, 145, 16), (160, 144, 16), (99, 96, -48), (99, 95, -48), (96, 95, -48), (95, 48, -48), (128, 127, -64),
                                            (127, 64, -64), (170, 0, 0), (170, 15, 0), (170, 16, 0)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_a_single_key_that_stands_out_at_an_edge(dtype, row, key, span, H, G, dim):
    """One query points at one key: at a page's border, far back, just inside or just outside the row's window or chunk, under a cap
    that still lets it stand out. Inside, the row's result is that key's value; outside, it is as if the key were not there. In a
    prompt, in a portion of two rows and in a single row."""
    def edit(c):
        c.k[0][key] *= 8.0
        c.q[0][row] = c.k[0][key].repeat_interleave(H // G, dim=0) / 8.0 * 6.0
    n = row + 1
    case = Paged(dtype, H, G, dim, [n], seed=row + key, edit=edit)
    scale, cap = 1.0 / dim ** 0.5, 25.0
    inside = span == 0 or (row - key < span if span > 0 else key // -span == row // -span)
    want = case.plain(0, row, n, span, scale, cap)
    near = (want[0] - case.v[0][key].double().repeat_interleave(H // G, dim=0)).abs().max()
    assert (float(near) < 0.05) == inside
    for lo in (0, row - 1, row):
        close(case.attend([(0, lo, n)], span, scale, cap)[-1:], want, dtype, f"rows from {lo}, span {span}", loose=2.0)


# ---- the rows of the attention ------------------------------------------------------------------------------------------------

def rot_tables(dims, base, n):
    ang = torch.outer(torch.arange(n, dtype=torch.float64), torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)],
                                                                          dtype=torch.float64))
    return ang.cos().float().to(DEV), ang.sin().float().to(DEV)


@pytest.mark.parametrize("H, G, dim, vdim, W", [(4, 2, 64, 64, 64), (4, 2, 128, 96, 128), (6, 2, 12, 20, 32), (3, 1, 10, 7, 16), (2, 2, 40, 48, 64)])
@pytest.mark.parametrize("every, coef", [(16, 0.5), (7, 0.3), (1, 1.0)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_queries_that_grow_with_their_position(dtype, every, coef, H, G, dim, vdim, W):
    o = ops()
    g = torch.Generator().manual_seed(dim)
    pos = [0, every - 2 if every > 1 else 3, every - 1, every, 2 * every - 1, 2 * every, 5 * every + 1, 1000]
    n, k_off = len(pos), -(-H * dim // 8) * 8
    v_off = k_off + -(-G * dim // 8) * 8
    src = torch.randn(n, v_off + G * vdim, generator=g).to(dtype)
    q = torch.full((n, H * W), float("nan"), dtype=dtype, device=DEV)
    kc, vc = (torch.full((2, G, 8, W), float("nan"), dtype=dtype, device=DEV) for _ in range(2))
    o.map_prepare(src.to(DEV), k_off, v_off, None, None, 1e-6, None, None, 0, "half", i32(pos), i32(list(range(n))), q, kc, vc, H, G, 1, dim,
                  vdim, W, 8, temp_every=every, temp_coef=coef)
    want = src[:, :H * dim].double().view(n, H, dim) * P.query_temperature(pos, {"coef": coef, "every": every})[:, None, None]
    close(q.view(n, H, W)[..., :dim], want, dtype, "queries")
    flat_k, flat_v = (c.permute(0, 2, 1, 3).reshape(-1, G, W)[:n] for c in (kc, vc))
    assert torch.equal(flat_k[..., :dim].cpu(), src[:, k_off:k_off + G * dim].view(n, G, dim))          # keys and values as they are
    assert torch.equal(flat_v[..., :vdim].cpu(), src[:, v_off:].view(n, G, vdim))
    assert not q.view(n, H, W)[..., dim:].float().abs().any() and not flat_k[..., dim:].float().abs().any() and not flat_v[..., vdim:].float().abs().any()


@pytest.mark.parametrize("H, G, dim, dims, W", [(4, 2, 64, 64, 64), (4, 2, 96, 32, 128), (5, 1, 24, 24, 32), (3, 1, 10, 6, 16), (2, 2, 40, 0, 48)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_values_that_are_the_keys_as_projected(dtype, H, G, dim, dims, W):
    """Norms over all columns, then rotation, for the cached key; the cached value is the projection itself, bit for bit."""
    o = ops()
    g = torch.Generator().manual_seed(dim + dims)
    n, eps, k_off = 12, 1e-4, -(-H * dim // 8) * 8
    src = torch.randn(n, k_off + G * dim, generator=g).to(dtype)
    qg, kg = torch.randn(H * dim, generator=g), torch.randn(G * dim, generator=g)
    cos, sin = rot_tables(dims, 50.0, n) if dims else (None, None)
    q = torch.full((n, H * W), float("nan"), dtype=dtype, device=DEV)
    kc, vc = (torch.full((2, G, 8, W), float("nan"), dtype=dtype, device=DEV) for _ in range(2))
    o.map_prepare(src.to(DEV), k_off, k_off, qg.to(DEV), kg.to(DEV), eps, cos, sin, dims, "half", i32(list(range(n))), i32(list(range(n))), q, kc,
                  vc, H, G, 1, dim, dim, W, 8)
    rot = {"dims": dims, "base": 50.0} if dims else None
    pos, raw = torch.arange(n), src[:, k_off:].double()
    close(q.view(n, H, W)[..., :dim], P.rotate_half(P.norm(src[:, :H * dim].double(), qg.double(), eps).view(n, H, dim), pos, rot), dtype, "queries")
    flat_k, flat_v = (c.permute(0, 2, 1, 3).reshape(-1, G, W)[:n] for c in (kc, vc))
    close(flat_k[..., :dim], P.rotate_half(P.norm(raw, kg.double(), eps).view(n, G, dim), pos, rot), dtype, "keys")
    assert torch.equal(flat_v[..., :dim].cpu(), src[:, k_off:].view(n, G, dim))


@pytest.mark.parametrize("rank, width", [(96, 128), (24, 24), (50, 64), (256, 256), (21, 21)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_rows_with_zeros_behind_them(dtype, rank, width):
    o = ops()
    g = torch.Generator().manual_seed(rank)
    src, gain = torch.randn(9, rank + 8, generator=g).to(dtype), torch.randn(rank, generator=g).to(dtype)
    cache = torch.full((4, 1, 4, width), float("nan"), dtype=dtype, device=DEV)
    slots = [3, 15, 0, 7, 8, 1, 2, 9, 4]
    o.latent_norm_store(src.to(DEV)[:, 8:], gain.to(DEV), 1e-4, i32(slots), cache)
    rows = cache.view(-1, width)
    close(rows[slots][:, :rank], P.norm(src[:, 8:].double(), gain.double(), 1e-4), dtype, "latent")
    assert not rows[slots][:, rank:].float().abs().any()
    assert torch.isnan(rows[[5, 6, 10, 11, 12, 13, 14]]).all()


@pytest.mark.parametrize("rows", [1, 8, 70])
@pytest.mark.parametrize("H, N, K", [(4, 128, 256), (3, 20, 24), (2, 7, 21), (5, 48, 96), (2, 1, 16)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_a_product_per_head_with_a_gate_per_value(dtype, H, N, K, rows):
    o = ops()
    g = torch.Generator().manual_seed(rows + N)
    a_head = K + 8
    a = torch.randn(rows, H * a_head, generator=g).to(dtype)
    w = (torch.randn(H, N, K, generator=g) / K ** 0.5).to(dtype)
    wide = torch.randn(rows, H * N + 8, generator=g).to(dtype) * 2
    out = torch.full((rows, H * N), float("nan"), dtype=dtype, device=DEV)
    o.gemm_heads(a.to(DEV), w.to(DEV), out, wide.to(DEV)[:, 8:], 1.5, a_head=a_head)
    want = torch.einsum("rhk,hnk->rhn", a.double().view(rows, H, a_head)[..., :K], w.double()).reshape(rows, -1)
    close(out, 1.5 * want * torch.sigmoid(wide[:, 8:].double()), dtype, "gated")


# ---- experts ----------------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("experts, top, gates", [(6, 2, 1), (5, 5, 1), (12, 3, 0), (3, 1, 1), (1, 1, 0)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_the_routers_bias_and_the_softmax_over_the_chosen(dtype, experts, top, gates):
    """A bias that turns most calls, chosen logits far apart (a softmax over ALL entries would hide nothing, one over the wrong ones
    would), logits so large that the exponentials of most entries vanish."""
    o = ops()
    for size in (1.0, 60.0):
        g = torch.Generator().manual_seed(experts * 10 + top)
        rows, dim = 40, 48
        h = torch.randn(rows, dim, generator=g).to(dtype)
        router = torch.randn(experts + gates, dim, generator=g) * 0.3 * size
        bias = (torch.randn(experts, generator=g) * 3 * size).to(dtype)
        table = torch.full((rows, experts + gates), float("nan"), device=DEV)
        o.route_experts(h.to(DEV), router.to(DEV), None, top, 1.0, True, table, gates=gates, softmax=True, bias=bias.to(DEV))
        w = {"router": router[:experts].double(), "router.b": bias.double()}
        gaps = []
        want = P.router_weights(h.double(), w, "", top, gaps)
        clear = gaps[0] > 1e-3 * size
        assert int(clear.sum()) >= rows - 4
        close(table[:, :experts].cpu()[clear], want[clear], torch.float32, "weights", loose=5.0 * size)
        if gates:
            close(table[:, experts], torch.sigmoid(h.double() @ router[experts].double()), torch.float32, "gate", loose=5.0)


def clamped_case(rows, K, E, ff, shared, seed, dtype, limits=(0.9, 1.6)):
    g = torch.Generator().manual_seed(seed)
    hidden = E * ff + shared
    x = torch.randn(rows, K, generator=g).to(dtype)
    gate, up = ((torch.randn(hidden, K, generator=g) * 2 / K ** 0.5).to(dtype) for _ in range(2))
    weights = torch.rand(rows, E + 1, generator=g) * (torch.rand(rows, E + 1, generator=g) < 0.6)
    limit = torch.cat([torch.full((E * ff,), limits[0]), torch.full((shared,), limits[1])]).double()
    a, b = x.double() @ gate.double().T, x.double() @ up.double().T
    a, b = torch.minimum(a, limit), torch.maximum(torch.minimum(b, limit), -limit)
    w = torch.cat([weights[:, :E].repeat_interleave(ff, dim=1), weights[:, E:].expand(-1, shared)], dim=1).double()
    return x, gate, up, weights, a * torch.sigmoid(1.702 * a) * (b + 1) * w


@pytest.mark.parametrize("rows, K, E, ff, shared", [(1, 64, 3, 16, 8), (8, 256, 5, 24, 40), (40, 512, 4, 96, 96), (64, 1024, 8, 128, 64), (100, 512, 3, 200, 104),
                                                    (150, 512, 4, 64, 32), (300, 256, 2, 40, 16), (513, 512, 4, 1024, 512), (700, 256, 7, 1024, 1024),
                                                    (33, 64, 2, 8, 0)])
def test_limits_and_weights_in_every_products_epilogue(rows, K, E, ff, shared):
    from jllm_serve_b200.parts.linear import Linear
    o = ops()
    x, gate, up, weights, want = clamped_case(rows, K, E, ff, shared, rows + ff, torch.bfloat16)
    hidden = E * ff + shared
    stacked = torch.stack([gate.view(hidden // 8, 8, K), up.view(hidden // 8, 8, K)], dim=1).reshape(2 * hidden, K).contiguous().to(DEV)
    words = [o.glu_descriptor("swish_clamped", l) for l in (0.9, 1.6)]
    table = weights.to(DEV) if shared else weights[:, :E].contiguous().to(DEV)
    lin = Linear(stacked)
    for weighted in (True, False):
        units = o.GluUnits(words[0], ff, E * ff if shared else 0, words[1], table if weighted else None)
        out = torch.full((rows, hidden), float("nan"), dtype=torch.bfloat16, device=DEV)
        lin.forward(x.to(DEV), out, swiglu=units)
        ref = want
        if not weighted:
            ref = clamped_case_unweighted(x, gate, up, E * ff, (0.9, 1.6))
        close(out, ref, torch.bfloat16, f"weighted={weighted}")
        if weighted:        # a unit whose weight is 0 gives exact zeros
            zero = torch.cat([weights[:, :E].repeat_interleave(ff, dim=1), weights[:, E:].expand(-1, shared)], dim=1) == 0
            assert not out.float().cpu()[zero].abs().any()
    a = x.to(DEV)
    for fn, fits in ((o.gemm_small_m, rows <= 64), (o.gemm_stream, rows <= 256), (o.gemm_tcgen05, True), (o.gemm_pair, rows > 128)):
        if not fits:
            continue
        out = torch.full((rows, hidden), float("nan"), dtype=torch.bfloat16, device=DEV)
        fn(a, lin.packed, out, swiglu=o.GluUnits(words[0], ff, E * ff if shared else 0, words[1], table))
        close(out, want, torch.bfloat16, fn.__name__)
    o.check_kernel_errors()


def clamped_case_unweighted(x, gate, up, routed, limits):
    limit = torch.full((gate.shape[0],), limits[1], dtype=torch.float64)
    limit[:routed] = limits[0]
    a, b = x.double() @ gate.double().T, x.double() @ up.double().T
    a, b = torch.minimum(a, limit), torch.maximum(torch.minimum(b, limit), -limit)
    return a * torch.sigmoid(1.702 * a) * (b + 1)


def test_units_that_do_not_come_in_eights_are_refused():
    from jllm_serve_b200.csrc.ops import KernelError
    o = ops()
    w = torch.zeros(2 * 24, 64, dtype=torch.bfloat16, device=DEV)
    x, out = torch.zeros(4, 64, dtype=torch.bfloat16, device=DEV), torch.zeros(4, 24, dtype=torch.bfloat16, device=DEV)
    table = torch.zeros(4, 2, device=DEV)
    with pytest.raises(KernelError, match="eights"):
        o.gemm_bf16(x, w, out, swiglu=o.GluUnits(o.glu_descriptor("swish_clamped", 1.0), 12, 12, 0, table))


@pytest.mark.parametrize("E, ff, shared", [(3, 16, 8), (5, 21, 13), (4, 40, 0), (1, 8, 24)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_the_clamped_unit_with_weights_on_its_results(dtype, E, ff, shared):
    o = ops()
    x, gate, up, weights, want = clamped_case(17, 32, E, ff, shared, ff, dtype)
    gate_up = torch.cat([x.double() @ gate.double().T, x.double() @ up.double().T], dim=1).to(dtype)
    out = torch.full((17, E * ff + shared), float("nan"), dtype=dtype, device=DEV)
    o.glu_clamped(gate_up.to(DEV), weights.to(DEV) if shared else weights[:, :E].contiguous().to(DEV), out, E, ff, 0.9, shared, 1.6, on_output=True)
    close(out, want, dtype, "units", loose=1.5)


def test_capped_values():
    o = ops()
    x = torch.randn(7, 301, generator=torch.Generator().manual_seed(2)) * 40
    got = x.to(DEV)
    o.softcap_values(got, 30.0)
    close(got, P.capped(x.double(), 30.0), torch.float32, "capped")


# ---- whole models through the step function -----------------------------------------------------------------------------------------

@functools.lru_cache(maxsize=None)
def plain_model(folder):
    return P.load_plain(folder)


@functools.lru_cache(maxsize=256)
def plain_rows(folder, tokens):
    """(logits, [T]: the closest call that a router had at a row or in front of it)."""
    gaps = []
    logits = P.forward(*plain_model(folder), list(tokens), gaps_out=gaps)
    margin = torch.stack(gaps).amin(dim=0) if gaps else torch.full((len(tokens),), float("inf"))
    return logits, margin


class Checker:
    """Rows against the plain implementation's float64 logits. float32: every row within the tolerance. bfloat16: rounding of a
    router's input may turn a close call between two experts, which changes that row outright (it only has to be finite) and, less,
    the rows that attend to it. So nine of ten other rows have to be within the tolerance, and the sums over the best nine tenths;
    where no router has a call to make (`strict`), all but three in a hundred, and the sums over all."""

    CLOSE_CALL = {"float32": 1e-4, "bfloat16": 0.12}

    def __init__(self, folder, sequences, dtype, what, slack=1.0):
        self.folder, self.sequences, self.dtype, self.what, self.slack = folder, sequences, dtype, what, slack
        self.plain, self.errors, self.squares, self.flips, self.ref2, self.scale, self.seen = {}, [], [], 0, 0.0, 0.0, set()
        self.skipped = 0

    def row(self, rid, position, got):
        if rid not in self.plain:
            self.plain[rid] = plain_rows(self.folder, tuple(self.sequences[rid]))
        want = self.plain[rid][0][position]
        assert torch.isfinite(got).all(), f"{self.what}: non-finite logits for {rid} position {position}"
        self.seen.add((rid, position))
        if float(self.plain[rid][1][position]) < self.CLOSE_CALL[self.dtype]:
            self.skipped += 1
            return
        d = got.double() - want
        self.errors.append((float(d.abs().max()), rid, position))
        self.squares.append(float((d * d).sum()))
        self.ref2 += float((want * want).sum())
        self.scale = max(self.scale, float(want.abs().max()))
        self.flips += int(got.argmax()) != int(want.argmax())

    def finish(self):
        for rid, toks in self.sequences.items():
            missing = [p for p in range(len(toks)) if (rid, p) not in self.seen]
            assert not missing, f"{self.what}: no logits for {rid} positions {missing[:5]}"
        assert self.errors, f"{self.what}: every row has a close call"
        assert self.dtype == "bfloat16" or self.skipped <= max(1, len(self.seen) // 100), f"{self.what}: {self.skipped} rows skipped"
        tol = (2 if self.dtype == "float32" else 3) * TOL[self.dtype] * self.scale * self.slack
        if self.dtype == "float32":
            tol *= 2                     # (row by row; the sums are held much closer)
        strict = self.dtype == "float32" or self.skipped == 0
        worst = max(self.errors)
        over = [e for e in self.errors if e[0] > tol]
        squares = sorted(self.squares)[:len(self.squares) if strict else -(-9 * len(self.squares) // 10)]
        rms = (sum(squares) / len(squares) / max(self.ref2 / len(self.squares), 1e-300)) ** 0.5
        print(f"{self.what} [{self.dtype}] rows {len(self.errors)} (+{self.skipped}): largest difference {worst[0]:.3e} at {worst[1:]} "
              f"({worst[0] / self.scale:.2e} of the largest |logit|), {len(over)} rows over, rms {rms:.2e}, flips {self.flips}")
        first = min(over, key=lambda e: (e[1], e[2])) if over else None
        allowed = 0 if self.dtype == "float32" else max(2, (3 if strict else 10) * len(self.errors) // 100)
        assert len(over) <= allowed, f"{self.what}: {len(over)} rows beyond {tol:.3e}, the first at {first}, the largest {worst}"
        assert rms <= (1 if self.dtype == "float32" else 2) * self.slack * RMS_TOL[self.dtype], f"{self.what}: rms {rms:.2e}"
        assert 1 - self.flips / len(self.errors) >= ARGMAX_SHARE[self.dtype] - 0.04 * self.slack, f"{self.what}: {self.flips} flips"


def run_trace(name, dtype, steps, sequences, what, **kw):
    from jllm_serve_b200.csrc import ops as o
    from jllm_serve_b200.engine import ModelRunner, Segment
    args = dict(dtype=dtype, page_size=16, max_tokens=traces.peak_tokens(steps, 16), max_batch_tokens=512, max_requests=4,
                ctx=1024, poison_freed_pages=True)
    slack = kw.pop("slack", 1.0)
    args.update(kw)
    folder = name if isinstance(name, Path) else narolorn_folder(name)
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
    return {f"r{i}": random_tokens(n, NAROLORN[name]["vocab"], seed + i) for i, n in enumerate(lengths)}


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
@pytest.mark.parametrize("name", ["A", "B", "C", "S"])
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
def test_long_decoding_while_windows_and_chunks_pass_and_pages_go_back(dtype):
    """300 tokens one by one with pages of 8: the windows and chunks pass over decoded tokens and the pages behind them go back to the
    pool, of every pass of the loop."""
    for name in ("A", "S"):
        seqs = sequences_for(name, (420,), seed=5)
        run_trace(name, dtype, traces.prompt_then_decode(seqs, tail=300), seqs, "300 tokens one by one", page_size=8)


def test_pages_that_are_used_again_start_clean():
    """One request at a time and few pages: every request gets the pages the one before it left."""
    seqs = sequences_for("A", (90, 3, 61, 1, 40), seed=8)
    run_trace("A", "float32", traces.whole(seqs), seqs, "one slot", max_requests=1, max_tokens=96)
    run_trace("A", "float32", traces.changing_portions(seqs, sizes=(2, 9, 2, 31)), seqs, "one slot, portions", max_requests=1,
              max_tokens=96)


def test_more_rows_than_a_batch_holds_run_as_several_batches():
    seqs = sequences_for("C", (300, 77), seed=12)
    run_trace("C", "float32", traces.all_together(seqs, tail=2), seqs, "a step in parts", max_batch_tokens=64)


def test_a_step_that_wants_nothing_and_then_one_that_does():
    """Portions without a wanted row leave the same cache behind (the last launch of the last layer is then left out)."""
    from jllm_serve_b200.engine import ModelRunner, Segment
    toks = random_tokens(60, NAROLORN["A"]["vocab"], 2)
    runner = ModelRunner(narolorn_folder("A"), dtype="float32", page_size=16, max_tokens=64, max_batch_tokens=64, max_requests=1, ctx=64)
    for lo, hi in ((0, 20), (20, 21), (21, 59)):
        assert runner.step([Segment("a", toks[lo:hi], lo, [])]).shape[0] == 0
    got = runner.step([Segment("a", toks[59:], 59, [0])]).float().cpu()
    close(got, P.forward(*plain_model(narolorn_folder("A")), toks)[59:], torch.float32, "last row")
    runner.close()


def test_a_captured_decode_step_equals_a_launched_one():
    """Decode steps of one shape are replayed from a graph: the same rows as launch by launch, bit for bit."""
    from jllm_serve_b200.engine import ModelRunner, Segment
    seqs = sequences_for("B", (40, 9, 77), seed=14)
    rows = {}
    for graphs in (False, True):
        runner = ModelRunner(narolorn_folder("B"), dtype="bfloat16", page_size=16, max_tokens=512, max_batch_tokens=256, max_requests=4,
                             ctx=512, cuda_graphs=graphs)
        assert runner.graph_safe
        runner.step([Segment(r, t[:-8], 0, []) for r, t in seqs.items()])
        out = []
        for k in range(8):
            out.append(runner.step([Segment(r, t[len(t) - 8 + k:len(t) - 7 + k], len(t) - 8 + k, [0]) for r, t in seqs.items()]).float().cpu())
        rows[graphs] = torch.stack(out)
        runner.close()
    assert torch.equal(rows[False], rows[True])


@pytest.mark.parametrize("seed", [9501, 9502, 9503, 9504, 9505, 9506, 9507, 9508, 9509, 9510])
def test_a_random_configuration_mixed_and_decoded(seed):
    """Configurations drawn at random: sizes, layer orders, loops, streams and constants in combinations that the fixed test models do
    not hold; requests mixed in steps with pages used again, and a tail decoded token by token."""
    import random
    cfg = random_narolorn(seed)
    folder = narolorn_folder_of(cfg, seed, q_gain=2.0)
    rng = random.Random(seed)
    lengths = [rng.randint(1, 30), rng.randint(40, 140), rng.randint(150, 300), rng.randint(2, 70), rng.randint(100, 200)]
    seqs = {f"r{i}": random_tokens(n, cfg["vocab"], seed + i) for i, n in enumerate(lengths)}
    shape = "; ".join(l["type"] for l in cfg["layers"])
    for dtype in ("float32", "bfloat16"):
        run_trace(folder, dtype, traces.mixed(seqs, max_live=4, portion=50, prefill_share=0.7), seqs, f"seed {seed} ({shape}) mixed", slack=2.0)
        run_trace(folder, dtype, traces.prompt_then_decode(seqs, tail=40), seqs, f"seed {seed} ({shape}) decoded tail", slack=2.0)


# ---- generation and the trace program ---------------------------------------------------------------------------------------------

def engine_for(name, dtype, **kw):
    from jllm_serve_b200.engine import Engine
    args = dict(dtype=dtype, page_size=8, max_tokens_cached=1024, max_batch_tokens=64, chunk=32, min_chunk=4, max_running=4,
                ctx=256)
    args.update(kw)
    return Engine(narolorn_folder(name), **args)


@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_float32_equals_plain(name):
    from jllm_serve_b200.sampling import SamplingParams
    cfg, w = P.load_plain(narolorn_folder(name))
    prompts = [random_tokens(n, NAROLORN[name]["vocab"], 40 + n) for n in (5, 17, 41, 2, 33, 9)]
    got = engine_for(name, "float32").generate(prompts, SamplingParams.greedy_params(12, ignore_eos=True))
    for p, r in zip(prompts, got):
        assert r.tokens == P.greedy_generate(cfg, w, p, 12) and r.finish_reason == "length"


def test_greedy_generation_bfloat16_follows_plain():
    from jllm_serve_b200.sampling import SamplingParams
    cfg, w = P.load_plain(narolorn_folder("S"))
    prompts = [random_tokens(n, NAROLORN["S"]["vocab"], 60 + n) for n in (9, 40, 70)]
    got = engine_for("S", "bfloat16").generate(prompts, SamplingParams.greedy_params(10, ignore_eos=True))
    for p, r in zip(prompts, got):
        logits = P.forward(cfg, w, p + r.tokens[:-1])
        for i, t in enumerate(r.tokens):
            row = logits[len(p) - 1 + i]
            assert float(row.max() - row[t]) <= 6 * TOL["bfloat16"] * float(logits.abs().max()), (i, t)


def test_generation_with_preemption_in_a_small_pool_equals_plain():
    from jllm_serve_b200.sampling import SamplingParams
    cfg, w = P.load_plain(narolorn_folder("A"))
    prompts = [random_tokens(n, NAROLORN["A"]["vocab"], 80 + n) for n in (60, 1, 33, 64, 100, 20)]
    params = SamplingParams.greedy_params(16, ignore_eos=True)
    got = engine_for("A", "float32", max_tokens_cached=200, max_batch_tokens=48).generate(prompts, params)
    for i, (p, r) in enumerate(zip(prompts, got)):
        assert r.tokens == P.greedy_generate(cfg, w, p, 16), f"request {i}"


def test_command_line_run_and_bench_on_a_narolorn_model(tmp_path):
    folder = narolorn_folder("D")
    prompt = random_tokens(11, NAROLORN["D"]["vocab"], 5)
    cmd = [sys.executable, str(ROOT / "bin" / "jllm"), "run", "--model", str(folder), "--dtype", "fp32", "--temp", "0",
           "--max-tokens", "7", "--ctx", "64", "--ignore-eos", "--tokens", ",".join(map(str, prompt))]
    proc = subprocess.run(cmd, capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    cfg, w = P.load_plain(folder)
    assert [int(t) for t in proc.stdout.strip().split(",")] == P.greedy_generate(cfg, w, prompt, 7)
    cfg_file = tmp_path / "config.json"
    cfg_file.write_text(json.dumps(NAROLORN["B"]))
    proc = subprocess.run([sys.executable, str(ROOT / "bin" / "jllm"), "bench", "--random-weights", "3", "--model-config",
                           str(cfg_file), "--ctx", "256", "--bench.prompt-tokens", "50", "--bench.max-tokens", "8",
                           "--bench.rounds", "2"], capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert proc.stdout.startswith("prefill 50 tok in") and "decode 8 tok in" in proc.stdout


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_program_on_a_narolorn_folder(dtype, tmp_path):
    seqs = sequences_for("A", (50, 7, 1, 90, 33), seed=30)
    steps = traces.mixed(seqs, max_live=4, portion=24)
    text = "".join(json.dumps(s) + "\n" for s in steps)
    proc = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(narolorn_folder("A")), "--dtype", dtype,
                           "--out", str(tmp_path), "--max-tokens", str(traces.peak_tokens(steps)), "--poison"],
                          input=text, capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == [f"done {s['step']}" for s in steps]
    import numpy as np
    vocab = NAROLORN["A"]["vocab"]
    checker = Checker(narolorn_folder("A"), seqs, dtype, "trace program")
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
