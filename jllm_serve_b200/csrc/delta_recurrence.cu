// A recurrence whose transition is a decay per key channel minus a rank-one removal (a generalized delta rule).
//
// Per head, with dk key channels and dv value channels, a request carries a state S [dk, dv] in 32-bit floats:
//     u_t = k_t / sqrt(sum(k_t^2) + 1e-6),   d_t = exp(-rate sigmoid(z_t)),   a_t = sigmoid(a_raw_t + a_bias)
//     S_t = diag(d_t) S_(t-1) - (a_t u_t) (u_t^T S_(t-1)) + k_t v_t^T,        o_t = S_t^T r_t
// r, k, v, a_raw are float32 columns of the mixer's stacked input product; z is the low-rank decay projection's result
// (float32, its bias included). Everything here is float32 arithmetic on the CUDA cores, in both precisions of a model.
//
// Two forms that differ only in how sums are grouped:
//
//   delta_recurrent   token by token. A thread keeps R rows of one state column in registers; LS neighbouring lanes share a
//                     column, so the dot product u^T S and the output are a few shuffles and no block ever waits within a token.
//                     The form of decode steps, and of sizes the other one does not take. A token's arithmetic is the same
//                     wherever its portion begins.
//
//   delta_chunk_*     prompt portions in chunks of 32 tokens. With L_t the sum of log d over the chunk's tokens up to t (per
//                     channel) and p_t = S_(t-1)^T u_t (what a token removes), every token of a chunk that starts with S0 has
//                         p_t = (u_t e^(L_(t-1)))^T S0 + sum_(s<t) [(u_t e^(L_(t-1))) . (k_s e^(-L_s)) v_s
//                                                                   - (u_t e^(L_(t-1))) . (a_s u_s e^(-L_s)) p_s]
//                     which is a unit lower triangular system for the p of the chunk; its solution is linear in S0:
//                     p = W S0 + U. Then
//                         o_t = Q_t^T S0 + O_t,     Q_t = r_t e^(L_t) - sum_(s<=t) Arb[t,s] W_s,   O_t = sum_(s<=t) Ark[t,s] v_s - Arb[t,s] U_s
//                         S   = M S0 + N,           M = diag(e^L) (I - sum_s e^(-L_s) a_s u_s W_s^T),  N = diag(e^L) sum_s e^(-L_s) (k_s v_s^T - a_s u_s U_s^T)
//                     `prepare` makes Q, O, M and N of ALL chunks at once (nothing there depends on the state), `walk` goes
//                     through a portion's chunks with one dk x dk times dk x 16 product each and leaves the state in front of
//                     every chunk where N was, `out` adds Q^T S0 for all chunks at once. rate bounds the exponents: over 32
//                     tokens L lies in [-32 rate, 0], and the host refuses a rate whose e^(32 rate) would leave the range.
#include "common.cuh"

namespace {

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }

template <typename T>
__global__ void __launch_bounds__(256)
delta_tanh_kernel(const float* __restrict__ src, int ld, T* __restrict__ out, int rows, int width) {
    pdl_wait();
    pdl_trigger();
    const int total = rows * width;
    for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < total; i += gridDim.x * blockDim.x) {
        const int r = i / width, c = i - r * width;
        out[i] = from_float<T>(tanhf(src[(size_t)r * ld + c]));
    }
}

struct DeltaSource {
    const float* proj;       // [rows, ld]
    const float* z;          // [rows, heads * dk]
    VecRef a_bias;           // [heads * dk]
    float rate;
    int ld, r_off, k_off, v_off, a_off;
};

// The norm and gate behind the recurrence, y[r, h] = o[r, h] / sqrt(mean(o[r, h]^2) + eps) * gain * sigmoid(gate): taken along where
// a block holds all of a head's value columns (y null: the results leave as they are, in `o`).
struct DeltaNorm {
    const float* gate;       // [rows, ld]
    void* y;                 // [rows, heads * dv] of type `dtype`, or null
    VecRef gain;             // [heads * dv]
    float eps;
    int ld, dtype;
};

// one warp: the dv results of (row, head) in shared memory -> y
__device__ __forceinline__ void head_norm_row(const DeltaNorm& nm, const float* res, size_t row, int h, int heads, int dv) {
    const int lane = threadIdx.x & 31;
    float ss = 0.f;
    for (int i = lane; i < dv; i += 32) ss = fmaf(res[i], res[i], ss);
    ss = warp_sum(ss);
    const float inv = 1.f / sqrtf(ss / (float)dv + nm.eps);
    const float* g = nm.gate + row * nm.ld + (size_t)h * dv;
    const size_t at = row * ((size_t)heads * dv) + (size_t)h * dv;
    for (int i = lane; i < dv; i += 32) {
        const float v = __fmul_rn(__fmul_rn(__fmul_rn(res[i], inv), nm.gain[h * dv + i]), sigmoid_f(g[i]));
        if (nm.dtype == JLLM_F32) static_cast<float*>(nm.y)[at + i] = v;
        else static_cast<__nv_bfloat16*>(nm.y)[at + i] = __float2bfloat16_rn(v);
    }
}

// ---- token by token -----------------------------------------------------------------------------------------------------
template <int LS, int R, int CB, int TOK>
__global__ void __launch_bounds__(LS * CB)
delta_recurrent_kernel(DeltaSource src, float* __restrict__ state, int num_slots, const int* __restrict__ seg_start,
                       const int* __restrict__ seg_len, const int* __restrict__ state_slots, float* __restrict__ o, DeltaNorm nm,
                       int heads, int dk, int dv) {
    constexpr int DKP = LS * R, THREADS = LS * CB;
    extern __shared__ __align__(16) float smem[];
    float* ks = smem;                    // [TOK][DKP] k
    float* ds = ks + TOK * DKP;          //            d
    float* rs = ds + TOK * DKP;          //            r
    float* as = rs + TOK * DKP;          //            a k
    float* vs = as + TOK * DKP;          // [TOK][CB]
    float* inv2 = vs + TOK * CB;         // [TOK]      1 / (sum(k^2) + 1e-6)
    float* res = inv2 + TOK;             // [TOK][CB]  results on their way to the norm
    const int seg = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * CB;
    const int tid = threadIdx.x, l = tid % LS, c = tid / LS, j = c0 + c;
    const int first = seg_start[seg], n = seg_len[seg], slot = state_slots[seg];
    if (!jllm_in_bounds(slot, num_slots, BOUNDS_SLOT)) {
        pdl_wait();
        return;
    }
    float* S = state + (((size_t)slot * heads + h) * dk) * dv;
    float s[R];
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const int i = 4 * (l + LS * (r >> 2)) + (r & 3);
        s[r] = (i < dk && j < dv) ? S[(size_t)i * dv + j] : 0.f;
    }
    // The step's tables and a slot's state are older than the kernel in front of this one (nothing between a slot's opening or
    // its last step and this launch is so close), so the state is on its way before that kernel's results are waited for.
    pdl_wait();
    pdl_trigger();
    for (int t0 = 0; t0 < n; t0 += TOK) {
        const int nt = min(TOK, n - t0);
        for (int e = tid; e < nt * DKP; e += THREADS) {
            const int t = e / DKP, i = e - t * DKP;
            float k = 0.f, d = 1.f, r = 0.f, a = 0.f;
            if (i < dk) {
                const size_t row = (size_t)(first + t0 + t);
                const float* p = src.proj + row * src.ld + (size_t)h * dk + i;
                k = p[src.k_off];
                r = p[src.r_off];
                d = expf(-__fmul_rn(src.rate, sigmoid_f(src.z[row * ((size_t)heads * dk) + (size_t)h * dk + i])));
                a = __fmul_rn(sigmoid_f(__fadd_rn(p[src.a_off], src.a_bias[h * dk + i])), k);
            }
            ks[e] = k;
            ds[e] = d;
            rs[e] = r;
            as[e] = a;
        }
        for (int e = tid; e < nt * CB; e += THREADS) {
            const int t = e / CB, cc = e - t * CB;
            vs[e] = c0 + cc < dv ? src.proj[(size_t)(first + t0 + t) * src.ld + src.v_off + (size_t)h * dv + c0 + cc] : 0.f;
        }
        __syncthreads();
        for (int t = tid >> 5; t < nt; t += THREADS / 32) {
            float ss = 0.f;
            for (int i = tid & 31; i < DKP; i += 32) ss = fmaf(ks[t * DKP + i], ks[t * DKP + i], ss);
            ss = warp_sum(ss);
            if ((tid & 31) == 0) inv2[t] = 1.f / (ss + 1e-6f);
        }
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            const float4* k4 = reinterpret_cast<const float4*>(ks + t * DKP);
            const float4* d4 = reinterpret_cast<const float4*>(ds + t * DKP);
            const float4* r4 = reinterpret_cast<const float4*>(rs + t * DKP);
            const float4* a4 = reinterpret_cast<const float4*>(as + t * DKP);
            float dot0 = 0.f, dot1 = 0.f;
#pragma unroll
            for (int q = 0; q < R / 4; ++q) {
                const float4 kk = k4[l + LS * q];
                dot0 = fmaf(kk.x, s[4 * q], dot0);
                dot1 = fmaf(kk.y, s[4 * q + 1], dot1);
                dot0 = fmaf(kk.z, s[4 * q + 2], dot0);
                dot1 = fmaf(kk.w, s[4 * q + 3], dot1);
            }
            float dot = dot0 + dot1;
#pragma unroll
            for (int m = 1; m < LS; m <<= 1) dot += __shfl_xor_sync(0xffffffffu, dot, m);
            const float p = -__fmul_rn(dot, inv2[t]), v = vs[t * CB + c];     // u (u^T S) = k (k^T S) / (sum(k^2) + 1e-6)
            float acc0 = 0.f, acc1 = 0.f;
#pragma unroll
            for (int q = 0; q < R / 4; ++q) {
                const float4 kk = k4[l + LS * q], dd = d4[l + LS * q], rr = r4[l + LS * q], aa = a4[l + LS * q];
                s[4 * q] = fmaf(aa.x, p, fmaf(dd.x, s[4 * q], __fmul_rn(kk.x, v)));
                s[4 * q + 1] = fmaf(aa.y, p, fmaf(dd.y, s[4 * q + 1], __fmul_rn(kk.y, v)));
                s[4 * q + 2] = fmaf(aa.z, p, fmaf(dd.z, s[4 * q + 2], __fmul_rn(kk.z, v)));
                s[4 * q + 3] = fmaf(aa.w, p, fmaf(dd.w, s[4 * q + 3], __fmul_rn(kk.w, v)));
                acc0 = fmaf(s[4 * q], rr.x, acc0);
                acc1 = fmaf(s[4 * q + 1], rr.y, acc1);
                acc0 = fmaf(s[4 * q + 2], rr.z, acc0);
                acc1 = fmaf(s[4 * q + 3], rr.w, acc1);
            }
            float acc = acc0 + acc1;
#pragma unroll
            for (int m = 1; m < LS; m <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, m);
            if (l == 0 && j < dv) {
                if (nm.y != nullptr) res[t * CB + c] = acc;
                else o[(size_t)(first + t0 + t) * ((size_t)heads * dv) + (size_t)h * dv + j] = acc;
            }
        }
        __syncthreads();
        if (nm.y != nullptr)         // (`res` is written again behind two more barriers)
            for (int t = tid >> 5; t < nt; t += THREADS / 32) head_norm_row(nm, res + t * CB, (size_t)(first + t0 + t), h, heads, dv);
    }
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const int i = 4 * (l + LS * (r >> 2)) + (r & 3);
        if (i < dk && j < dv) S[(size_t)i * dv + j] = s[r];
    }
}

template <int LS, int R, int CB, int TOK>
int launch_recurrent(const DeltaSource& src, float* state, int num_slots, const int* seg_start, const int* seg_len,
                     const int* state_slots, float* o, const DeltaNorm& nm, int segments, int heads, int dk, int dv,
                     cudaStream_t stream) {
    const size_t smem = (size_t)(TOK * (4 * LS * R + 2 * CB) + TOK) * sizeof(float);
    auto kernel = delta_recurrent_kernel<LS, R, CB, TOK>;
    if (smem > 48 * 1024 &&
        cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
        return jllm_fail(JLLM_CUDA_ERROR, "delta_recurrent: %zu bytes of shared memory refused", smem);
    jllm_launch(kernel, dim3(segments, heads, (dv + CB - 1) / CB), dim3(LS * CB), smem, stream, LAUNCH_DEPENDENT, src, state,
                num_slots, seg_start, seg_len, state_slots, o, nm, heads, dk, dv);
    return jllm_check_launch("delta_recurrent");
}

// ---- prompt portions in chunks --------------------------------------------------------------------------------------------
constexpr int C = 32;            // tokens of a chunk
constexpr int LDS = C + 4;       // row length of the score matrices

// chunk number of a segment's first chunk among all: a segment's chunks are numbered from here on and never meet the next one's
// (ceil(n / C) <= n / C + 1, and the whole parts of a sum are at least the sum of the whole parts)
__device__ __forceinline__ int chunk_base(int first, int seg) { return first / C + seg; }

__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void fma4(float (&acc)[4], float a, const float4& b) {
    acc[0] = fmaf(a, b.x, acc[0]);
    acc[1] = fmaf(a, b.y, acc[1]);
    acc[2] = fmaf(a, b.z, acc[2]);
    acc[3] = fmaf(a, b.w, acc[3]);
}

// acc[a][0..3] += sign * sum_s A[t(a)][s] B[s][i0 .. i0 + 3], t(a) = ty + 8 a: a 4 x 4 tile of a C x C times C x width product
template <int SIGN>
__device__ __forceinline__ void tile_rows(float (&acc)[4][4], const float* A, const float* B, int ldb, int ty, int i0) {
#pragma unroll 2
    for (int s = 0; s < C; s += 4) {
        float4 av[4];
#pragma unroll
        for (int a = 0; a < 4; ++a) av[a] = ld4(A + (ty + 8 * a) * LDS + s);
        const float4 b0 = ld4(B + (s + 0) * ldb + i0), b1 = ld4(B + (s + 1) * ldb + i0), b2 = ld4(B + (s + 2) * ldb + i0),
                     b3 = ld4(B + (s + 3) * ldb + i0);
#pragma unroll
        for (int a = 0; a < 4; ++a) {
            fma4(acc[a], SIGN * av[a].x, b0);
            fma4(acc[a], SIGN * av[a].y, b1);
            fma4(acc[a], SIGN * av[a].z, b2);
            fma4(acc[a], SIGN * av[a].w, b3);
        }
    }
}

// D: the key and value width where both are that, known to the compiler; 0: read from the arguments
constexpr int PREP_THREADS = 256;
template <int D>
__global__ void __launch_bounds__(PREP_THREADS, D == 64 ? 3 : 1)
delta_chunk_prepare_kernel(DeltaSource src, const int* __restrict__ seg_start, const int* __restrict__ seg_len,
                           float* __restrict__ qp, float* __restrict__ o, float* __restrict__ M, float* __restrict__ N, int heads,
                           int dk_arg, int dv_arg) {
    const int dk = D ? D : dk_arg, dv = D ? D : dv_arg;
    extern __shared__ __align__(16) float smem[];
    const int ldk = dk + 4, ldv = dv + 4;
    float* Bm = smem;                    // [C][ldk]  u_t e^(L_(t-1)), then W
    float* Rm = Bm + C * ldk;            // [C][ldk]  r_t e^(L_t)
    float* Ab = Rm + C * ldk;            // [C][ldk]  a_s u_s e^(-L_s)
    float* Kb = Ab + C * ldk;            // [C][ldk]  k_s e^(-L_s)
    float* Vm = Kb + C * ldk;            // [C][ldv]
    float* Um = Vm + C * ldv;            // [C][ldv]
    float* sc = Um + C * ldv;            // [4][C][LDS]: u.au, u.k (s < t), r.au, r.k (s <= t)
    float* dend = sc + 4 * C * LDS;      // [dk]      e^L
    float* inv = dend + dk;              // [C]       1 / sqrt(sum(k^2) + 1e-6)
    pdl_wait();
    pdl_trigger();
    const int seg = blockIdx.z, h = blockIdx.y, t0 = blockIdx.x * C, n = seg_len[seg];
    if (t0 >= n) return;
    const int nt = min(C, n - t0), tid = threadIdx.x;
    constexpr int threads = PREP_THREADS;
    const int first = seg_start[seg];
    const size_t row0 = (size_t)first + t0, hk = (size_t)heads * dk, hv = (size_t)heads * dv;
    const size_t chunk = (size_t)chunk_base(first, seg) + blockIdx.x;

    // the rows as they are: log d, r, a, k, v (zeros behind the portion's end: such tokens change nothing)
    const int k4 = dk >> 2, v4 = dv >> 2;
    for (int e = tid; e < C * k4; e += threads) {
        const int t = e / k4, i = (e - t * k4) * 4;
        float4 ld = make_float4(0.f, 0.f, 0.f, 0.f), r = ld, a = ld, k = ld;
        if (t < nt) {
            const float* p = src.proj + (row0 + t) * src.ld + (size_t)h * dk + i;
            const float4 z = ld4(src.z + (row0 + t) * hk + (size_t)h * dk + i), ar = ld4(p + src.a_off);
            const int b = h * dk + i;
            r = ld4(p + src.r_off);
            k = ld4(p + src.k_off);
            ld = make_float4(-__fmul_rn(src.rate, sigmoid_f(z.x)), -__fmul_rn(src.rate, sigmoid_f(z.y)),
                             -__fmul_rn(src.rate, sigmoid_f(z.z)), -__fmul_rn(src.rate, sigmoid_f(z.w)));
            a = make_float4(sigmoid_f(ar.x + src.a_bias[b]), sigmoid_f(ar.y + src.a_bias[b + 1]),
                            sigmoid_f(ar.z + src.a_bias[b + 2]), sigmoid_f(ar.w + src.a_bias[b + 3]));
        }
        st4(Bm + t * ldk + i, ld);
        st4(Rm + t * ldk + i, r);
        st4(Ab + t * ldk + i, a);
        st4(Kb + t * ldk + i, k);
    }
    for (int e = tid; e < C * v4; e += threads) {
        const int t = e / v4, i = (e - t * v4) * 4;
        st4(Vm + t * ldv + i, t < nt ? ld4(src.proj + (row0 + t) * src.ld + src.v_off + (size_t)h * dv + i)
                                     : make_float4(0.f, 0.f, 0.f, 0.f));
    }
    __syncthreads();
    for (int t = tid >> 5; t < C; t += threads >> 5) {
        float ss = 0.f;
        for (int i = tid & 31; i < dk; i += 32) ss = fmaf(Kb[t * ldk + i], Kb[t * ldk + i], ss);
        ss = warp_sum(ss);
        if ((tid & 31) == 0) inv[t] = 1.f / sqrtf(ss + 1e-6f);
    }
    __syncthreads();
    for (int i = tid; i < dk; i += threads) {
        float L = 0.f, before = 1.f;
#pragma unroll 4
        for (int t = 0; t < C; ++t) {
            L += Bm[t * ldk + i];
            const float now = expf(L), back = expf(-L), k = Kb[t * ldk + i], u = __fmul_rn(k, inv[t]);
            Bm[t * ldk + i] = __fmul_rn(u, before);
            Rm[t * ldk + i] = __fmul_rn(Rm[t * ldk + i], now);
            Ab[t * ldk + i] = __fmul_rn(__fmul_rn(Ab[t * ldk + i], u), back);
            Kb[t * ldk + i] = __fmul_rn(k, back);
            before = now;
        }
        dend[i] = before;
    }
    __syncthreads();
    // the four score matrices
    for (int tile = tid; tile < 256; tile += threads) {
        const int which = tile >> 6, ty = tile & 7, sx = (tile >> 3) & 7;
        const float* A = (which & 2) ? Rm : Bm;
        const float* B = (which & 1) ? Kb : Ab;
        float acc[4][4] = {};
        for (int i = 0; i < dk; i += 4) {
            float4 av[4], bv[4];
#pragma unroll
            for (int a = 0; a < 4; ++a) {
                av[a] = ld4(A + (ty + 8 * a) * ldk + i);
                bv[a] = ld4(B + (sx + 8 * a) * ldk + i);
            }
#pragma unroll
            for (int a = 0; a < 4; ++a)
#pragma unroll
                for (int b = 0; b < 4; ++b)
                    acc[a][b] = fmaf(av[a].w, bv[b].w, fmaf(av[a].z, bv[b].z, fmaf(av[a].y, bv[b].y, fmaf(av[a].x, bv[b].x, acc[a][b]))));
        }
        float* dst = sc + which * C * LDS;
        const int incl = (which & 2) ? 1 : 0;
#pragma unroll
        for (int a = 0; a < 4; ++a)
#pragma unroll
            for (int b = 0; b < 4; ++b) {
                const int t = ty + 8 * a, s = sx + 8 * b;
                dst[t * LDS + s] = s < t + incl ? acc[a][b] : 0.f;
            }
    }
    __syncthreads();
    // the triangular system (I + [u.au]) X = [u e^(L_(t-1)) | [u.k] V]: the values' right-hand side first, as a product ...
    const float *uau = sc, *uk = sc + C * LDS, *rau = sc + 2 * C * LDS, *rk = sc + 3 * C * LDS;
    for (int tile = tid; tile < 8 * v4; tile += threads) {
        const int ty = tile & 7, i0 = (tile >> 3) * 4;
        float acc[4][4] = {};
        tile_rows<1>(acc, uk, Vm, ldv, ty, i0);
#pragma unroll
        for (int a = 0; a < 4; ++a) st4(Um + (ty + 8 * a) * ldv + i0, make_float4(acc[a][0], acc[a][1], acc[a][2], acc[a][3]));
    }
    __syncthreads();
    // ... then a thread per column, in place
    for (int col = tid; col < dk + dv; col += threads) {
        float* mine = col >= dk ? Um + (col - dk) : Bm + col;
        const int ldm = col >= dk ? ldv : ldk;
        float x[C];
#pragma unroll
        for (int t = 0; t < C; ++t) {
            float a0 = mine[t * ldm], a1 = 0.f;
#pragma unroll
            for (int s = 0; s < t; s += 4) {
                const float4 m = ld4(uau + t * LDS + s);         // (zeros from s = t on)
                a0 = fmaf(-m.x, x[s], a0);
                if (s + 1 < t) a1 = fmaf(-m.y, x[s + 1], a1);
                if (s + 2 < t) a0 = fmaf(-m.z, x[s + 2], a0);
                if (s + 3 < t) a1 = fmaf(-m.w, x[s + 3], a1);
            }
            x[t] = a0 + a1;
            mine[t * ldm] = x[t];
        }
    }
    __syncthreads();
    // what a token reads of the state in front of the chunk (Q) and of the chunk's own tokens (O)
    for (int tile = tid; tile < 8 * (k4 + v4); tile += threads) {
        const bool own = tile >= 8 * k4;
        const int ty = tile & 7, i0 = ((own ? tile - 8 * k4 : tile) >> 3) * 4;
        float acc[4][4];
        if (own) {
#pragma unroll
            for (int a = 0; a < 4; ++a) acc[a][0] = acc[a][1] = acc[a][2] = acc[a][3] = 0.f;
            tile_rows<1>(acc, rk, Vm, ldv, ty, i0);
            tile_rows<-1>(acc, rau, Um, ldv, ty, i0);
        } else {
#pragma unroll
            for (int a = 0; a < 4; ++a) {
                const float4 r = ld4(Rm + (ty + 8 * a) * ldk + i0);
                acc[a][0] = r.x; acc[a][1] = r.y; acc[a][2] = r.z; acc[a][3] = r.w;
            }
            tile_rows<-1>(acc, rau, Bm, ldk, ty, i0);
        }
#pragma unroll
        for (int a = 0; a < 4; ++a)
            if (ty + 8 * a < nt) {
                float* dst = own ? o + (row0 + ty + 8 * a) * hv + (size_t)h * dv + i0 : qp + (row0 + ty + 8 * a) * hk + (size_t)h * dk + i0;
                st4(dst, make_float4(acc[a][0], acc[a][1], acc[a][2], acc[a][3]));
            }
    }
    // the chunk's transition M and what it adds, N
    float* Mc = M + (chunk * heads + h) * (size_t)dk * dk;
    float* Nc = N + (chunk * heads + h) * (size_t)dk * dv;
    for (int tile = tid; tile < k4 * k4; tile += threads) {
        const int i0 = (tile % k4) * 4, j0 = (tile / k4) * 4;
        float acc[4][4] = {};
#pragma unroll 4
        for (int s = 0; s < C; ++s) {
            const float4 a = ld4(Ab + s * ldk + i0), w = ld4(Bm + s * ldk + j0);
            fma4(acc[0], -a.x, w);
            fma4(acc[1], -a.y, w);
            fma4(acc[2], -a.z, w);
            fma4(acc[3], -a.w, w);
        }
#pragma unroll
        for (int a = 0; a < 4; ++a) {
            const float d = dend[i0 + a];
            float m[4];
#pragma unroll
            for (int b = 0; b < 4; ++b) m[b] = __fmul_rn(d, acc[a][b] + (i0 + a == j0 + b ? 1.f : 0.f));
            st4(Mc + (size_t)(i0 + a) * dk + j0, make_float4(m[0], m[1], m[2], m[3]));
        }
    }
    for (int tile = tid; tile < k4 * v4; tile += threads) {
        const int i0 = (tile % k4) * 4, j0 = (tile / k4) * 4;
        float acc[4][4] = {};
#pragma unroll 4
        for (int s = 0; s < C; ++s) {
            const float4 a = ld4(Ab + s * ldk + i0), k = ld4(Kb + s * ldk + i0), v = ld4(Vm + s * ldv + j0), u = ld4(Um + s * ldv + j0);
            fma4(acc[0], k.x, v);
            fma4(acc[1], k.y, v);
            fma4(acc[2], k.z, v);
            fma4(acc[3], k.w, v);
            fma4(acc[0], -a.x, u);
            fma4(acc[1], -a.y, u);
            fma4(acc[2], -a.z, u);
            fma4(acc[3], -a.w, u);
        }
#pragma unroll
        for (int a = 0; a < 4; ++a) {
            const float d = dend[i0 + a];
            st4(Nc + (size_t)(i0 + a) * dv + j0,
                make_float4(__fmul_rn(d, acc[a][0]), __fmul_rn(d, acc[a][1]), __fmul_rn(d, acc[a][2]), __fmul_rn(d, acc[a][3])));
        }
    }
}

// S <- M S + N through a portion's chunks, a block per (segment, head, 16 value columns); N of a chunk is replaced by the state
// in front of it. M of the next chunks is on its way (cp.async, STAGES buffers) while this one's product runs.
// A thread makes a 4 x 4 tile of the product over one of JS parts of the sum; the parts meet in shared memory.
constexpr int WCB = 16;
constexpr int WALK_THREADS = 256;
template <int D, int STAGES, int JS>
__global__ void __launch_bounds__(WALK_THREADS)
delta_chunk_walk_kernel(const float* __restrict__ M, float* __restrict__ N, float* __restrict__ state, int num_slots,
                        const int* __restrict__ seg_start, const int* __restrict__ seg_len, const int* __restrict__ state_slots,
                        int heads, int dk_arg, int dv_arg) {
    const int dk = D ? D : dk_arg, dv = D ? D : dv_arg;
    extern __shared__ __align__(16) float smem[];
    const int ldm = dk + 4, c0 = blockIdx.x * WCB, h = blockIdx.y, seg = blockIdx.z;
    float* Ms = smem;                        // [STAGES][dk][ldm]
    float* Ns = Ms + STAGES * dk * ldm;      // [STAGES][dk][WCB]
    float* Ss = Ns + STAGES * dk * WCB;      // [dk][WCB]
    float* part = Ss + dk * WCB;             // [JS][dk][WCB]
    pdl_wait();
    pdl_trigger();
    const int first = seg_start[seg], n = seg_len[seg], slot = state_slots[seg];
    if (n <= 0 || !jllm_in_bounds(slot, num_slots, BOUNDS_SLOT)) return;
    constexpr int threads = WALK_THREADS;
    const int chunks = (n + C - 1) / C, tid = threadIdx.x, k4 = dk >> 2, cols = min(WCB, dv - c0);
    const size_t base = (size_t)chunk_base(first, seg);
    float* S = state + (((size_t)slot * heads + h) * dk) * dv + c0;
    auto fetch = [&](int ch, int b) {
        const float* m = M + ((base + ch) * heads + h) * (size_t)dk * dk;
        const float* nn = N + ((base + ch) * heads + h) * (size_t)dk * dv + c0;
        for (int e = tid; e < dk * k4; e += threads) {
            const int i = e / k4, x = (e - i * k4) * 4;
            const uint32_t dst = (uint32_t)__cvta_generic_to_shared(Ms + (size_t)b * dk * ldm + i * ldm + x);
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(m + (size_t)i * dk + x) : "memory");
        }
        for (int e = tid; e < dk * (WCB / 4); e += threads) {
            const int i = e / (WCB / 4), x = (e - i * (WCB / 4)) * 4;
            if (x < cols) {
                const uint32_t dst = (uint32_t)__cvta_generic_to_shared(Ns + b * dk * WCB + i * WCB + x);
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(nn + (size_t)i * dv + x) : "memory");
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    for (int e = tid; e < dk * WCB; e += threads) {
        const int i = e / WCB, x = e - i * WCB;
        Ss[e] = x < cols ? S[(size_t)i * dv + x] : 0.f;
        if (x >= cols)
            for (int b = 0; b < STAGES; ++b) Ns[b * dk * WCB + e] = 0.f;
    }
#pragma unroll
    for (int p = 0; p < STAGES - 1; ++p) {       // (an empty group where there is no such chunk: the counts stay the same)
        if (p < chunks) fetch(p, p);
        else asm volatile("cp.async.commit_group;" ::: "memory");
    }
    // this thread's tile: rows ig + k4 a, columns 4 cg .. 4 cg + 3; its part of the sum: groups of four [j_lo, j_hi)
    const int tile = tid % (k4 * (WCB / 4)), jp = tid / (k4 * (WCB / 4)), ig = tile / (WCB / 4), cg = (tile % (WCB / 4)) * 4;
    const int j_lo = jp * k4 / JS * 4, j_hi = (jp + 1) * k4 / JS * 4;
    int b = 0;
    for (int ch = 0; ch < chunks; ++ch) {
        // (the buffer that is filled now was read for the last time in front of the middle barrier of the turn before)
        if (ch + STAGES - 1 < chunks) fetch(ch + STAGES - 1, b == 0 ? STAGES - 1 : b - 1);
        else asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 1) : "memory");
        __syncthreads();
        float* out = N + ((base + ch) * heads + h) * (size_t)dk * dv + c0;
        for (int e = tid; e < dk * (WCB / 4); e += threads) {
            const int i = e / (WCB / 4), x = (e - i * (WCB / 4)) * 4;
            if (x < cols) st4(out + (size_t)i * dv + x, ld4(Ss + i * WCB + x));
        }
        if (jp < JS) {
            const float* m = Ms + (size_t)b * dk * ldm;
            float acc[4][4];
#pragma unroll
            for (int a = 0; a < 4; ++a) {
                const float4 v = jp == 0 ? ld4(Ns + b * dk * WCB + (ig + k4 * a) * WCB + cg) : make_float4(0.f, 0.f, 0.f, 0.f);
                acc[a][0] = v.x; acc[a][1] = v.y; acc[a][2] = v.z; acc[a][3] = v.w;
            }
#pragma unroll 2
            for (int j = j_lo; j < j_hi; j += 4) {
                const float4 s0 = ld4(Ss + j * WCB + cg), s1 = ld4(Ss + (j + 1) * WCB + cg), s2 = ld4(Ss + (j + 2) * WCB + cg),
                             s3 = ld4(Ss + (j + 3) * WCB + cg);
#pragma unroll
                for (int a = 0; a < 4; ++a) {
                    const float4 mv = ld4(m + (ig + k4 * a) * ldm + j);
                    fma4(acc[a], mv.x, s0);
                    fma4(acc[a], mv.y, s1);
                    fma4(acc[a], mv.z, s2);
                    fma4(acc[a], mv.w, s3);
                }
            }
#pragma unroll
            for (int a = 0; a < 4; ++a)
                st4(part + (jp * dk + ig + k4 * a) * WCB + cg, make_float4(acc[a][0], acc[a][1], acc[a][2], acc[a][3]));
        }
        __syncthreads();
        for (int e = tid * 4; e < dk * WCB; e += threads * 4) {
            float4 v = ld4(part + e);
#pragma unroll
            for (int p = 1; p < JS; ++p) {
                const float4 w = ld4(part + p * dk * WCB + e);
                v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w;
            }
            st4(Ss + e, v);
        }
        b = b + 1 == STAGES ? 0 : b + 1;
    }
    __syncthreads();
    for (int e = tid; e < dk * WCB; e += threads) {
        const int i = e / WCB, x = e - i * WCB;
        if (x < cols) S[(size_t)i * dv + x] = Ss[e];
    }
}

// o_t += Q_t^T S0 for all chunks at once (N holds the states in front of the chunks), and the norm and gate behind it (with
// nm.y null the sums go back to o)
template <int D>
__global__ void __launch_bounds__(128)
delta_chunk_out_kernel(const float* __restrict__ qp, const float* __restrict__ N, const int* __restrict__ seg_start,
                       const int* __restrict__ seg_len, float* __restrict__ o, DeltaNorm nm, int heads, int dk_arg, int dv_arg) {
    const int dk = D ? D : dk_arg, dv = D ? D : dv_arg;
    extern __shared__ __align__(16) float smem[];
    const int ldk = dk + 4, ldv = dv + 4;
    float* Qs = smem;                    // [C][ldk]
    float* Ss = Qs + C * ldk;            // [dk][ldv]
    float* Os = Ss + dk * ldv;           // [C][ldv]
    pdl_wait();
    pdl_trigger();
    const int seg = blockIdx.z, h = blockIdx.y, t0 = blockIdx.x * C, n = seg_len[seg];
    if (t0 >= n) return;
    constexpr int threads = 128;
    const int nt = min(C, n - t0), tid = threadIdx.x, k4 = dk >> 2, v4 = dv >> 2, first = seg_start[seg];
    const size_t row0 = (size_t)first + t0, hk = (size_t)heads * dk, hv = (size_t)heads * dv;
    const float* S = N + (((size_t)chunk_base(first, seg) + blockIdx.x) * heads + h) * (size_t)dk * dv;
    // the norm's share of this thread: sixteen lanes a row, eight rows a turn; heads of 64 have their gates on the way from here on
    const int sub = tid & 15, nrow = tid >> 4;
    float4 gates[4];
    if constexpr (D == 64) {
        if (nm.y != nullptr) {
#pragma unroll
            for (int q = 0; q < 4; ++q)
                gates[q] = nrow + 8 * q < nt ? ld4(nm.gate + (row0 + nrow + 8 * q) * nm.ld + (size_t)h * dv + sub * 4)
                                             : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    }
    for (int e = tid; e < C * k4; e += threads) {
        const int t = e / k4, i = (e - t * k4) * 4;
        st4(Qs + t * ldk + i, t < nt ? ld4(qp + (row0 + t) * hk + (size_t)h * dk + i) : make_float4(0.f, 0.f, 0.f, 0.f));
    }
    for (int e = tid; e < dk * v4; e += threads) {
        const int i = e / v4, x = (e - i * v4) * 4;
        st4(Ss + i * ldv + x, ld4(S + (size_t)i * dv + x));
    }
    __syncthreads();
    for (int tile = tid; tile < 8 * v4; tile += threads) {
        const int ty = tile & 7, j0 = (tile >> 3) * 4;
        float acc[4][4] = {};
#pragma unroll 2
        for (int i = 0; i < dk; i += 4) {
            float4 qv[4];
#pragma unroll
            for (int a = 0; a < 4; ++a) qv[a] = ld4(Qs + (ty + 8 * a) * ldk + i);
            const float4 s0 = ld4(Ss + i * ldv + j0), s1 = ld4(Ss + (i + 1) * ldv + j0), s2 = ld4(Ss + (i + 2) * ldv + j0),
                         s3 = ld4(Ss + (i + 3) * ldv + j0);
#pragma unroll
            for (int a = 0; a < 4; ++a) {
                fma4(acc[a], qv[a].x, s0);
                fma4(acc[a], qv[a].y, s1);
                fma4(acc[a], qv[a].z, s2);
                fma4(acc[a], qv[a].w, s3);
            }
        }
#pragma unroll
        for (int a = 0; a < 4; ++a) {
            const int t = ty + 8 * a;
            if (t >= nt) continue;
            float* src = o + (row0 + t) * hv + (size_t)h * dv + j0;
            const float4 old = ld4(src);
            st4(nm.y != nullptr ? Os + t * ldv + j0 : src,
                make_float4(old.x + acc[a][0], old.y + acc[a][1], old.z + acc[a][2], old.w + acc[a][3]));
        }
    }
    if (nm.y == nullptr) return;
    __syncthreads();
    if constexpr (D == 64) {
        float g[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) g[k] = nm.gain[h * dv + sub * 4 + k];
#pragma unroll
        for (int q = 0; q < 4; ++q) {
            const int t = nrow + 8 * q;
            const float4 v = ld4(Os + t * ldv + sub * 4);        // (rows behind the portion's end: whatever lies there, not stored)
            float ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w)));
#pragma unroll
            for (int m = 1; m < 16; m <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
            const float inv = 1.f / sqrtf(ss / (float)D + nm.eps);
            const float r0 = v.x * inv * g[0] * sigmoid_f(gates[q].x), r1 = v.y * inv * g[1] * sigmoid_f(gates[q].y);
            const float r2 = v.z * inv * g[2] * sigmoid_f(gates[q].z), r3 = v.w * inv * g[3] * sigmoid_f(gates[q].w);
            if (t >= nt) continue;
            const size_t at = (row0 + t) * hv + (size_t)h * dv + sub * 4;
            if (nm.dtype == JLLM_F32) {
                st4(static_cast<float*>(nm.y) + at, make_float4(r0, r1, r2, r3));
            } else {
                const __nv_bfloat162 lo = __floats2bfloat162_rn(r0, r1), hi = __floats2bfloat162_rn(r2, r3);
                uint2 u;
                u.x = *reinterpret_cast<const uint32_t*>(&lo);
                u.y = *reinterpret_cast<const uint32_t*>(&hi);
                *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(nm.y) + at) = u;
            }
        }
    } else {
        for (int t = tid >> 5; t < nt; t += threads >> 5) head_norm_row(nm, Os + t * ldv, row0 + t, h, heads, dv);
    }
}

template <int D>
int launch_chunked(const DeltaSource& src, const DeltaNorm& nm, float* state, int num_slots, const int* seg_start, const int* seg_len,
                   const int* state_slots, float* o, float* qp, float* M, float* N, int segments, int max_len, int heads, int dk,
                   int dv, cudaStream_t stream) {
    constexpr int STAGES = D == 64 ? 4 : 2, JS = D == 64 ? 4 : 2;      // (256 threads, dk tiles: JS x dk <= 256)
    const size_t prep = (size_t)(4 * C * (dk + 4) + 2 * C * (dv + 4) + 4 * C * LDS + dk + C) * sizeof(float);
    const size_t walk = (size_t)(STAGES * dk * (dk + 4) + (STAGES + 1 + JS) * dk * WCB) * sizeof(float);
    const size_t outs = (size_t)(C * (dk + 4) + dk * (dv + 4) + C * (dv + 4)) * sizeof(float);
    static bool ready = false;
    if (!ready) {
        constexpr int W = D ? D : 128;
        const int most_prep = (int)((6 * C * (W + 4) + 4 * C * LDS + W + C) * sizeof(float));
        const int most_walk = (int)((STAGES * W * (W + 4) + (STAGES + 1 + JS) * W * WCB) * sizeof(float));
        const int most_out = (int)((2 * C * (W + 4) + W * (W + 4)) * sizeof(float));
        if (cudaFuncSetAttribute(delta_chunk_prepare_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, most_prep) != cudaSuccess ||
            cudaFuncSetAttribute(delta_chunk_walk_kernel<D, STAGES, JS>, cudaFuncAttributeMaxDynamicSharedMemorySize, most_walk) != cudaSuccess ||
            cudaFuncSetAttribute(delta_chunk_out_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, most_out) != cudaSuccess)
            return jllm_fail(JLLM_CUDA_ERROR, "delta_chunked: shared memory refused");
        ready = true;
    }
    const int chunks = (max_len + C - 1) / C;
    jllm_launch(delta_chunk_prepare_kernel<D>, dim3(chunks, heads, segments), dim3(PREP_THREADS), prep, stream, LAUNCH_DEPENDENT, src,
                seg_start, seg_len, qp, o, M, N, heads, dk, dv);
    if (int code = jllm_check_launch("delta_chunk_prepare")) return code;
    jllm_launch(delta_chunk_walk_kernel<D, STAGES, JS>, dim3((dv + WCB - 1) / WCB, heads, segments), dim3(WALK_THREADS), walk, stream,
                LAUNCH_DEPENDENT, (const float*)M, N, state, num_slots, seg_start, seg_len, state_slots, heads, dk, dv);
    if (int code = jllm_check_launch("delta_chunk_walk")) return code;
    jllm_launch(delta_chunk_out_kernel<D>, dim3(chunks, heads, segments), dim3(128), outs, stream, LAUNCH_DEPENDENT, (const float*)qp,
                (const float*)N, seg_start, seg_len, o, nm, heads, dk, dv);
    return jllm_check_launch("delta_chunk_out");
}

}  // namespace

JLLM_BOUNDS_READER(delta_recurrence)

// out [rows, width] of type `dtype` = tanh of a float32 view [rows, ld].
JLLM_EXPORT int jllm_delta_tanh(const float* src, int ld, void* out, int dtype, int rows, int width, cudaStream_t stream) {
    JLLM_REQUIRE(rows >= 0 && width > 0 && (long long)rows * width < (1ll << 31), "delta_tanh: rows=%d width=%d", rows, width);
    if (rows == 0) return JLLM_OK;
    const int blocks = min(4096, (rows * width + 255) / 256);
    if (dtype == JLLM_F32)
        jllm_launch(delta_tanh_kernel<float>, dim3(blocks), dim3(256), 0, stream, LAUNCH_DEPENDENT, src, ld, (float*)out, rows, width);
    else
        jllm_launch(delta_tanh_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, LAUNCH_DEPENDENT, src, ld,
                    (__nv_bfloat16*)out, rows, width);
    return jllm_check_launch("delta_tanh");
}

// proj [rows, ld] float32 with r, k, a_raw (heads x dk) and v (heads x dv) at the given columns; z [rows, heads x dk] float32;
// a_bias [heads x dk]; state [slots, heads, dk, dv] float32, read and written in place; o [rows, heads x dv] float32. With y
// [rows, heads x dv] of type `y_dtype` (heads of at most 64 values: JLLM_UNSUPPORTED, with nothing launched, where a block does not
// hold a head's columns) the norm and gate behind the recurrence are taken along and o is not written.
JLLM_EXPORT int jllm_delta_recurrent(const float* proj, int ld, int r_off, int k_off, int v_off, int a_off, const float* z,
                                     const void* a_bias, int bias_dtype, float rate, float* state, int num_slots,
                                     const int* seg_start, const int* seg_len, const int* state_slots, float* o,
                                     const float* gate, int ld_gate, const void* gain, int gain_dtype, float eps, void* y,
                                     int y_dtype, int segments, int heads, int dk, int dv, cudaStream_t stream) {
    JLLM_REQUIRE(segments >= 0 && heads > 0 && heads <= 65535 && dk > 0 && dk <= 1024 && dv > 0 && dv <= 65535 * 8,
                 "delta_recurrent: segments=%d heads=%d dk=%d (at most 1024) dv=%d", segments, heads, dk, dv);
    if (segments == 0) return JLLM_OK;
    const DeltaSource src{proj, z, VecRef{a_bias, bias_dtype}, rate, ld, r_off, k_off, v_off, a_off};
    const DeltaNorm nm{gate, y, VecRef{gain, gain_dtype}, eps, ld_gate, y_dtype};
#define JLLM_DELTA(LS, R, CB, TOK)                                                                                             \
    return launch_recurrent<LS, R, CB, TOK>(src, state, num_slots, seg_start, seg_len, state_slots, o, nm, segments, heads, dk, dv, \
                                            stream)
    if (y != nullptr) {
        if (dk > 64 || dv > 64) return JLLM_UNSUPPORTED;
        if (dv <= 32) JLLM_DELTA(4, 16, 32, 8);
        JLLM_DELTA(4, 16, 64, 8);
    }
    if (dk <= 32) JLLM_DELTA(4, 8, 32, 8);
    if (dk <= 64) JLLM_DELTA(4, 16, 32, 8);
    if (dk <= 128) JLLM_DELTA(8, 16, 32, 8);
    if (dk <= 256) JLLM_DELTA(16, 16, 16, 8);
    if (dk <= 512) JLLM_DELTA(32, 16, 8, 4);
    JLLM_DELTA(32, 32, 8, 4);
#undef JLLM_DELTA
}

// The same for prompt portions, in chunks of 32 tokens: three launches (the last one takes the norm and gate along with y). qp [rows, heads x dk], M [chunks, heads, dk, dk] and N
// [chunks, heads, dk, dv] float32 scratch, chunks >= rows / 32 + segments. JLLM_UNSUPPORTED, with nothing launched, where the
// sizes are not taken.
JLLM_EXPORT int jllm_delta_chunked(const float* proj, int ld, int r_off, int k_off, int v_off, int a_off, const float* z,
                                   const void* a_bias, int bias_dtype, float rate, float* state, int num_slots,
                                   const int* seg_start, const int* seg_len, const int* state_slots, float* o, float* qp, float* M,
                                   float* N, const float* gate, int ld_gate, const void* gain, int gain_dtype, float eps,
                                   void* y, int y_dtype, int segments, int max_len, int heads, int dk, int dv,
                                   cudaStream_t stream) {
    if (dk % 4 || dv % 4 || dk > 128 || dv > 128 || dk <= 0 || dv <= 0 || ld % 4 || r_off % 4 || k_off % 4 || v_off % 4 || a_off % 4 ||
        ((uintptr_t)proj % 16) || ((uintptr_t)z % 16) || !(rate * C <= 60.f) || segments > 65535 || heads > 65535)
        return JLLM_UNSUPPORTED;
    if (segments <= 0 || max_len <= 0) return JLLM_OK;
    const DeltaSource src{proj, z, VecRef{a_bias, bias_dtype}, rate, ld, r_off, k_off, v_off, a_off};
    const DeltaNorm nm{gate, y, VecRef{gain, gain_dtype}, eps, ld_gate, y_dtype};
#define JLLM_CHUNKED(D)                                                                                                        \
    return launch_chunked<D>(src, nm, state, num_slots, seg_start, seg_len, state_slots, o, qp, M, N, segments, max_len, heads, dk, \
                             dv, stream)
    if (dk == 64 && dv == 64 && (y == nullptr || (ld_gate % 4 == 0 && ((uintptr_t)gate % 16) == 0 && ((uintptr_t)y % 16) == 0)))
        JLLM_CHUNKED(64);
    if (dk == 128 && dv == 128) JLLM_CHUNKED(128);
    JLLM_CHUNKED(0);
#undef JLLM_CHUNKED
}
