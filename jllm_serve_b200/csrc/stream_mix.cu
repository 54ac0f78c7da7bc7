// Hyper-connections: a residual of several streams X_1 .. X_S (float32, [rows, S, dim]) instead of one. A part reads a weighted sum
// of them, and behind the part the streams are mixed among each other and each takes the part's result y with a weight of its own:
//
//   X_t <- sum_s mix[s, t] X_s + out[t] y        (all streams from the old ones)
//   u    = sum_s in'[s] X_s,   h = u / sqrt(mean(u^2) + eps) * gain        (the NEXT part's input, in the compute type)
//
// One launch between a part and the next does both: a block per row holds the row's streams in registers, so they are read once
// and written once. The same launch has two more uses. `x0` (the embedded rows): all streams begin as copies of it, and the
// first part's input is made. A last launch with `row_index`, which does not write the streams back: for the rows that are asked
// for, mix, sum (in' all ones) and the model's last norm.
//
// The streams were written by a launch in front of the part's, which has ended before the part's last product (this launch's
// predecessor) let it start: they are fetched before the wait for that product. All arithmetic is float32, sums in ascending s with
// y last; a row's result depends on that row alone.
#include "common.cuh"

namespace {

constexpr int MAX_STREAMS = 16;

__device__ __forceinline__ void add_scaled4(float4& a, float f, const float4& v) {
    a.x = fmaf(f, v.x, a.x);
    a.y = fmaf(f, v.y, a.y);
    a.z = fmaf(f, v.z, a.z);
    a.w = fmaf(f, v.w, a.w);
}
__device__ __forceinline__ float4 scaled4(float f, const float4& v) {
    return make_float4(__fmul_rn(f, v.x), __fmul_rn(f, v.y), __fmul_rn(f, v.z), __fmul_rn(f, v.w));
}

// coef: mix [S, S] (from, to), then out [S]; read: in' [S]. A thread holds N groups of four values of every stream.
template <int S, int N, typename Tout>
__global__ void __launch_bounds__(512)
stream_mix_kernel(float* __restrict__ X, const float* __restrict__ x0, const float* __restrict__ y, const float* __restrict__ coef,
                  const float* __restrict__ read, VecRef gain, Tout* __restrict__ out, const int* __restrict__ row_index, int dim,
                  float eps, int write) {
    __shared__ float scratch[33];
    const int r = blockIdx.x, src = row_index ? row_index[r] : r, groups = dim >> 2;
    float4* xr = reinterpret_cast<float4*>(X + (size_t)src * S * dim);
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 v[S][N];
    if (x0 == nullptr) {
#pragma unroll
        for (int s = 0; s < S; ++s)
#pragma unroll
            for (int k = 0; k < N; ++k) {
                const int i = threadIdx.x + k * blockDim.x;
                v[s][k] = i < groups ? __ldcg(xr + (size_t)s * groups + i) : zero;
            }
    }
    // (so are the weights, which nobody writes)
    float m[S * S + S], in[S];
#pragma unroll
    for (int j = 0; j < S * S + S; ++j) m[j] = coef != nullptr ? __ldg(coef + j) : 0.f;
#pragma unroll
    for (int j = 0; j < S; ++j) in[j] = read != nullptr ? __ldg(read + j) : 0.f;
    if (read != nullptr && r < 8) prefetch_lines(gain.p, (size_t)dim * (gain.dtype == JLLM_F32 ? 4 : 2));
    pdl_wait();
    pdl_trigger();
    if (x0 != nullptr) {
        const float4* b = reinterpret_cast<const float4*>(x0 + (size_t)src * dim);
#pragma unroll
        for (int k = 0; k < N; ++k) {
            const int i = threadIdx.x + k * blockDim.x;
            v[0][k] = i < groups ? b[i] : zero;
#pragma unroll
            for (int s = 1; s < S; ++s) v[s][k] = v[0][k];
        }
    }
    if (y != nullptr) {
        const float4* yr = reinterpret_cast<const float4*>(y + (size_t)src * dim);
        float4 yv[N];
#pragma unroll
        for (int k = 0; k < N; ++k) {
            const int i = threadIdx.x + k * blockDim.x;
            yv[k] = i < groups ? yr[i] : zero;
        }
#pragma unroll
        for (int k = 0; k < N; ++k) {
            float4 n[S];
#pragma unroll
            for (int t = 0; t < S; ++t) {
                n[t] = scaled4(m[t], v[0][k]);
#pragma unroll
                for (int s = 1; s < S; ++s) add_scaled4(n[t], m[s * S + t], v[s][k]);
                add_scaled4(n[t], m[S * S + t], yv[k]);
            }
#pragma unroll
            for (int t = 0; t < S; ++t) v[t][k] = n[t];
        }
    }
    if (write) {
#pragma unroll
        for (int s = 0; s < S; ++s)
#pragma unroll
            for (int k = 0; k < N; ++k) {
                const int i = threadIdx.x + k * blockDim.x;
                if (i < groups) xr[(size_t)s * groups + i] = v[s][k];
            }
    }
    if (read == nullptr) return;
    float4 u[N];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < N; ++k) {
        u[k] = scaled4(in[0], v[0][k]);
#pragma unroll
        for (int s = 1; s < S; ++s) add_scaled4(u[k], in[s], v[s][k]);
        ss = fmaf(u[k].x, u[k].x, fmaf(u[k].y, u[k].y, fmaf(u[k].z, u[k].z, fmaf(u[k].w, u[k].w, ss))));
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.f / sqrtf(ss / (float)dim + eps);
    Tout* dst = out + (size_t)r * dim;
#pragma unroll
    for (int k = 0; k < N; ++k) {
        const int i = threadIdx.x + k * blockDim.x;
        if (i >= groups) continue;
        float g[4];
        if (gain.dtype == JLLM_F32) {
            const float4 gv = reinterpret_cast<const float4*>(gain.p)[i];
            g[0] = gv.x; g[1] = gv.y; g[2] = gv.z; g[3] = gv.w;
        } else {
            const uint2 raw = reinterpret_cast<const uint2*>(gain.p)[i];
            const __nv_bfloat16* e = reinterpret_cast<const __nv_bfloat16*>(&raw);
#pragma unroll
            for (int c = 0; c < 4; ++c) g[c] = __bfloat162float(e[c]);
        }
        const float o0 = __fmul_rn(__fmul_rn(u[k].x, inv), g[0]), o1 = __fmul_rn(__fmul_rn(u[k].y, inv), g[1]);
        const float o2 = __fmul_rn(__fmul_rn(u[k].z, inv), g[2]), o3 = __fmul_rn(__fmul_rn(u[k].w, inv), g[3]);
        if constexpr (sizeof(Tout) == 4) {
            reinterpret_cast<float4*>(dst)[i] = make_float4(o0, o1, o2, o3);
        } else {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(o0, o1), hi = __floats2bfloat162_rn(o2, o3);
            uint2 p;
            p.x = *reinterpret_cast<const uint32_t*>(&lo);
            p.y = *reinterpret_cast<const uint32_t*>(&hi);
            reinterpret_cast<uint2*>(dst)[i] = p;
        }
    }
}

// Any number of streams up to MAX_STREAMS and any width: two passes, the second of which does the first's sums anew (and stores).
template <typename Tout>
__global__ void __launch_bounds__(256)
stream_mix_any_kernel(float* __restrict__ X, const float* __restrict__ x0, const float* __restrict__ y, const float* __restrict__ coef,
                      const float* __restrict__ read, VecRef gain, Tout* __restrict__ out, const int* __restrict__ row_index, int dim,
                      float eps, int write, int S) {
    __shared__ float scratch[33];
    __shared__ float m[MAX_STREAMS * MAX_STREAMS + 2 * MAX_STREAMS];
    pdl_wait();
    pdl_trigger();
    const int r = blockIdx.x, src = row_index ? row_index[r] : r;
    float* xr = X + (size_t)src * S * dim;
    if (coef != nullptr)
        for (int j = threadIdx.x; j < S * S + S; j += blockDim.x) m[j] = coef[j];
    if (read != nullptr)
        for (int j = threadIdx.x; j < S; j += blockDim.x) m[S * S + S + j] = read[j];
    __syncthreads();
    // the streams' new values at place i, and their weighted sum
    auto place = [&](int i, float (&n)[MAX_STREAMS]) {
        float v[MAX_STREAMS];
#pragma unroll
        for (int s = 0; s < MAX_STREAMS; ++s)
            if (s < S) v[s] = x0 != nullptr ? x0[(size_t)src * dim + i] : xr[(size_t)s * dim + i];
        const float yv = y != nullptr ? y[(size_t)src * dim + i] : 0.f;
        float u = 0.f;
#pragma unroll
        for (int t = 0; t < MAX_STREAMS; ++t) {
            if (t >= S) continue;
            n[t] = v[t];
            if (y != nullptr) {
                float a = __fmul_rn(m[t], v[0]);
#pragma unroll
                for (int s = 1; s < MAX_STREAMS; ++s)
                    if (s < S) a = fmaf(m[s * S + t], v[s], a);
                n[t] = fmaf(m[S * S + t], yv, a);
            }
            if (read != nullptr) u = t == 0 ? __fmul_rn(m[S * S + S], n[0]) : fmaf(m[S * S + S + t], n[t], u);
        }
        return u;
    };
    float n[MAX_STREAMS];
    float inv = 1.f;
    if (read != nullptr) {
        float ss = 0.f;
        for (int i = threadIdx.x; i < dim; i += blockDim.x) {
            const float u = place(i, n);
            ss = fmaf(u, u, ss);
        }
        ss = block_sum(ss, scratch);
        inv = 1.f / sqrtf(ss / (float)dim + eps);
    }
    for (int i = threadIdx.x; i < dim; i += blockDim.x) {
        const float u = place(i, n);
        if (write) {
#pragma unroll
            for (int s = 0; s < MAX_STREAMS; ++s)
                if (s < S) xr[(size_t)s * dim + i] = n[s];
        }
        if (read != nullptr) out[(size_t)r * dim + i] = from_float<Tout>(__fmul_rn(__fmul_rn(u, inv), gain[i]));
    }
}

template <int S, typename Tout>
void launch(int groups, float* X, const float* x0, const float* y, const float* coef, const float* read, VecRef gain, Tout* out,
            const int* row_index, int rows, int dim, float eps, int write, cudaStream_t stream) {
    // two groups a thread where that fills at least four warps, up to 512 threads; then four
    int threads = 128;
    while (threads < 512 && threads * 2 < groups) threads *= 2;
#define JLLM_MIX(N)                                                                                                            \
    jllm_launch(stream_mix_kernel<S, N, Tout>, dim3(rows), dim3(threads), 0, stream, LAUNCH_DEPENDENT, X, x0, y, coef, read, gain, out, \
                row_index, dim, eps, write)
    if (groups <= threads) JLLM_MIX(1);
    else if (groups <= 2 * threads) JLLM_MIX(2);
    else JLLM_MIX(4);
#undef JLLM_MIX
}

}  // namespace

// X [rows, streams, dim] float32. x0 [rows, dim] float32 or null: the streams begin as copies of it. y [rows, dim] float32 or null,
// with coef = mix [streams, streams] and out [streams] behind it. read [streams] or null: out[r] = the norm of the weighted sum, in
// `out_dtype`. row_index (or null): row r of `out` comes from row row_index[r] of X and y (`write` must then be 0). `write`: the
// streams' new values are stored.
JLLM_EXPORT int jllm_stream_mix(float* X, int streams, const float* x0, const float* y, const float* coef, const float* read,
                                const void* gain, int gain_dtype, void* out, int out_dtype, const int* row_index, int rows, int dim,
                                float eps, int write, cudaStream_t stream) {
    JLLM_REQUIRE(rows >= 0 && dim > 0 && streams >= 1 && streams <= MAX_STREAMS, "stream_mix: rows=%d dim=%d streams=%d (at most %d)",
                 rows, dim, streams, MAX_STREAMS);
    JLLM_REQUIRE((y == nullptr || coef != nullptr) && (read == nullptr || (out != nullptr && gain != nullptr)) &&
                     !(write && row_index != nullptr) && !(x0 != nullptr && y != nullptr),
                 "stream_mix: a result needs its weights, a read its gain and output, picked rows are not written back");
    if (rows == 0 || (!write && read == nullptr)) return JLLM_OK;
    const VecRef g{gain, gain_dtype};
    const int groups = dim / 4;
    const bool vec = dim % 4 == 0 && groups <= 2048 && streams <= 4 &&
                     (((uintptr_t)X | (uintptr_t)x0 | (uintptr_t)y | (uintptr_t)out | (uintptr_t)gain) % 16) == 0;
#define JLLM_GO(S, T) launch<S, T>(groups, X, x0, y, coef, read, g, (T*)out, row_index, rows, dim, eps, write, stream)
    if (vec && out_dtype == JLLM_F32) {
        if (streams == 1) JLLM_GO(1, float); else if (streams == 2) JLLM_GO(2, float); else if (streams == 3) JLLM_GO(3, float); else JLLM_GO(4, float);
    } else if (vec) {
        if (streams == 1) JLLM_GO(1, __nv_bfloat16); else if (streams == 2) JLLM_GO(2, __nv_bfloat16);
        else if (streams == 3) JLLM_GO(3, __nv_bfloat16); else JLLM_GO(4, __nv_bfloat16);
    } else if (out_dtype == JLLM_F32) {
        jllm_launch(stream_mix_any_kernel<float>, dim3(rows), dim3(256), 0, stream, LAUNCH_DEPENDENT, X, x0, y, coef, read, g, (float*)out,
                    row_index, dim, eps, write, streams);
    } else {
        jllm_launch(stream_mix_any_kernel<__nv_bfloat16>, dim3(rows), dim3(256), 0, stream, LAUNCH_DEPENDENT, X, x0, y, coef, read, g,
                    (__nv_bfloat16*)out, row_index, dim, eps, write, streams);
    }
#undef JLLM_GO
    return jllm_check_launch("stream_mix");
}
