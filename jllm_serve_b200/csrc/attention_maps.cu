// The rows of an attention whose heads are not one block of one width each ("wide" attention): what happens between the input
// product and the paged attention, and behind it.
//
//   map_prepare      from the stacked projection's rows [q | k | v]: an optional RMS norm over ALL query (key) columns of a row at
//                    once with a gain per column; rotation of the first rotary_dim values of every map; then
//                      * query (head h, map m) to its own row of `width` values, its `dim` values at place m * dim, zeros elsewhere;
//                      * the maps of a key head side by side into ONE cached row of `width` values, zeros behind them;
//                      * the value into the value row, zeros behind it (v_off = k_off: the values are the keys as projected).
//                    Queries may grow with their position: q times 1 + temp_coef ln(floor((p + 1) / temp_every) + 1).
//                    A query's dot product with a cached row is then the dot product with its own map alone, so an attention with
//                    heads x maps query heads and kv_heads key / value heads of one width computes all maps over values that are
//                    cached once, on the kernels that were built for plain heads.
//   map_difference   o_h = a_(h,1) - lambda a_(h,2) from the two maps' results, over its root mean square, times `out_scale`.
//
// Float32 arithmetic; T is the type of projections and cache.
#include "common.cuh"

namespace {

template <typename T, int N>
__device__ __forceinline__ void load_piece(const T* p, float (&o)[N]) {
    if constexpr (N * sizeof(T) == 16) {
        const uint4 raw = *reinterpret_cast<const uint4*>(p);
        const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
        for (int k = 0; k < N; ++k) o[k] = to_float(e[k]);
    } else {
#pragma unroll
        for (int k = 0; k < N; ++k) o[k] = to_float(p[k]);
    }
}
template <typename T, int N>
__device__ __forceinline__ void store_piece(T* p, const float (&o)[N]) {
    if constexpr (N * sizeof(T) == 16) {
        uint4 raw;
        T* e = reinterpret_cast<T*>(&raw);
#pragma unroll
        for (int k = 0; k < N; ++k) e[k] = from_float<T>(o[k]);
        *reinterpret_cast<uint4*>(p) = raw;
    } else {
#pragma unroll
        for (int k = 0; k < N; ++k) p[k] = from_float<T>(o[k]);
    }
}

struct MapShape {
    int heads, kv_heads, maps, dim, vdim, width, page_size, rotary_dim, pairing;
    int ld, k_off, v_off, ld_q;
    int temp_every;            // 0: the queries are not multiplied
    float temp_coef;
};

// One block per row. N values a thread at a time (N > 1 only where every piece of every part is whole and aligned).
template <typename T, int N>
__global__ void __launch_bounds__(256)
map_prepare_kernel(const T* __restrict__ src, MapShape s, const float* __restrict__ q_gain, const float* __restrict__ k_gain, float eps,
                   const float* __restrict__ cos_t, const float* __restrict__ sin_t, const int* __restrict__ positions,
                   const int* __restrict__ slots, T* __restrict__ q_out, T* __restrict__ k_cache, T* __restrict__ v_cache,
                   int write_kv, int num_slots) {
    __shared__ float scratch[33];
    pdl_wait();
    pdl_trigger();
    const size_t r = blockIdx.x;
    const T* row = src + r * s.ld;
    const int q_cols = s.heads * s.maps * s.dim, k_cols = s.kv_heads * s.maps * s.dim, tid = threadIdx.x;
    auto root = [&](const T* p, int n) {         // 1 / root mean square of n values
        float ss = 0.f;
        for (int i = tid * N; i < n; i += blockDim.x * N) {
            float v[N];
            load_piece<T, N>(p + i, v);
#pragma unroll
            for (int k = 0; k < N; ++k) ss = fmaf(v[k], v[k], ss);
        }
        ss = block_sum(ss, scratch);
        return 1.f / sqrtf(ss / (float)n + eps);
    };
    float inv_q = 1.f, inv_k = 1.f;
    if (q_gain != nullptr) inv_q = root(row, q_cols);
    if (k_gain != nullptr && write_kv) inv_k = root(row + s.k_off, k_cols);
    const int half = s.rotary_dim >> 1;
    const float* cs = s.rotary_dim ? cos_t + (size_t)positions[r] * half : nullptr;
    const float* sn = s.rotary_dim ? sin_t + (size_t)positions[r] * half : nullptr;
    // N values from place i on of the map that begins at column `col` of `part`
    auto take = [&](const T* part, const float* gain, float inv, int col, int i, float (&o)[N]) {
        load_piece<T, N>(part + col + i, o);
        if (gain != nullptr) {
#pragma unroll
            for (int k = 0; k < N; ++k) o[k] = __fmul_rn(__fmul_rn(o[k], inv), gain[col + i + k]);
        }
        if (i < s.rotary_dim) {
            if (s.pairing == 0) {
                // (the pieces of a map are whole on either side of rotary_dim and of half: the host chose N so)
                const bool low = i < half;
                const int pi = low ? i + half : i - half;
                float w[N];
                load_piece<T, N>(part + col + pi, w);
#pragma unroll
                for (int k = 0; k < N; ++k) {
                    if (gain != nullptr) w[k] = __fmul_rn(__fmul_rn(w[k], inv), gain[col + pi + k]);
                    const int a = (low ? i : pi) + k;
                    o[k] = low ? __fmaf_rn(o[k], cs[a], -__fmul_rn(w[k], sn[a])) : __fmaf_rn(o[k], cs[a], __fmul_rn(w[k], sn[a]));
                }
            } else if constexpr (N > 1) {
#pragma unroll
                for (int k = 0; k < N; k += 2) {
                    const int a = (i + k) >> 1;
                    const float u = o[k], v = o[k + 1];
                    o[k] = __fmaf_rn(u, cs[a], -__fmul_rn(v, sn[a]));
                    o[k + 1] = __fmaf_rn(v, cs[a], __fmul_rn(u, sn[a]));
                }
            } else {
                const int pi = i ^ 1, a = i >> 1;
                float w = to_float(part[col + pi]);
                if (gain != nullptr) w = __fmul_rn(__fmul_rn(w, inv), gain[col + pi]);
                o[0] = (i & 1) ? __fmaf_rn(o[0], cs[a], __fmul_rn(w, sn[a])) : __fmaf_rn(o[0], cs[a], -__fmul_rn(w, sn[a]));
            }
        }
    };
    const int W = s.width;
    const float temp = s.temp_every > 0 ? fmaf(s.temp_coef, logf((float)((positions[r] + 1) / s.temp_every + 1)), 1.f) : 1.f;
    for (int e = tid * N; e < s.heads * s.maps * W; e += blockDim.x * N) {
        const int hm = e / W, i = e - hm * W - (hm % s.maps) * s.dim;
        float o[N] = {};
        if (i >= 0 && i < s.dim) {
            take(row, q_gain, inv_q, hm * s.dim, i, o);
            if (s.temp_every > 0) {
#pragma unroll
                for (int k = 0; k < N; ++k) o[k] = __fmul_rn(o[k], temp);
            }
        }
        store_piece<T, N>(q_out + r * s.ld_q + e, o);
    }
    if (!write_kv) return;
    const int slot = slots[r];
    if (!jllm_in_bounds(slot, num_slots, BOUNDS_SLOT)) return;
    const size_t page = slot / s.page_size, off = slot % s.page_size;
    for (int e = tid * N; e < s.kv_heads * W; e += blockDim.x * N) {
        const int g = e / W, cc = e - g * W, m = cc / s.dim;
        float o[N] = {}, v[N] = {};
        if (m < s.maps) take(row + s.k_off, k_gain, inv_k, (g * s.maps + m) * s.dim, cc - m * s.dim, o);
        if (cc < s.vdim) load_piece<T, N>(row + s.v_off + (size_t)g * s.vdim + cc, v);
        const size_t at = ((page * s.kv_heads + g) * s.page_size + off) * W + cc;
        store_piece<T, N>(k_cache + at, o);
        store_piece<T, N>(v_cache + at, v);
    }
}

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}
__device__ __forceinline__ float4 gained4(float4 v, float f, float4 g) {
    return make_float4(__fmul_rn(__fmul_rn(v.x, f), g.x), __fmul_rn(__fmul_rn(v.y, f), g.y), __fmul_rn(__fmul_rn(v.z, f), g.z),
                       __fmul_rn(__fmul_rn(v.w, f), g.w));
}

// The same for rows that are normed and rotated by halves (or not at all), where every piece is whole and aligned: the row's queries
// and keys are read once, into shared memory as float32, both sums of squares meet in one reduction, and a thread turns both pieces of
// a pair, so a gain and an angle are read once. Four values a thread at a time: neighbouring threads then read neighbouring 16 bytes.
template <typename T>
__global__ void __launch_bounds__(256)
map_prepare_normed_kernel(const T* __restrict__ src, MapShape s, const float* __restrict__ q_gain, const float* __restrict__ k_gain, float eps,
                          const float* __restrict__ cos_t, const float* __restrict__ sin_t, const int* __restrict__ positions,
                          const int* __restrict__ slots, T* __restrict__ q_out, T* __restrict__ k_cache, T* __restrict__ v_cache,
                          int write_kv, int num_slots) {
    extern __shared__ __align__(16) float staged[];        // the query columns, then the key columns
    __shared__ float sums[2][8];
    const size_t r = blockIdx.x;
    const int q_cols = s.heads * s.maps * s.dim, k_cols = write_kv ? s.kv_heads * s.maps * s.dim : 0, tid = threadIdx.x;
    // (positions and slots came from the host before the step)
    const int pos = positions[r], slot = write_kv ? slots[r] : 0, half = s.rotary_dim >> 1, W = s.width;
    const float* cs = s.rotary_dim ? cos_t + (size_t)pos * half : nullptr;
    const float* sn = s.rotary_dim ? sin_t + (size_t)pos * half : nullptr;
    const float temp = s.temp_every > 0 ? fmaf(s.temp_coef, logf((float)((pos + 1) / s.temp_every + 1)), 1.f) : 1.f;
    pdl_wait();
    pdl_trigger();
    const T* row = src + r * s.ld;
    float ss[2] = {0.f, 0.f};
    for (int i = tid * 4; i < q_cols + k_cols; i += 1024) {
        const float4 v = load4(i < q_cols ? row + i : row + s.k_off + (i - q_cols));
        const float a = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w)));
        if (i < q_cols) ss[0] += a;
        else ss[1] += a;
        store4(staged + i, v);
    }
#pragma unroll
    for (int w = 0; w < 2; ++w) {
        const float part = warp_sum(ss[w]);
        if ((tid & 31) == 0) sums[w][tid >> 5] = part;
    }
    __syncthreads();
    float inv[2];
#pragma unroll
    for (int w = 0; w < 2; ++w) {
        float all = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) all += sums[w][i];
        inv[w] = 1.f / sqrtf(all / (float)max(1, w == 0 ? q_cols : k_cols) + eps);
    }
    // both pieces of the pair at place i < half of the map whose columns begin at `col` of `part`, times f, to dst and dst + half
    auto turn = [&](const float* part, const float* gain, float f, int col, int i, float t, T* dst) {
        const float4 u = gained4(load4(part + col + i), f, load4(gain + col + i));
        const float4 w = gained4(load4(part + col + half + i), f, load4(gain + col + half + i));
        const float4 c = load4(cs + i), d = load4(sn + i);
        float4 a, b;
        a.x = __fmaf_rn(u.x, c.x, -__fmul_rn(w.x, d.x)); b.x = __fmaf_rn(w.x, c.x, __fmul_rn(u.x, d.x));
        a.y = __fmaf_rn(u.y, c.y, -__fmul_rn(w.y, d.y)); b.y = __fmaf_rn(w.y, c.y, __fmul_rn(u.y, d.y));
        a.z = __fmaf_rn(u.z, c.z, -__fmul_rn(w.z, d.z)); b.z = __fmaf_rn(w.z, c.z, __fmul_rn(u.z, d.z));
        a.w = __fmaf_rn(u.w, c.w, -__fmul_rn(w.w, d.w)); b.w = __fmaf_rn(w.w, c.w, __fmul_rn(u.w, d.w));
        if (t != 1.f) {
            a = make_float4(__fmul_rn(a.x, t), __fmul_rn(a.y, t), __fmul_rn(a.z, t), __fmul_rn(a.w, t));
            b = make_float4(__fmul_rn(b.x, t), __fmul_rn(b.y, t), __fmul_rn(b.z, t), __fmul_rn(b.w, t));
        }
        store4(dst + i, a);
        store4(dst + half + i, b);
    };
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    const int pairs = half >> 2, q_items = pairs + ((W - s.rotary_dim) >> 2);
    for (int e = tid; e < s.heads * s.maps * q_items; e += 256) {
        const int hm = e / q_items, j = e - hm * q_items, at = (hm % s.maps) * s.dim;        // (the map's place in its row of W values)
        T* dst = q_out + r * s.ld_q + (size_t)hm * W;
        if (j < pairs) {
            turn(staged, q_gain, inv[0], hm * s.dim, j * 4, temp, dst + at);
        } else {
            int p = (j - pairs) * 4;
            if (p >= at) p += s.rotary_dim;
            const int i = p - at;
            float4 v = zero;
            if (i >= 0 && i < s.dim) {
                v = gained4(load4(staged + hm * s.dim + i), inv[0], load4(q_gain + hm * s.dim + i));
                if (temp != 1.f) v = make_float4(__fmul_rn(v.x, temp), __fmul_rn(v.y, temp), __fmul_rn(v.z, temp), __fmul_rn(v.w, temp));
            }
            store4(dst + p, v);
        }
    }
    if (!write_kv || !jllm_in_bounds(slot, num_slots, BOUNDS_SLOT)) return;
    const size_t page = slot / s.page_size, off = slot % s.page_size;
    const float* keys = staged + q_cols;
    const int kv_items = s.maps * pairs + ((W - s.maps * s.rotary_dim) >> 2), plain = s.dim - s.rotary_dim;
    for (int e = tid; e < s.kv_heads * kv_items; e += 256) {
        const int g = e / kv_items, j = e - g * kv_items;
        T* dst = k_cache + ((page * s.kv_heads + g) * s.page_size + off) * W;
        if (j < s.maps * pairs) {
            const int m = j / pairs;
            turn(keys, k_gain, inv[1], (g * s.maps + m) * s.dim, (j - m * pairs) * 4, 1.f, dst + m * s.dim);
        } else {
            const int p = (j - s.maps * pairs) * 4, m = plain > 0 ? p / plain : s.maps;
            if (m < s.maps) {
                const int i = s.rotary_dim + p - m * plain, col = (g * s.maps + m) * s.dim + i;
                store4(dst + m * s.dim + i, gained4(load4(keys + col), inv[1], load4(k_gain + col)));
            } else {
                store4(dst + s.maps * s.rotary_dim + p, zero);
            }
        }
    }
    const bool own = s.v_off == s.k_off;                   // the values are the keys as projected
    for (int e = tid * 4; e < s.kv_heads * W; e += 1024) {
        const int g = e / W, cc = e - g * W;
        const float4 v = cc >= s.vdim ? zero : own ? load4(keys + g * s.vdim + cc) : load4(row + s.v_off + (size_t)g * s.vdim + cc);
        store4(v_cache + ((page * s.kv_heads + g) * s.page_size + off) * W + cc, v);
    }
}

// One warp per (row, head); V values a lane at a time.
template <typename T, int V>
__global__ void __launch_bounds__(256)
map_difference_kernel(const T* __restrict__ att, int ld, int width, float lambda, float eps, float out_scale, T* __restrict__ y, int ld_y,
                      int rows, int heads, int vdim) {
    pdl_wait();
    pdl_trigger();
    const int w = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (w >= rows * heads) return;
    const int r = w / heads, h = w - r * heads;
    const T* a = att + (size_t)r * ld + (size_t)(2 * h) * width;
    const T* b = a + width;
    auto diff = [&](int i, float (&o)[V]) {
        float u[V], v[V];
        if constexpr (V == 4 && sizeof(T) == 2) {
            const uint2 ra = *reinterpret_cast<const uint2*>(a + i), rb = *reinterpret_cast<const uint2*>(b + i);
            const T *ea = reinterpret_cast<const T*>(&ra), *eb = reinterpret_cast<const T*>(&rb);
#pragma unroll
            for (int k = 0; k < V; ++k) { u[k] = to_float(ea[k]); v[k] = to_float(eb[k]); }
        } else {
#pragma unroll
            for (int k = 0; k < V; ++k) { u[k] = to_float(a[i + k]); v[k] = to_float(b[i + k]); }
        }
#pragma unroll
        for (int k = 0; k < V; ++k) o[k] = u[k] - __fmul_rn(lambda, v[k]);
    };
    float ss = 0.f;
    for (int i = lane * V; i < vdim; i += 32 * V) {
        float o[V];
        diff(i, o);
#pragma unroll
        for (int k = 0; k < V; ++k) ss = fmaf(o[k], o[k], ss);
    }
    ss = warp_sum(ss);
    const float inv = 1.f / sqrtf(ss / (float)vdim + eps);
    T* dst = y + (size_t)r * ld_y + (size_t)h * vdim;
    for (int i = lane * V; i < vdim; i += 32 * V) {
        float o[V];
        diff(i, o);
#pragma unroll
        for (int k = 0; k < V; ++k) o[k] = __fmul_rn(__fmul_rn(o[k], inv), out_scale);
        if constexpr (V == 4 && sizeof(T) == 2) {
            uint2 raw;
            T* e = reinterpret_cast<T*>(&raw);
#pragma unroll
            for (int k = 0; k < V; ++k) e[k] = from_float<T>(o[k]);
            *reinterpret_cast<uint2*>(dst + i) = raw;
        } else {
#pragma unroll
            for (int k = 0; k < V; ++k) dst[i + k] = from_float<T>(o[k]);
        }
    }
}

}  // namespace

JLLM_BOUNDS_READER(attention_maps)

// src [rows, ld] of type `dtype`: queries (heads x maps x dim) from column 0, keys (kv_heads x maps x dim) at k_off, values
// (kv_heads x vdim) at v_off; q_gain / k_gain float32 [their columns] or null (no norm); q_out [rows, ld_q]; caches [pages, kv_heads,
// page_size, width]. write_kv 0: queries only.
JLLM_EXPORT int jllm_map_prepare(const void* src, int dtype, int ld, int k_off, int v_off, const float* q_gain, const float* k_gain,
                                 float eps, const float* cos_t, const float* sin_t, int rotary_dim, int pairing, const int* positions,
                                 const int* slots, void* q_out, int ld_q, void* k_cache, void* v_cache, int write_kv, int rows,
                                 int heads, int kv_heads, int maps, int dim, int vdim, int width, int page_size,
                                 int temp_every, float temp_coef, cudaStream_t stream) {
    JLLM_REQUIRE(rows >= 0 && heads > 0 && kv_heads > 0 && maps > 0 && dim > 0 && vdim > 0, "map_prepare: rows=%d heads=%d/%d maps=%d dim=%d/%d",
                 rows, heads, kv_heads, maps, dim, vdim);
    JLLM_REQUIRE(width >= maps * dim && width >= vdim && ld_q >= heads * maps * width, "map_prepare: width=%d for %d maps of %d and values of %d",
                 width, maps, dim, vdim);
    JLLM_REQUIRE(rotary_dim >= 0 && rotary_dim <= dim && rotary_dim % 2 == 0, "map_prepare: rotary_dim=%d dim=%d", rotary_dim, dim);
    if (rows == 0) return JLLM_OK;
    const MapShape s{heads, kv_heads, maps, dim, vdim, width, page_size, rotary_dim, pairing, ld, k_off, v_off, ld_q, temp_every, temp_coef};
    const int num_slots = jllm_pool_pages() * page_size;
    const int per = dtype == JLLM_F32 ? 4 : 8;
    auto whole = [&](long long n) { return n % per == 0; };
    const bool vec = whole(dim) && whole(vdim) && whole(width) && whole(ld) && whole(k_off) && whole(v_off) && whole(ld_q) &&
                     whole(rotary_dim) && whole(rotary_dim / 2) &&
                     (((uintptr_t)src | (uintptr_t)q_out | (uintptr_t)k_cache | (uintptr_t)v_cache) % 16) == 0;
    const size_t staged_bytes = ((size_t)heads * maps * dim + (size_t)kv_heads * maps * dim) * sizeof(float);
    const bool gains_whole = (((uintptr_t)q_gain | (uintptr_t)k_gain | (uintptr_t)cos_t | (uintptr_t)sin_t) % 16) == 0;
    if (vec && gains_whole && q_gain != nullptr && (k_gain != nullptr || !write_kv) && staged_bytes <= 46 * 1024 &&
        (pairing == 0 || rotary_dim == 0)) {
#define JLLM_MAP_NORMED(T)                                                                                                       \
    jllm_launch(map_prepare_normed_kernel<T>, dim3(rows), dim3(256), staged_bytes, stream, LAUNCH_DEPENDENT, (const T*)src, s, q_gain, k_gain, \
                eps, cos_t, sin_t, positions, slots, (T*)q_out, (T*)k_cache, (T*)v_cache, write_kv, num_slots)
        if (dtype == JLLM_F32) JLLM_MAP_NORMED(float);
        else JLLM_MAP_NORMED(__nv_bfloat16);
#undef JLLM_MAP_NORMED
        return jllm_check_launch("map_prepare");
    }
#define JLLM_MAP_PREPARE(T, N)                                                                                                 \
    jllm_launch(map_prepare_kernel<T, N>, dim3(rows), dim3(256), 0, stream, LAUNCH_DEPENDENT, (const T*)src, s, q_gain, k_gain, eps, cos_t, \
                sin_t, positions, slots, (T*)q_out, (T*)k_cache, (T*)v_cache, write_kv, num_slots)
    if (dtype == JLLM_F32) {
        if (vec) JLLM_MAP_PREPARE(float, 4);
        else JLLM_MAP_PREPARE(float, 1);
    } else {
        if (vec) JLLM_MAP_PREPARE(__nv_bfloat16, 8);
        else JLLM_MAP_PREPARE(__nv_bfloat16, 1);
    }
#undef JLLM_MAP_PREPARE
    return jllm_check_launch("map_prepare");
}

// att [rows, ld] of type `dtype`: query head h's two maps at columns 2 h width and (2 h + 1) width, vdim values each; y [rows, ld_y]
// with head h at h * vdim.
JLLM_EXPORT int jllm_map_difference(const void* att, int dtype, int ld, int width, float lambda, float eps, float out_scale, void* y,
                                    int ld_y, int rows, int heads, int vdim, cudaStream_t stream) {
    JLLM_REQUIRE(rows >= 0 && heads > 0 && vdim > 0 && width >= vdim && ld >= 2 * heads * width && ld_y >= heads * vdim,
                 "map_difference: rows=%d heads=%d vdim=%d width=%d", rows, heads, vdim, width);
    if (rows == 0) return JLLM_OK;
    const dim3 grid(((long long)rows * heads + 7) / 8);
    const bool vec = vdim % 4 == 0 && width % 4 == 0 && ld % 4 == 0 && ld_y % 4 == 0 && (((uintptr_t)att | (uintptr_t)y) % 16) == 0;
#define JLLM_MAP_DIFF(T, V)                                                                                                    \
    jllm_launch(map_difference_kernel<T, V>, grid, dim3(256), 0, stream, LAUNCH_DEPENDENT, (const T*)att, ld, width, lambda, eps,    \
                out_scale, (T*)y, ld_y, rows, heads, vdim)
    if (dtype == JLLM_F32) JLLM_MAP_DIFF(float, 1);
    else if (vec) JLLM_MAP_DIFF(__nv_bfloat16, 4);
    else JLLM_MAP_DIFF(__nv_bfloat16, 1);
#undef JLLM_MAP_DIFF
    return jllm_check_launch("map_difference");
}
