// Shared pieces of the sm_100a kernels: element types, error reporting, block reductions.
//
// Every exported launcher returns 0 on success and a non-zero code otherwise; the text of the
// last error of the calling thread is read with jllm_last_error(). Launchers never allocate:
// the caller passes inputs, outputs and (where a kernel needs it) scratch memory.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <cstdarg>
#include <cstdio>

#define JLLM_EXPORT extern "C" __attribute__((visibility("default")))

enum JllmDtype : int { JLLM_F32 = 0, JLLM_BF16 = 1 };

enum JllmError : int {
    JLLM_OK = 0,
    JLLM_BAD_ARGUMENT = 1,   // a size or option the kernels refuse
    JLLM_CUDA_ERROR = 2,     // a CUDA call failed
    JLLM_UNSUPPORTED = 3,    // a combination that is not built
};

int jllm_fail(int code, const char* fmt, ...);
int jllm_check_launch(const char* what);
int jllm_device_sm_count();      // SMs of the current device (asked once), 0 if unknown
int jllm_pool_pages();           // pages of the cache pool in use, as the host declared them (0 = unknown)

#define JLLM_REQUIRE(cond, ...)                                   \
    do {                                                          \
        if (!(cond)) return jllm_fail(JLLM_BAD_ARGUMENT, __VA_ARGS__); \
    } while (0)

// ---- bounds checks of what the kernels read through tables (a build with -DJLLM_CHECK_BOUNDS) --------------------
// The kernels follow page tables, slot lists and token ids that the host packed. In the ordinary build they trust
// them. In the checked build (a second library, chosen with JLLM_B200_CHECK_BOUNDS=1) every table index, page id,
// cache slot and token id is compared with its limit first; an access that would leave its array is SKIPPED (a key
// then counts as absent, a write is dropped) and the first such case is recorded in a word of this translation unit:
// {what, index, limit, how many}. Nothing traps and nothing hangs: the host reads the words after the step
// (`jllm_bounds_error_<file>`) and raises. A limit of 0 or less means "not known to this caller": only negative
// indices are caught then.
enum : int { BOUNDS_TABLE_INDEX = 1, BOUNDS_PAGE = 2, BOUNDS_SLOT = 3, BOUNDS_TOKEN = 4, BOUNDS_ROW = 5 };
#ifdef JLLM_CHECK_BOUNDS
constexpr bool kCheckBounds = true;
static __device__ int jllm_bounds_word[4];
__device__ __noinline__ static void jllm_bounds_record(int what, long long index, long long limit) {
    if (atomicAdd(&jllm_bounds_word[3], 1) == 0) {
        jllm_bounds_word[0] = what;
        jllm_bounds_word[1] = (int)max(-2147483647ll, min(2147483647ll, index));
        jllm_bounds_word[2] = (int)max(-2147483647ll, min(2147483647ll, limit));
    }
}
#define JLLM_BOUNDS_READER(file)                                                                   \
    JLLM_EXPORT int jllm_bounds_error_##file(int* out4) {                                          \
        int zero[4] = {0, 0, 0, 0};                                                                \
        if (cudaMemcpyFromSymbol(out4, jllm_bounds_word, sizeof(zero)) != cudaSuccess) return JLLM_CUDA_ERROR; \
        if (out4[3] && cudaMemcpyToSymbol(jllm_bounds_word, zero, sizeof(zero)) != cudaSuccess) return JLLM_CUDA_ERROR; \
        return JLLM_OK;                                                                            \
    }
#else
constexpr bool kCheckBounds = false;
#define JLLM_BOUNDS_READER(file)                                  \
    JLLM_EXPORT int jllm_bounds_error_##file(int* out4) {         \
        out4[0] = out4[1] = out4[2] = out4[3] = 0;                \
        return JLLM_OK;                                           \
    }
#endif

// True if `index` may be used; always true in the ordinary build (the check compiles to nothing).
__device__ __forceinline__ bool jllm_in_bounds(long long index, long long limit, int what) {
#ifdef JLLM_CHECK_BOUNDS
    if (index < 0 || (limit > 0 && index >= limit)) {
        jllm_bounds_record(what, index, limit);
        return false;
    }
#endif
    return true;
}

// The page of block `b` of a request's table; in the checked build -1 if the block lies outside the table's row or the
// page outside the pool (the caller then skips the access).
__device__ __forceinline__ long long jllm_page_of(const int* __restrict__ table, int b, int table_len, int num_pages) {
#ifdef JLLM_CHECK_BOUNDS
    if (!jllm_in_bounds(b, table_len, BOUNDS_TABLE_INDEX)) return -1;
    const int page = table[b];
    return jllm_in_bounds(page, num_pages, BOUNDS_PAGE) ? page : -1;
#else
    return table[b];
#endif
}

// ---- programmatic dependent launch ---------------------------------------------------------------------
// A decode step is a chain of some hundreds of short kernels. Launched the ordinary way each one starts
// only when its predecessor has drained, and its own ramp-up (block scheduling, first loads) is dead time.
// With programmatic dependent launch the next kernel's blocks become resident while the predecessor still
// runs: they may do work that does not depend on it (a matrix product fetches its first weights), then
// wait with pdl_wait() until the predecessor has completed and its writes are visible. Every kernel calls
// pdl_wait() before it reads anything a predecessor wrote or writes anything a predecessor may read, and
// only then pdl_trigger(), so at most one successor is resident early. Without the launch attribute both
// calls return at once.
//
// One thing limits this. An SM cannot change how its memory is split between shared memory and L1 while blocks
// are resident on it. A kernel whose blocks arrive while a predecessor with a large shared-memory allocation (the
// staged decode attention, the tcgen05 kernels) still holds the SM runs with that predecessor's split, that is
// with little L1, and so does every kernel that overlaps it in turn, until one launch waits for the SMs to drain.
// The row kernel of the decode products re-reads its activations through L1 (every block reads all of them) and
// runs at half its speed that way. A launch that says it wants L1 (LAUNCH_DEPENDENT_WANTS_L1) is therefore made
// plainly when a large-shared-memory kernel has been launched since the last plain launch.
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_trigger() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

// Weights are nobody's output: a kernel may ask for its own before it waits for its predecessor. `bytes` from `p` on, whole lines,
// asked of memory by the block's threads together.
__device__ __forceinline__ void prefetch_lines(const void* p, size_t bytes) {
    const char* c = static_cast<const char*>(p);
    for (size_t i = (size_t)threadIdx.x * 128; i < bytes; i += (size_t)blockDim.x * 128)
        asm volatile("prefetch.global.L2 [%0];" ::"l"(c + i));
}

bool jllm_pdl_enabled();
enum : int { LAUNCH_PLAIN = 0, LAUNCH_DEPENDENT = 1, LAUNCH_DEPENDENT_WANTS_L1 = 2 };
bool jllm_launch_overlaps(size_t dynamic_smem, int how);     // decides, and keeps the record the decision needs

template <typename... KArgs, typename... Args>
inline cudaError_t jllm_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                               int how, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = jllm_launch_overlaps(smem, how) ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}

// ---- element access: everything is computed in float -------------------------------------------------

__device__ __forceinline__ float to_float(float v) { return v; }
__device__ __forceinline__ float to_float(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T from_float(float v);
template <> __device__ __forceinline__ float from_float<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_float<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// ---- which keys a row sees ------------------------------------------------------------------------------
// Every attention kernel takes one number, `window`, for the span of keys a row at position P sees besides P itself:
//   0       every earlier key,
//   w > 0   the last w keys (a sliding window),
//   -c < 0  the keys of P's own chunk (position p lies in chunk p / c: a row never sees over a chunk's edge, whatever
//           portions its prompt is fed in).
// The first visible key does not decrease with P, which is what the tile kernels' edge tests rely on.
__host__ __device__ __forceinline__ int jllm_first_key(int P, int window) {
    return window > 0 ? (P + 1 - window > 0 ? P + 1 - window : 0) : (window < 0 ? P - P % (-window) : 0);
}

// With a window, a request's first `keep` keys may stay visible to every later row (`keep` 0: none): a row at P sees the
// keys [0, min(keep, first)) and [first, P]. The kernels that take this walk a row's visible keys by an index u that counts
// them in ascending order: u < kept is key u, u >= kept is key first + (u - kept), with kept = jllm_kept_keys(first, keep).
__host__ __device__ __forceinline__ int jllm_kept_keys(int first, int window, int keep) {
    return window > 0 && keep > 0 ? (keep < first ? keep : first) : 0;
}
__host__ __device__ __forceinline__ bool jllm_key_visible(int key, int P, int first, int keep) {
    return key <= P && (key >= first || key < keep);
}

// ---- the gate of a gated feed-forward: act(gate) * up -----------------------------------------------------
// `kind` is what the products' launchers take as their `swiglu` argument: 0 no gating, 1 silu (z / (1 + exp(-z))),
// 2 the tanh form of GELU, 0.5 z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))) = z / (1 + exp(-2 u)) with u the tanh's
// argument. `fast`: the tensor-core epilogues, whose result is rounded to bfloat16 anyway, use the fast exponential.
enum : int { GLU_NONE = 0, GLU_SILU = 1, GLU_GELU_TANH = 2 };
template <bool FAST>
__device__ __forceinline__ float glu_act(float z, int kind) {
    float t = z;
    if (kind == GLU_GELU_TANH) t = 1.5957691216057308f * __fmaf_rn(0.044715f * z, z * z, z);    // 2 sqrt(2 / pi) (z + c z^3)
    if constexpr (FAST) return __fdividef(z, 1.f + __expf(-t));
    return z / (1.f + expf(-t));
}

// The gated unit of a feed-forward from its two inputs. `word` is the products' `swiglu` argument: the activation's number
// (act(gate) * up), or, for the clamped unit, 3 in its two lowest bits and the float32 bits of the limit above them (the
// limit's own two lowest bits dropped): g sigmoid(1.702 g) (u + 1) with g = min(gate, limit), u = clamp(up, -limit, limit).
enum : int { GLU_SWISH_CLAMPED = 3 };
constexpr float kSwishAlpha = 1.702f;
template <bool FAST>
__device__ __forceinline__ float glu_unit(float gate, float up, int word) {
    if ((word & 3) == GLU_SWISH_CLAMPED) {
        const float limit = __int_as_float(word & ~3);
        const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
        const float t = kSwishAlpha * g;
        if constexpr (FAST) return __fdividef(g, 1.f + __expf(-t)) * (u + 1.f);
        return __fmul_rn(g / (1.f + expf(-t)), u + 1.f);
    }
    return __fmul_rn(glu_act<FAST>(gate, word), up);
}

// What a product's epilogue is told about the gated unit it applies: `word` as above (0: no gating). A mixture of experts whose
// units are stacked in one product says more: units from `split` on are another feed-forward's (a shared expert's) with a word of
// their own, and with `weights` ([rows, ld_w] float32) unit u's result is multiplied by weights[row, u / ff], a unit's from `split`
// on by weights[row, split / ff].
struct GluArgs {
    int word, word_behind, split, ff, ld_w;
    const float* weights;
    __host__ __device__ __forceinline__ explicit operator bool() const { return word != 0; }
    __device__ __forceinline__ int word_of(int unit) const { return unit < split ? word : word_behind; }
    __device__ __forceinline__ float weight(int row, int unit) const {
        return weights[(size_t)row * ld_w + min((unit < split ? unit : split) / ff, ld_w - 1)];
    }
    // whether eight units from a multiple of 8 on always share their word and their weight (the products' epilogues count on it)
    bool in_eights() const { return weights == nullptr && split == 0x7fffffff ? true : (ff & 7) == 0 && ((split & 7) == 0 || split == 0x7fffffff); }
    template <bool FAST>
    __device__ __forceinline__ float apply(float gate, float up, int row, int unit) const {
        const float y = glu_unit<FAST>(gate, up, word_of(unit));
        return weights != nullptr ? __fmul_rn(y, weight(row, unit)) : y;
    }
};
// ... from a launcher's two arguments: the word, and (or null) a host struct of what is said beyond it
struct GluMore {
    int word_behind, split, ff, ld_w;
    const float* weights;
};
inline GluArgs glu_args(int word, const void* more) {
    if (more == nullptr) return GluArgs{word, word, 0x7fffffff, 1, 0, nullptr};
    const GluMore& m = *static_cast<const GluMore*>(more);
    return GluArgs{word, m.split > 0 ? m.word_behind : word, m.split > 0 ? m.split : 0x7fffffff, m.ff > 0 ? m.ff : 1, m.ld_w, m.weights};
}

// ---- scores under a cap: c tanh(s / c) ------------------------------------------------------------------------
// tanh(x) = 1 - 2 / (e^(2x) + 1) by the special-function unit's exponential and reciprocal: within a few units of the seventh
// digit of 1 everywhere (an error in the SCORE of that times the cap), and exactly +-1 far out.
__device__ __forceinline__ float unit_tanh(float x) {
    float t;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(t) : "f"(x * 2.885390081777927f));      // 2 log2(e)
    return 1.f - __fdividef(2.f, t + 1.f);
}
// What the bfloat16 attention kernels are told: a raw dot product d becomes the base-2 score out * tanh(in * d) with in =
// scale / cap and out = cap * log2(e). out = 0: no cap. A prompt tile's scores go through `tile`: where none of a warp's values lies
// beyond the cap (|x| <= 1 for x = in * d, nearly always) tanh is an odd polynomial of degree 13, two values at a time on the
// multiply-add pipes (the special-function unit is what bounds these kernels' softmax); else `operator()`.
// The polynomial interpolates tanh(x) / x at the seven Chebyshev points of x^2 in [0, 1]: within 1.2e-7 in float32.
struct ScoreCap {
    float in, out;
    __host__ __device__ __forceinline__ explicit operator bool() const { return out != 0.f; }
    __device__ __forceinline__ float operator()(float d) const { return out * unit_tanh(in * d); }

    __device__ static __forceinline__ uint64_t both(float v) {
        uint64_t p;
        asm("mov.b64 %0, {%1, %1};" : "=l"(p) : "f"(v));
        return p;
    }
    // N x M raw products of a warp's threads, as the bits of floats; all threads of the warp call it
    template <int N, int M>
    __device__ __forceinline__ void tile(uint32_t (&v)[N][M]) const {
        float far[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int c = 0; c < N; ++c)
#pragma unroll
            for (int i = 0; i < M; ++i) far[i & 3] = fmaxf(far[i & 3], fabsf(__uint_as_float(v[c][i])));
        const float reach = fmaxf(fmaxf(far[0], far[1]), fmaxf(far[2], far[3])) * in;
        if (__all_sync(0xffffffffu, reach <= 1.f)) {
            const uint64_t c0 = both(out * 0.9999999403953552f), c1 = both(out * -0.3333282768726349f), c2 = both(out * 0.13325075805187225f),
                           c3 = both(out * -0.053451646119356155f), c4 = both(out * 0.02027970738708973f),
                           c5 = both(out * -0.0061943246982991695f), c6 = both(out * 0.0010380251333117485f), k = both(in);
#pragma unroll
            for (int c = 0; c < N; ++c)
#pragma unroll
                for (int i = 0; i < M; i += 2) {
                    uint64_t x, t, q;
                    asm("mov.b64 %0, {%1, %2};" : "=l"(x) : "r"(v[c][i]), "r"(v[c][i + 1]));
                    asm("mul.rn.f32x2 %0, %0, %1;" : "+l"(x) : "l"(k));
                    asm("mul.rn.f32x2 %0, %1, %1;" : "=l"(t) : "l"(x));
                    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(q) : "l"(c6), "l"(t), "l"(c5));
                    asm("fma.rn.f32x2 %0, %0, %1, %2;" : "+l"(q) : "l"(t), "l"(c4));
                    asm("fma.rn.f32x2 %0, %0, %1, %2;" : "+l"(q) : "l"(t), "l"(c3));
                    asm("fma.rn.f32x2 %0, %0, %1, %2;" : "+l"(q) : "l"(t), "l"(c2));
                    asm("fma.rn.f32x2 %0, %0, %1, %2;" : "+l"(q) : "l"(t), "l"(c1));
                    asm("fma.rn.f32x2 %0, %0, %1, %2;" : "+l"(q) : "l"(t), "l"(c0));
                    asm("mul.rn.f32x2 %0, %0, %1;" : "+l"(q) : "l"(x));
                    asm("mov.b64 {%0, %1}, %2;" : "=r"(v[c][i]), "=r"(v[c][i + 1]) : "l"(q));
                }
        } else {
#pragma unroll
            for (int c = 0; c < N; ++c)
#pragma unroll
                for (int i = 0; i < M; ++i) v[c][i] = __float_as_uint((*this)(__uint_as_float(v[c][i])));
        }
    }
};
inline ScoreCap score_cap(float cap, float scale) { return cap > 0.f ? ScoreCap{scale / cap, cap * 1.4426950408889634f} : ScoreCap{0.f, 0.f}; }

// N gated units whose activation is one word's, as a product's epilogue has them: the activation is chosen ONCE, in front of the loop
// (a choice per unit makes a chain of branches of it, and a thread's units wait for one another).
template <int N, typename Gate, typename Up>
__device__ __forceinline__ void glu_units(int word, Gate gate, Up up, float factor, float (&out)[N]) {
    if ((word & 3) == GLU_SWISH_CLAMPED) {
        const float limit = __int_as_float(word & ~3);
#pragma unroll
        for (int j = 0; j < N; ++j) {
            const float g = fminf(gate(j), limit), u = fminf(fmaxf(up(j), -limit), limit);
            out[j] = __fmul_rn(__fdividef(g, 1.f + __expf(-kSwishAlpha * g)) * (u + 1.f), factor);
        }
    } else if (word == GLU_GELU_TANH) {
#pragma unroll
        for (int j = 0; j < N; ++j) out[j] = __fmul_rn(__fmul_rn(glu_act<true>(gate(j), GLU_GELU_TANH), up(j)), factor);
    } else {
#pragma unroll
        for (int j = 0; j < N; ++j) out[j] = __fmul_rn(__fmul_rn(glu_act<true>(gate(j), GLU_SILU), up(j)), factor);
    }
}

// What a product does with its result, the launchers' `accumulate` argument: 0 store it, 1 add it to what `out` holds, 2
// store max(v, 0)^2 (the activation of an ungated feed-forward; behind the bias).
enum : int { EPI_STORE = 0, EPI_ADD = 1, EPI_RELU2 = 2 };
__device__ __forceinline__ float epilogue_act(float v, int how) {
    if (how != EPI_RELU2) return v;
    const float z = fmaxf(v, 0.f);
    return __fmul_rn(z, z);
}

// A vector (gain, bias) whose stored type is known only at run time.
struct VecRef {
    const void* p;
    int dtype;
    __device__ __forceinline__ float operator[](int i) const {
        return dtype == JLLM_F32 ? static_cast<const float*>(p)[i]
                                 : __bfloat162float(static_cast<const __nv_bfloat16*>(p)[i]);
    }
};

// ---- reductions with a fixed order: the result of a row never depends on what else is in the batch ----

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// Sum over a block of up to 1024 threads; every thread gets the result. `scratch` holds 33 floats.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    if (warp == 0) {
        float t = lane < warps ? scratch[lane] : 0.f;
        t = warp_sum(t);
        if (lane == 0) scratch[32] = t;
    }
    __syncthreads();
    return scratch[32];
}

__device__ __forceinline__ float block_max(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
    v = warp_max(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    if (warp == 0) {
        float t = lane < warps ? scratch[lane] : -INFINITY;
        t = warp_max(t);
        if (lane == 0) scratch[32] = t;
    }
    __syncthreads();
    return scratch[32];
}
