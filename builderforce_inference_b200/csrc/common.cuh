// Shared helpers of the sm_100a kernel library: storage types, conversions, reductions and the
// error convention of the exported C functions.
//
// Every exported function returns 0 on success.  On failure it returns a non-zero code and
// leaves a message that bfi_last_error() hands out; nothing is launched in that case.
// Storage types are named by code: 0 = float32, 1 = bfloat16.  Arithmetic is float32 everywhere.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <cstdarg>
#include <cstdio>

#define BFI_F32 0
#define BFI_BF16 1

#define BFI_PAGE_TOKENS 64

// status word bits (device side checks record and skip; they never trap)
#define BFI_STATUS_BAD_TOKEN 1
#define BFI_STATUS_NO_PAGE 2
#define BFI_STATUS_BAD_POSITION 4

typedef __nv_bfloat16 bf16;

extern "C" const char* bfi_last_error();
int bfi_fail(const char* fmt, ...);
int bfi_check_launch(const char* what);
int bfi_sm_count();

// Programmatic dependent launch.  When enabled, every kernel is launched with the attribute that
// lets it start while its predecessor in the stream drains.  A kernel may touch nothing but
// constant weights before pdl_wait(), which returns once the predecessor has completed and its
// writes are visible; without the attribute the instruction returns at once.
extern int g_bfi_pdl;

#ifdef BFI_TRACE
// Timeline of a step, for builds made with -DBFI_TRACE (environment variable BFI_B200_TRACE=1): the
// first thread of every block stamps the global timer when the block starts (0), when its wait for
// the kernel before it returns (1) and, in the kernels that say so, when it is done (2).  Records
// are {grid id << 32 | what << 28 | linear block id, nanoseconds}; every source file has a buffer of
// its own (BFI_TRACE_EXPORT at its end gives it a reader).
#define BFI_TRACE_RECORDS (1 << 18)
static __device__ unsigned long long g_bfi_trace[2 + 2 * BFI_TRACE_RECORDS];
__device__ __forceinline__ void bfi_trace(unsigned what) {
    if (threadIdx.x == 0 && threadIdx.y == 0 && threadIdx.z == 0) {
        unsigned long long now, gid;
        asm volatile("mov.u64 %0, %%globaltimer;" : "=l"(now));
        asm volatile("mov.u64 %0, %%gridid;" : "=l"(gid));
        const unsigned long long i = atomicAdd(&g_bfi_trace[0], 1ull);
        if (i < BFI_TRACE_RECORDS) {
            const unsigned long long blk = blockIdx.x + (unsigned long long)gridDim.x * (blockIdx.y + (unsigned long long)gridDim.y * blockIdx.z);
            g_bfi_trace[2 + 2 * i] = (gid << 32) | ((unsigned long long)what << 28) | (blk & 0xFFFFFFFull);
            g_bfi_trace[3 + 2 * i] = now;
        }
    }
}
#define BFI_TRACE_END() bfi_trace(2)
#define BFI_TRACE_EXPORT(name)                                                                                   \
    extern "C" long bfi_trace_read_##name(unsigned long long* host, long cap) {                                  \
        unsigned long long head[2] = {0, 0};                                                                     \
        cudaDeviceSynchronize();                                                                                 \
        cudaMemcpyFromSymbol(head, g_bfi_trace, sizeof(head));                                                   \
        long n = (long)(head[0] < BFI_TRACE_RECORDS ? head[0] : BFI_TRACE_RECORDS);                              \
        if (n > cap) n = cap;                                                                                    \
        if (n > 0) cudaMemcpyFromSymbol(host, g_bfi_trace, (size_t)n * 16, 16);                                  \
        head[0] = 0;                                                                                             \
        cudaMemcpyToSymbol(g_bfi_trace, head, sizeof(head));                                                     \
        return n;                                                                                                \
    }
#else
#define BFI_TRACE_END()
#define BFI_TRACE_EXPORT(name)
#endif

__device__ __forceinline__ void pdl_wait() {
    asm volatile("griddepcontrol.wait;" ::: "memory");
#ifdef BFI_TRACE
    bfi_trace(1);
#endif
}
__device__ __forceinline__ void pdl_trigger() {
#ifdef BFI_TRACE
    bfi_trace(0);
#endif
    asm volatile("griddepcontrol.launch_dependents;");
}

template <typename... KArgs, typename... Args>
static inline cudaError_t bfi_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                                     cudaStream_t stream, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = g_bfi_pdl ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...);
}

#define BFI_REQUIRE(cond, ...)                  \
    do {                                        \
        if (!(cond)) return bfi_fail(__VA_ARGS__); \
    } while (0)

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }

template <typename T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

// Loads a value of storage type `dtype` (runtime code) at element index i.
__device__ __forceinline__ float load_as_f32(const void* p, int dtype, size_t i) {
    return dtype == BFI_F32 ? reinterpret_cast<const float*>(p)[i]
                            : __bfloat162float(reinterpret_cast<const bf16*>(p)[i]);
}
__device__ __forceinline__ void store_from_f32(void* p, int dtype, size_t i, float v) {
    if (dtype == BFI_F32)
        reinterpret_cast<float*>(p)[i] = v;
    else
        reinterpret_cast<bf16*>(p)[i] = __float2bfloat16_rn(v);
}

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

// Sum over a block of up to 1024 threads; every thread gets the result.  `scratch` holds 33 floats.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int n_warps = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    if (warp == 0) {
        float t = lane < n_warps ? scratch[lane] : 0.0f;
        t = warp_sum(t);
        if (lane == 0) scratch[32] = t;
    }
    __syncthreads();
    return scratch[32];
}
__device__ __forceinline__ float block_max(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int n_warps = (blockDim.x + 31) >> 5;
    v = warp_max(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    if (warp == 0) {
        float t = lane < n_warps ? scratch[lane] : -INFINITY;
        t = warp_max(t);
        if (lane == 0) scratch[32] = t;
    }
    __syncthreads();
    return scratch[32];
}

// The gated activation of a feed-forward, as the matrix products' gated epilogue applies it to a
// (gate, up) pair.  Kind 0, the sigmoid family: with g' = min(g, limit) and u' = clamp(u, -limit, limit)
// (limit <= 0: no clamping)
//     g' * sigmoid(alpha * g') * (u' + shift)
// alpha 1, no limit and shift 0 is SiLU(gate) * up, and evaluates to the same bits as that formula.
// Kind 1, the tanh form of GELU:  0.5 g (1 + tanh(sqrt(2/pi) (g + 0.044715 g^3))) * u.
// With `in_scale` (float32, rows of `in_stride`) gate and up of row m and output column j are first
// multiplied by in_scale[m][j / in_cols]: a factor per row and group of columns on the product's input
// (an expert's weight, with the experts' columns side by side; a factor of 0 leaves 0 behind).
// A library holds ONE set of constants per host thread (bfi_set_gate), which every product launched
// from that thread with the gated epilogue takes along as a kernel argument.
#define BFI_GATE_SIGMOID 0
#define BFI_GATE_GELU_TANH 1
struct GateAct {
    float alpha, limit, shift;
    int kind;
    const float* in_scale;
    long in_stride;
    int in_cols;
};
extern thread_local GateAct g_bfi_gate;

__device__ __forceinline__ float gate_in_scale(const GateAct& a, int m, int j) {
    return a.in_scale[(size_t)m * a.in_stride + j / a.in_cols];
}

// The squared ReLU of a product that stores max(acc, 0)^2 (epilogue code 3 of the matrix products).
#define BFI_EPI_RELU_SQUARED 3
__device__ __forceinline__ float relu_squared(float v) {
    v = fmaxf(v, 0.0f);
    return v * v;
}

// 0.5 g (1 + tanh(y)) = g * sigmoid(2 y): one exponential, no cancellation for large |y|
__device__ __forceinline__ float gelu_tanh_exact(float g) {
    const float y = 0.7978845608028654f * (g + 0.044715f * g * g * g);
    float s;
    if (y >= 0.0f) {
        s = 1.0f / (1.0f + expf(-2.0f * y));
    } else {
        const float e = expf(2.0f * y);
        s = e / (1.0f + e);
    }
    return g * s;
}

__device__ __forceinline__ float gate_mul_exact(float g, float u, const GateAct a) {
    if (a.kind == BFI_GATE_GELU_TANH) return gelu_tanh_exact(g) * u;
    if (a.limit > 0.0f) {
        g = fminf(g, a.limit);
        u = fminf(fmaxf(u, -a.limit), a.limit);
    }
    const float z = a.alpha * g;
    float s;                       // overflow-safe two-branch sigmoid
    if (z >= 0.0f) {
        s = 1.0f / (1.0f + expf(-z));
    } else {
        const float e = expf(z);
        s = e / (1.0f + e);
    }
    return g * s * (u + a.shift);
}
__device__ __forceinline__ float gate_mul_fast(float g, float u, const GateAct a) {
    if (a.kind == BFI_GATE_GELU_TANH) {
        const float y = 0.7978845608028654f * (g + 0.044715f * g * g * g);
        return __fdividef(g, 1.0f + __expf(-2.0f * y)) * u;
    }
    if (a.limit > 0.0f) {
        g = fminf(g, a.limit);
        u = fminf(fmaxf(u, -a.limit), a.limit);
    }
    return __fdividef(g, 1.0f + __expf(-a.alpha * g)) * (u + a.shift);
}

// Soft-capped attention scores, cap * tanh(s / cap), as the bfloat16 attention kernels apply them to their
// float32 scores: these give the tanh, and the softmax's scale is then the cap (score_scale).  score_tanh holds
// for every score: tanh(x) = 1 - 2 / (1 + e^2x), an absolute error of a few float32 roundings of 1, so a score is
// right to about 1e-6 of the cap; e^2x overflowing to infinity gives 1, vanishing gives -1.  It costs two
// special-function operations.  score_tanh_near holds for scores within the cap, |x| <= 1, and costs none:
// tanh(x) = x P(x^2) with P the polynomial of degree 6 that is closest to tanh(sqrt u) / sqrt u on [0, 1]
// (relative error 5e-8, by the exchange algorithm).
struct ScoreCap {
    float in, in2, near_;      // scale / cap, 2 log2 e scale / cap, and the largest |q . k| that is near
};
static inline ScoreCap score_cap(float scale, float cap) {
    ScoreCap c = {0.0f, 0.0f, 0.0f};
    if (cap > 0.0f) c.in = scale / cap, c.in2 = 2.0f * 1.4426950408889634f * c.in, c.near_ = c.in > 0.0f ? 1.0f / c.in : 0.0f;
    return c;
}
// what the softmax multiplies q . k (or its tanh) by, in units of log2 e
static inline float score_scale(float scale, float cap) { return (cap > 0.0f ? cap : scale) * 1.4426950408889634f; }
__device__ __forceinline__ float score_tanh(float qk, const ScoreCap c) {
    float e, r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(c.in2 * qk));
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.0f + e));
    return fmaf(-2.0f, r, 1.0f);
}
// Four scores in place, step by step side by side: written out, so that no step waits for the one before it.
__device__ __forceinline__ void score_tanh_near(float* qk, const ScoreCap c) {
#define BFI_TANH_STEP(COEF)               \
    "fma.rn.f32 p0, p0, u0, " COEF ";\n"  \
    "fma.rn.f32 p1, p1, u1, " COEF ";\n"  \
    "fma.rn.f32 p2, p2, u2, " COEF ";\n"  \
    "fma.rn.f32 p3, p3, u3, " COEF ";\n"
    // coefficients from u^6 down: 1.0410226e-3, -6.2033790e-3, 2.0289980e-2, -5.3457030e-2, 0.13325204, -0.33332839, 0.99999995
    asm volatile("{\n.reg .f32 u0, u1, u2, u3, p0, p1, p2, p3;\n"
        "mul.rn.f32 %0, %0, %4;\nmul.rn.f32 %1, %1, %4;\nmul.rn.f32 %2, %2, %4;\nmul.rn.f32 %3, %3, %4;\n"
        "mul.rn.f32 u0, %0, %0;\nmul.rn.f32 u1, %1, %1;\nmul.rn.f32 u2, %2, %2;\nmul.rn.f32 u3, %3, %3;\n"
        "fma.rn.f32 p0, u0, 0f3A8872EC, 0fBBCB45B7;\nfma.rn.f32 p1, u1, 0f3A8872EC, 0fBBCB45B7;\nfma.rn.f32 p2, u2, 0f3A8872EC, 0fBBCB45B7;\nfma.rn.f32 p3, u3, 0f3A8872EC, 0fBBCB45B7;\n"
        BFI_TANH_STEP("0f3CA6372C") BFI_TANH_STEP("0fBD5AF5C3") BFI_TANH_STEP("0f3E087339") BFI_TANH_STEP("0fBEAAAA05") BFI_TANH_STEP("0f3F7FFFFF")
        "mul.rn.f32 %0, %0, p0;\nmul.rn.f32 %1, %1, p1;\nmul.rn.f32 %2, %2, p2;\nmul.rn.f32 %3, %3, p3;\n}"
        : "+f"(qk[0]), "+f"(qk[1]), "+f"(qk[2]), "+f"(qk[3])
        : "f"(c.in));
#undef BFI_TANH_STEP
}

static inline int dtype_size(int dtype) { return dtype == BFI_F32 ? 4 : 2; }
static inline bool dtype_ok(int dtype) { return dtype == BFI_F32 || dtype == BFI_BF16; }
