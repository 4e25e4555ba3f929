// A residual stream held several times ("hyper-connections"), and the norm that computes no statistics.
//
//   bfi_dynamic_tanh:  h[r, :] = tanh(alpha * u) * w + b,   u = x[rows[r], :]                          (streams 1)
//                                                           u = sum_a read[a] * X[rows[r], a, :]       (streams > 1)
//                      read null: the plain sum.  With `u_out` the sum itself is written too (float32).
//   bfi_stream_mix:    one sublayer's output into the copies, all copies from the old ones:
//                      y = scale * (c0 * y0 + c1 * y1)                        (y1 and scale may be absent)
//                      X[t, b, :] = sum_a mix[a, b] * X[t, a, :] + write[b] * y
//                      and, when asked, what the next sublayer reads, out of the copies just made: the weighted sum
//                      u (float32) and / or its dynamic tanh h in the activation type.
//
// X is float32 [tokens][streams][width] in every run dtype, y0 and y1 are float32; read, write, mix
// ([from][to]) and alpha are float32; scale, w and b float32 or bfloat16.  Everything is elementwise in
// the channel, so a thread owns 4 channels (or 1, where rows do not cut into 16-byte pieces) of one
// token: it reads each copy once, writes it once, and the next sublayer's input costs no further read.
#include "common.cuh"

#define ST_MAX_STREAMS 32

struct DynTanh {
    const float* alpha;       // null: no norm
    const void *w, *b;
    int w_dtype, b_dtype;
    void* h;
    int h_dtype;
    long h_stride;
};

template <int W>
struct StVec {
    float v[W];
};
template <int W>
__device__ __forceinline__ StVec<W> st_load(const float* p) {
    StVec<W> r;
    if (W == 4) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        r.v[0] = x.x, r.v[1 % W] = x.y, r.v[2 % W] = x.z, r.v[3 % W] = x.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int W>
__device__ __forceinline__ void st_store(float* p, const StVec<W>& r) {
    if (W == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1 % W], r.v[2 % W], r.v[3 % W]);
    else *p = r.v[0];
}
// a weight vector of either storage type
template <int W>
__device__ __forceinline__ StVec<W> st_load_any(const void* p, int dtype, size_t i) {
    StVec<W> r;
    if (W == 4 && dtype == BFI_BF16) {
        const uint2 raw = *reinterpret_cast<const uint2*>(reinterpret_cast<const bf16*>(p) + i);
        const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
        const float2 a = __bfloat1622float2(h2[0]), b = __bfloat1622float2(h2[1]);
        r.v[0] = a.x, r.v[1 % W] = a.y, r.v[2 % W] = b.x, r.v[3 % W] = b.y;
        return r;
    }
    if (dtype == BFI_F32) return st_load<W>(reinterpret_cast<const float*>(p) + i);
    r.v[0] = load_as_f32(p, dtype, i);
    return r;
}
template <int W>
__device__ __forceinline__ void st_store_any(void* p, int dtype, size_t i, const StVec<W>& r) {
    if (W == 4 && dtype == BFI_BF16) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(r.v[0], r.v[1 % W]), hi = __floats2bfloat162_rn(r.v[2 % W], r.v[3 % W]);
        uint2 packed;
        packed.x = *reinterpret_cast<const uint32_t*>(&lo);
        packed.y = *reinterpret_cast<const uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(reinterpret_cast<bf16*>(p) + i) = packed;
    } else if (dtype == BFI_F32) {
        st_store<W>(reinterpret_cast<float*>(p) + i, r);
    } else {
        store_from_f32(p, dtype, i, r.v[0]);
    }
}

// The norm of one piece: the weights were fetched before the wait for the kernel before this one.
template <int W>
struct StNormPiece {
    StVec<W> w, b;
    float alpha;
    __device__ __forceinline__ void fetch(const DynTanh& n, int c) {
        if (n.alpha == nullptr) return;
        alpha = *n.alpha;
        w = st_load_any<W>(n.w, n.w_dtype, c);
        b = st_load_any<W>(n.b, n.b_dtype, c);
    }
    __device__ __forceinline__ void put(const DynTanh& n, size_t row, int c, const StVec<W>& u) const {
        if (n.alpha == nullptr) return;
        StVec<W> r;
#pragma unroll
        for (int k = 0; k < W; ++k) r.v[k] = fmaf(tanhf(alpha * u.v[k]), w.v[k], b.v[k]);
        st_store_any<W>(n.h, n.h_dtype, row * n.h_stride + c, r);
    }
};

// S: the number of copies where it is known at compile time (0: any, up to ST_MAX_STREAMS)
template <int S, int W>
__global__ void __launch_bounds__(128)
dynamic_tanh_kernel(const float* __restrict__ x, long x_stride, const int* __restrict__ rows, int s_any,
                    const float* __restrict__ read, int width, const DynTanh n, float* __restrict__ u_out, long u_stride) {
    pdl_trigger();
    const int s = S ? S : s_any;
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * W;
    if (c >= width) return;
    const size_t r = blockIdx.x;
    const size_t src = rows ? (size_t)rows[r] : r;
    StNormPiece<W> piece;
    piece.fetch(n, c);
    pdl_wait();
    StVec<W> u;
    const float* xr = x + src * x_stride + c;
    if (s == 1 && read == nullptr) {
        u = st_load<W>(xr);
    } else {
#pragma unroll
        for (int k = 0; k < W; ++k) u.v[k] = 0.0f;
#pragma unroll
        for (int a = 0; a < (S ? S : ST_MAX_STREAMS); ++a) {
            if (!S && a >= s) break;
            const StVec<W> v = st_load<W>(xr + (size_t)a * width);
            const float f = read ? read[a] : 1.0f;
#pragma unroll
            for (int k = 0; k < W; ++k) u.v[k] = fmaf(f, v.v[k], u.v[k]);
        }
    }
    if (u_out) st_store<W>(u_out + r * u_stride + c, u);
    piece.put(n, r, c, u);
}

struct StreamMix {
    const float *mix, *write, *read;      // [s][s] as [from][to], [s], [s] (read null: nothing is made for the next sublayer)
    const float *y0, *y1;
    long y0_stride, y1_stride;
    float c0, c1;
    const void* scale;                    // null: 1
    int scale_dtype;
    float* u_out;
    long u_stride;
};

template <int S, int W>
__global__ void __launch_bounds__(128)
stream_mix_kernel(float* __restrict__ x, long x_stride, int s_any, int width, const StreamMix m, const DynTanh n) {
    pdl_trigger();
    const int s = S ? S : s_any;
    constexpr int CAP = S ? S : ST_MAX_STREAMS;
    __shared__ float coef[CAP * CAP + 2 * CAP];          // mix, write, read
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * W;
    for (int i = threadIdx.x; i < s * s + 2 * s; i += blockDim.x)
        coef[i] = i < s * s ? m.mix[i] : (i < s * s + s ? m.write[i - s * s] : (m.read ? m.read[i - s * s - s] : 0.0f));
    const bool ok = c < width;
    StNormPiece<W> piece;
    StVec<W> sc;
#pragma unroll
    for (int k = 0; k < W; ++k) sc.v[k] = 1.0f;
    if (ok) {
        piece.fetch(n, c);
        if (m.scale) sc = st_load_any<W>(m.scale, m.scale_dtype, c);
    }
    __syncthreads();
    pdl_wait();
    if (!ok) return;
    const size_t t = blockIdx.x;
    float* xr = x + t * x_stride + c;
    StVec<W> in[CAP], y = st_load<W>(m.y0 + t * m.y0_stride + c);
#pragma unroll
    for (int a = 0; a < CAP; ++a) {
        if (!S && a >= s) break;
        in[a] = st_load<W>(xr + (size_t)a * width);
    }
    if (m.y1) {
        const StVec<W> y1 = st_load<W>(m.y1 + t * m.y1_stride + c);
#pragma unroll
        for (int k = 0; k < W; ++k) y.v[k] = m.c0 * y.v[k] + m.c1 * y1.v[k];
    } else if (m.c0 != 1.0f) {
#pragma unroll
        for (int k = 0; k < W; ++k) y.v[k] *= m.c0;
    }
    StVec<W> u;
#pragma unroll
    for (int k = 0; k < W; ++k) y.v[k] *= sc.v[k], u.v[k] = 0.0f;
#pragma unroll
    for (int b = 0; b < CAP; ++b) {
        if (!S && b >= s) break;
        StVec<W> o;
        const float wr = coef[s * s + b], rd = coef[s * s + s + b];
#pragma unroll
        for (int k = 0; k < W; ++k) o.v[k] = wr * y.v[k];
#pragma unroll
        for (int a = 0; a < CAP; ++a) {
            if (!S && a >= s) break;
            const float f = coef[a * s + b];
#pragma unroll
            for (int k = 0; k < W; ++k) o.v[k] = fmaf(f, in[a].v[k], o.v[k]);
        }
        st_store<W>(xr + (size_t)b * width, o);
#pragma unroll
        for (int k = 0; k < W; ++k) u.v[k] = fmaf(rd, o.v[k], u.v[k]);
    }
    if (m.read == nullptr) return;
    if (m.u_out) st_store<W>(m.u_out + t * m.u_stride + c, u);
    piece.put(n, t, c, u);
}

static bool st_aligned(const void* p, long stride, int dtype) {
    return p == nullptr || (((uintptr_t)p & (dtype == BFI_F32 ? 15 : 7)) == 0 && stride % 4 == 0);
}

#define BFI_STREAM_CASES(LAUNCH, W)              \
    switch (streams) {                           \
        case 1: LAUNCH(1, W); break;             \
        case 2: LAUNCH(2, W); break;             \
        case 3: LAUNCH(3, W); break;             \
        case 4: LAUNCH(4, W); break;             \
        case 8: LAUNCH(8, W); break;             \
        default: LAUNCH(0, W); break;            \
    }

extern "C" int bfi_dynamic_tanh(const float* x, long x_stride, const int* rows, int streams, const float* read, int n_rows, int width,
                                const float* alpha, const void* w, int w_dtype, const void* b, int b_dtype, void* h, int h_dtype,
                                long h_stride, float* u_out, long u_stride, cudaStream_t stream) {
    BFI_REQUIRE(n_rows >= 0 && width > 0 && streams >= 1 && streams <= ST_MAX_STREAMS, "dynamic_tanh: bad sizes rows=%d width=%d streams=%d (at most %d)",
                n_rows, width, streams, ST_MAX_STREAMS);
    BFI_REQUIRE(dtype_ok(w_dtype) && dtype_ok(b_dtype) && dtype_ok(h_dtype), "dynamic_tanh: unknown dtype code");
    BFI_REQUIRE(x_stride >= (long)streams * width, "dynamic_tanh: row stride shorter than the row");
    BFI_REQUIRE(alpha == nullptr || (w != nullptr && b != nullptr && h != nullptr && h_stride >= width), "dynamic_tanh: the norm needs its weight, bias and an output");
    BFI_REQUIRE(u_out == nullptr || u_stride >= width, "dynamic_tanh: the sum's row stride is shorter than the row");
    if (n_rows == 0) return 0;
    const DynTanh n = {alpha, w, b, w_dtype, b_dtype, h, h_dtype, h_stride};
    const bool vec = width % 4 == 0 && st_aligned(x, x_stride, BFI_F32) && st_aligned(w, 4, w_dtype) && st_aligned(b, 4, b_dtype) &&
                     st_aligned(h, h_stride, h_dtype) && st_aligned(u_out, u_stride, BFI_F32);
    const int pieces = vec ? width / 4 : width;
    const dim3 grid(n_rows, (pieces + 127) / 128);
    BFI_REQUIRE(grid.y <= 65535, "dynamic_tanh: rows of %d values are too long", width);
#define BFI_DT(SS, WW) bfi_launch(dynamic_tanh_kernel<SS, WW>, grid, dim3(128), 0, stream, x, x_stride, rows, streams, read, width, n, u_out, u_stride)
    if (vec) { BFI_STREAM_CASES(BFI_DT, 4) } else { BFI_STREAM_CASES(BFI_DT, 1) }
#undef BFI_DT
    return bfi_check_launch("dynamic_tanh");
}

extern "C" int bfi_stream_mix(float* x, long x_stride, int streams, int n_rows, int width, const float* y0, long y0_stride, float c0,
                              const float* y1, long y1_stride, float c1, const void* scale, int scale_dtype, const float* mix,
                              const float* write, const float* read, const float* alpha, const void* w, int w_dtype, const void* b,
                              int b_dtype, void* h, int h_dtype, long h_stride, float* u_out, long u_stride, cudaStream_t stream) {
    BFI_REQUIRE(n_rows >= 0 && width > 0 && streams >= 1 && streams <= ST_MAX_STREAMS, "stream_mix: bad sizes rows=%d width=%d streams=%d (at most %d)",
                n_rows, width, streams, ST_MAX_STREAMS);
    BFI_REQUIRE(dtype_ok(scale_dtype) && dtype_ok(w_dtype) && dtype_ok(b_dtype) && dtype_ok(h_dtype), "stream_mix: unknown dtype code");
    BFI_REQUIRE(x_stride >= (long)streams * width && y0_stride >= width && (y1 == nullptr || y1_stride >= width), "stream_mix: row stride shorter than the row");
    BFI_REQUIRE(mix != nullptr && write != nullptr && y0 != nullptr, "stream_mix: the matrix, the output weights and the sublayer's output are required");
    BFI_REQUIRE(alpha == nullptr || (read != nullptr && w != nullptr && b != nullptr && h != nullptr && h_stride >= width),
                "stream_mix: the next norm needs its input weights, weight, bias and an output");
    BFI_REQUIRE(u_out == nullptr || (read != nullptr && u_stride >= width), "stream_mix: the next sublayer's sum needs its input weights");
    if (n_rows == 0) return 0;
    const DynTanh n = {alpha, w, b, w_dtype, b_dtype, h, h_dtype, h_stride};
    const StreamMix m = {mix, write, read, y0, y1, y0_stride, y1_stride, c0, c1, scale, scale_dtype, u_out, u_stride};
    const bool vec = width % 4 == 0 && st_aligned(x, x_stride, BFI_F32) && st_aligned(y0, y0_stride, BFI_F32) && st_aligned(y1, y1_stride, BFI_F32) &&
                     st_aligned(scale, 4, scale_dtype) && st_aligned(w, 4, w_dtype) && st_aligned(b, 4, b_dtype) && st_aligned(h, h_stride, h_dtype) &&
                     st_aligned(u_out, u_stride, BFI_F32);
    const int pieces = vec ? width / 4 : width;
    const dim3 grid(n_rows, (pieces + 127) / 128);
    BFI_REQUIRE(grid.y <= 65535, "stream_mix: rows of %d values are too long", width);
#define BFI_SM(SS, WW) bfi_launch(stream_mix_kernel<SS, WW>, grid, dim3(128), 0, stream, x, x_stride, streams, width, m, n)
    if (vec) { BFI_STREAM_CASES(BFI_SM, 4) } else { BFI_STREAM_CASES(BFI_SM, 1) }
#undef BFI_SM
    return bfi_check_launch("stream_mix");
}

BFI_TRACE_EXPORT(streams)
