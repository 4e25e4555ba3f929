// The matrix memory (mlstm.cuh), the general kernels: any sizes, any step shape, float32 or bfloat16
// storage of the projections, float32 arithmetic and float32 state.
//
// bfi_mlstm_scan walks a sequence's new tokens in order; a block owns `vb` columns of one head of one
// sequence, thread (g, c) rows g, g + groups, ... of column c in shared memory.  The gates' logits come
// as float32 rows [tokens][2 * heads] (input gates, then forget gates).
//
// bfi_mlstm_step is for steps in which every sequence brings one token: a block owns 32 to 128 columns and
// keeps its part of the state in registers, asked for (with n, m and the gates' weight rows) before the wait
// for the kernel that makes q, k and v.  The gates' logits are made here, from the layer's input and the
// head's two weight rows, so a step needs no product of its own for them.  Everything a token needs is
// linear in the old state once the gates are known,
//     n_t . q = a (n . q) + b (k . q)          S_t^T q = a (S^T q) + b (k . q) v          a, b the two factors
// so all sums (both logits, n . q, k . q and the columns of S^T q) are taken in one pass with one barrier.
#include "mlstm.cuh"

template <typename T>
__global__ void mlstm_scan_kernel(const T* __restrict__ proj, long stride, int q_off, int k_off, int v_off,
                                  const float* __restrict__ gates, long gate_stride, const MemGates gp, float q_scale,
                                  float* __restrict__ out, long out_stride, float* __restrict__ state, float* __restrict__ tails,
                                  const int* __restrict__ cu_seqlens, const int* __restrict__ seq_slot, int H, int D, int V, int vb,
                                  int v_blocks) {
    pdl_trigger();
    extern __shared__ float sm[];
    float* S = sm;                     // [D][vb]
    float* n = S + (size_t)D * vb;     // [D]
    float* qs = n + D;                 // [D]
    float* ks = qs + D;                // [D]
    float* red = ks + D;               // [threads]
    __shared__ float scratch[33];
    __shared__ int last;
    const int seq = blockIdx.y;
    const int slot = seq_slot[seq];
    if (slot < 0) return;
    const int h = blockIdx.x / v_blocks;
    const int v0 = (blockIdx.x - h * v_blocks) * vb;
    const int t0 = cu_seqlens[seq], nt = cu_seqlens[seq + 1] - t0;
    const int c = threadIdx.x % vb, g = threadIdx.x / vb, ng = blockDim.x / vb;
    const bool col_ok = v0 + c < V;
    // the state earlier steps left (zero for a fresh slot) does not come from this step's kernels
    float* sp = state + (((size_t)slot * H + h) * D) * V + v0;
    float* tail = tails + ((size_t)slot * H + h) * (D + 2);
    for (int d = g; d < D; d += ng) S[d * vb + c] = col_ok ? sp[(size_t)d * V + c] : 0.0f;
    for (int d = threadIdx.x; d < D; d += blockDim.x) n[d] = tail[d];
    float m = tail[D];
    __syncthreads();
    if (threadIdx.x == 0) last = mem_last_reader(tail, D, v_blocks) ? 1 : 0;
    pdl_wait();
    for (int t = 0; t < nt; ++t) {
        const T* row = proj + (size_t)(t0 + t) * stride + (size_t)h * D;
        const float* gr = gates + (size_t)(t0 + t) * gate_stride;
        const float gi = mem_log_input(gp, gr[h], h), gf = mem_log_forget(gp, gr[H + h], h);
        const float m_new = fmaxf(gf + m, gi);
        const float keep = expf(gf + m - m_new), put = expf(gi - m_new);
        m = m_new;
        float nq = 0.0f;
        for (int d = threadIdx.x; d < D; d += blockDim.x) {
            const float qv = to_f32(row[q_off + d]) * q_scale, kv = put * to_f32(row[k_off + d]);
            qs[d] = qv;
            ks[d] = kv;
            n[d] = fmaf(keep, n[d], kv);
            nq = fmaf(n[d], qv, nq);
        }
        const float vv = col_ok ? to_f32(proj[(size_t)(t0 + t) * stride + v_off + (size_t)h * V + v0 + c]) : 0.0f;
        nq = block_sum(nq, scratch);                       // its barriers also publish q and k
        float acc = 0.0f;
        for (int d = g; d < D; d += ng) {
            const float s = fmaf(keep, S[d * vb + c], ks[d] * vv);
            S[d * vb + c] = s;
            acc = fmaf(s, qs[d], acc);
        }
        red[threadIdx.x] = acc;
        __syncthreads();
        if (threadIdx.x < vb && col_ok) {
            float o = 0.0f;
            for (int i = 0; i < ng; ++i) o += red[i * vb + threadIdx.x];
            out[(size_t)(t0 + t) * out_stride + (size_t)h * V + v0 + c] = o / mem_denominator(nq, m);
        }
    }
    if (col_ok)
        for (int d = g; d < D; d += ng) sp[(size_t)d * V + c] = S[d * vb + c];
    if (last && nt > 0) {
        for (int d = threadIdx.x; d < D; d += blockDim.x) tail[d] = n[d];
        if (threadIdx.x == 0) tail[D] = m;
    }
}

extern "C" int bfi_mlstm_scan(const void* proj, int dtype, long stride, int q_off, int k_off, int v_off, const float* gates,
                              long gate_stride, const float* bias_i, const float* bias_f, float cap, float q_scale, float* out,
                              long out_stride, float* state, float* tails, const int* cu_seqlens, const int* seq_slot, int n_seqs,
                              int H, int D, int V, cudaStream_t stream) {
    BFI_REQUIRE(dtype_ok(dtype), "mlstm_scan: unknown dtype code %d", dtype);
    BFI_REQUIRE(H > 0 && D > 0 && V > 0, "mlstm_scan: bad sizes heads=%d dim=%d vdim=%d", H, D, V);
    BFI_REQUIRE(cap > 0.0f, "mlstm_scan: the gates' cap must be positive");
    BFI_REQUIRE(out_stride >= (long)H * V && gate_stride >= 2L * H, "mlstm_scan: a row stride is shorter than the heads");
    if (n_seqs <= 0) return 0;
    int vb = V < 64 ? V : 64;
    auto bytes = [&](int cols, int threads) { return ((size_t)D * cols + 3 * (size_t)D + threads) * sizeof(float); };
    while (vb > 1 && bytes(vb, 256) > 200 * 1024) vb = (vb + 1) / 2;
    const int v_blocks = (V + vb - 1) / vb;
    int threads = vb * (256 / vb);
    if (threads < 32) threads = vb * ((32 + vb - 1) / vb);
    const size_t smem = bytes(vb, threads);
    BFI_REQUIRE(smem <= 200 * 1024, "mlstm_scan: a head of %d x %d does not fit shared memory", D, V);
    BFI_REQUIRE((long)H * v_blocks <= 2147483647L && n_seqs <= 65535, "mlstm_scan: too many heads or sequences for one launch");
    const MemGates gp = {bias_i, bias_f, cap};
    cudaError_t e = cudaSuccess;
#define BFI_MEM_SCAN(TT)                                                                                                         \
    do {                                                                                                                         \
        if (smem > 48 * 1024) e = cudaFuncSetAttribute(mlstm_scan_kernel<TT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        if (e == cudaSuccess)                                                                                                    \
            bfi_launch(mlstm_scan_kernel<TT>, dim3(H * v_blocks, n_seqs), dim3(threads), smem, stream, (const TT*)proj, stride, q_off, k_off, \
                       v_off, gates, gate_stride, gp, q_scale, out, out_stride, state, tails, cu_seqlens, seq_slot, H, D, V, vb, v_blocks); \
    } while (0)
    if (dtype == BFI_F32) BFI_MEM_SCAN(float);
    else BFI_MEM_SCAN(bf16);
#undef BFI_MEM_SCAN
    if (e != cudaSuccess) return bfi_fail("mlstm_scan: cannot reserve %zu bytes of shared memory: %s", smem, cudaGetErrorString(e));
    return bfi_check_launch("mlstm_scan");
}

// ------------------------------------------------------------------------------------------
// One new token per sequence
// ------------------------------------------------------------------------------------------
#define MEM_STEP_THREADS 256
#define MEM_STEP_MAX_D 256

// a row's part of the state: W neighbouring columns
template <int W>
struct MemCols {
    float v[W];
    __device__ __forceinline__ void zero() {
#pragma unroll
        for (int j = 0; j < W; ++j) v[j] = 0.0f;
    }
    __device__ __forceinline__ void load(const float* p) {
        if (W == 4) {
            const float4 x = *reinterpret_cast<const float4*>(p);
            v[0] = x.x, v[1 % W] = x.y, v[2 % W] = x.z, v[3 % W] = x.w;
        } else {
            v[0] = *p;
        }
    }
    __device__ __forceinline__ void store(float* p) const {
        if (W == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1 % W], v[2 % W], v[3 % W]);
        else *p = v[0];
    }
};

// 8 consecutive values of either storage type, as they are in memory
template <typename T>
struct MemRaw8;
template <>
struct MemRaw8<bf16> {
    uint4 a;
    __device__ __forceinline__ void load(const bf16* p) { a = *reinterpret_cast<const uint4*>(p); }
    __device__ __forceinline__ float dot(const MemRaw8<bf16>& o) const {
        const uint32_t x[4] = {a.x, a.y, a.z, a.w}, y[4] = {o.a.x, o.a.y, o.a.z, o.a.w};
        float s = 0.0f;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            s = fmaf(__uint_as_float(x[i] << 16), __uint_as_float(y[i] << 16), s);
            s = fmaf(__uint_as_float(x[i] & 0xffff0000u), __uint_as_float(y[i] & 0xffff0000u), s);
        }
        return s;
    }
};
template <>
struct MemRaw8<float> {
    float4 a, b;
    __device__ __forceinline__ void load(const float* p) {
        a = *reinterpret_cast<const float4*>(p);
        b = *reinterpret_cast<const float4*>(p + 4);
    }
    __device__ __forceinline__ float dot(const MemRaw8<float>& o) const {
        float s = a.x * o.a.x;
        s = fmaf(a.y, o.a.y, s), s = fmaf(a.z, o.a.z, s), s = fmaf(a.w, o.a.w, s);
        s = fmaf(b.x, o.b.x, s), s = fmaf(b.y, o.b.y, s), s = fmaf(b.z, o.b.z, s), s = fmaf(b.w, o.b.w, s);
        return s;
    }
};

// A block owns CT * VW columns; thread (g, c) rows g, g + G, ... of columns c * VW .. + VW - 1.
// VEC: the input's and the weights' rows are cut into whole 16-byte pieces.
template <typename T, int VW, int CT, int RPT, bool VEC>
__global__ void __launch_bounds__(MEM_STEP_THREADS, 2)
mlstm_step_kernel(const T* __restrict__ proj, long stride, int q_off, int k_off, int v_off, const T* __restrict__ x, long x_stride,
                  const T* __restrict__ w_gate, int width, const MemGates gp, float q_scale, float* __restrict__ out, long out_stride,
                  float* __restrict__ state, float* __restrict__ tails, const int* __restrict__ cu_seqlens,
                  const int* __restrict__ seq_slot, int H, int D, int V, int v_blocks) {
    pdl_trigger();
    constexpr int G = MEM_STEP_THREADS / CT, COLS = CT * VW, WARPS = MEM_STEP_THREADS / 32;
    __shared__ float qs[G * RPT], ks[G * RPT];
    __shared__ __align__(16) float red[WARPS][COLS];
    __shared__ float sums[4][WARPS];
    __shared__ int last;
    const int seq = blockIdx.y;
    const int slot = seq_slot[seq];
    if (slot < 0) return;
    const int h = blockIdx.x / v_blocks;
    const int v0 = (blockIdx.x - h * v_blocks) * COLS;
    const int tid = threadIdx.x, c = tid % CT, g = tid / CT, warp = tid >> 5, lane = tid & 31;
    const bool col_ok = v0 + c * VW < V;
    float* sp = state + (((size_t)slot * H + h) * D) * V + v0 + c * VW;
    float* tail = tails + ((size_t)slot * H + h) * (D + 2);
    MemCols<VW> S[RPT];
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int d = g + G * i;
        if (col_ok && d < D) S[i].load(sp + (size_t)d * V);
        else S[i].zero();
    }
    const float n_old = tid < D ? tail[tid] : 0.0f;       // D <= 256: a row a thread
    const float m_old = tail[D];
    const T* wi = w_gate + (size_t)h * width;             // the head's input gate row, its forget gate row H rows on
    const T* wf = wi + (size_t)H * width;
    MemRaw8<T> ri, rf;
    if (VEC && tid * 8 < width) ri.load(wi + tid * 8), rf.load(wf + tid * 8);
    __syncthreads();                                      // every thread holds its n and m
    if (tid == 0) last = mem_last_reader(tail, D, v_blocks) ? 1 : 0;
    pdl_wait();
    const int t = cu_seqlens[seq];
    const T* row = proj + (size_t)t * stride;
    const T* xr = x + (size_t)t * x_stride;
    float zi = 0.0f, zf = 0.0f, nq = 0.0f, kq = 0.0f;
    if (tid < D) {
        const float qv = to_f32(row[q_off + (size_t)h * D + tid]) * q_scale, kv = to_f32(row[k_off + (size_t)h * D + tid]);
        qs[tid] = qv;
        ks[tid] = kv;
        nq = n_old * qv;
        kq = kv * qv;
    }
    float vv[VW];
#pragma unroll
    for (int j = 0; j < VW; ++j) vv[j] = col_ok ? to_f32(row[v_off + (size_t)h * V + v0 + c * VW + j]) : 0.0f;
    if (VEC) {
        MemRaw8<T> rx;
        if (tid * 8 < width) {
            rx.load(xr + tid * 8);
            zi = ri.dot(rx), zf = rf.dot(rx);
        }
        for (int j = (tid + MEM_STEP_THREADS) * 8; j < width; j += MEM_STEP_THREADS * 8) {
            ri.load(wi + j), rf.load(wf + j), rx.load(xr + j);
            zi += ri.dot(rx), zf += rf.dot(rx);
        }
    } else {
        for (int j = tid; j < width; j += MEM_STEP_THREADS) {
            const float xv = to_f32(xr[j]);
            zi = fmaf(to_f32(wi[j]), xv, zi), zf = fmaf(to_f32(wf[j]), xv, zf);
        }
    }
    zi = warp_sum(zi), zf = warp_sum(zf), nq = warp_sum(nq), kq = warp_sum(kq);
    if (lane == 0) sums[0][warp] = zi, sums[1][warp] = zf, sums[2][warp] = nq, sums[3][warp] = kq;
    __syncthreads();
    float acc[VW];
#pragma unroll
    for (int j = 0; j < VW; ++j) acc[j] = 0.0f;
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int d = g + G * i;
        const float qv = d < D ? qs[d] : 0.0f;
#pragma unroll
        for (int j = 0; j < VW; ++j) acc[j] = fmaf(S[i].v[j], qv, acc[j]);
    }
#pragma unroll
    for (int o = CT; o < 32; o <<= 1)                     // the warp's other rows of the same columns
#pragma unroll
        for (int j = 0; j < VW; ++j) acc[j] += __shfl_xor_sync(0xffffffffu, acc[j], o);
    if (lane < CT)
#pragma unroll
        for (int j = 0; j < VW; ++j) red[warp][c * VW + j] = acc[j];
    zi = zf = nq = kq = 0.0f;
#pragma unroll
    for (int i = 0; i < WARPS; ++i) zi += sums[0][i], zf += sums[1][i], nq += sums[2][i], kq += sums[3][i];
    const float gi = mem_log_input(gp, zi, h), gf = mem_log_forget(gp, zf, h);
    const float m = fmaxf(gf + m_old, gi);
    const float keep = expf(gf + m_old - m), put = expf(gi - m);
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int d = g + G * i;
        if (d < D && col_ok) {
            const float kv = put * ks[d];
#pragma unroll
            for (int j = 0; j < VW; ++j) S[i].v[j] = fmaf(keep, S[i].v[j], kv * vv[j]);
            S[i].store(sp + (size_t)d * V);
        }
    }
    __syncthreads();
    if (tid < COLS && v0 + tid < V) {
        float o = 0.0f;
#pragma unroll
        for (int i = 0; i < WARPS; ++i) o += red[i][tid];
        const float v = to_f32(row[v_off + (size_t)h * V + v0 + tid]);
        o = fmaf(keep, o, put * kq * v);
        out[(size_t)t * out_stride + (size_t)h * V + v0 + tid] = o / mem_denominator(fmaf(keep, nq, put * kq), m);
    }
    if (last) {
        if (tid < D) tail[tid] = fmaf(keep, n_old, put * ks[tid]);
        if (tid == 0) tail[D] = m;
    }
}

template <typename T>
static void launch_mem_step(const void* proj, long stride, int q_off, int k_off, int v_off, const void* x, long x_stride, const void* w_gate,
                            int width, const MemGates& gp, float q_scale, float* out, long out_stride, float* state, float* tails,
                            const int* cu_seqlens, const int* seq_slot, int n_seqs, int H, int D, int V, cudaStream_t stream) {
    const dim3 block(MEM_STEP_THREADS);
    const bool vec = width % 8 == 0 && x_stride % 8 == 0 && ((uintptr_t)x & 15) == 0 && ((uintptr_t)w_gate & 15) == 0;
#define BFI_MEM_STEP(VW, CT, R, VV)                                                                                             \
    do {                                                                                                                        \
        const int v_blocks = (V + VW * CT - 1) / (VW * CT);                                                                     \
        bfi_launch(mlstm_step_kernel<T, VW, CT, R, VV>, dim3(H * v_blocks, n_seqs), block, 0, stream, (const T*)proj, stride, q_off, k_off, \
                   v_off, (const T*)x, x_stride, (const T*)w_gate, width, gp, q_scale, out, out_stride, state, tails, cu_seqlens, seq_slot, \
                   H, D, V, v_blocks);                                                                                          \
    } while (0)
    if (vec && V % 4 == 0 && ((uintptr_t)state & 15) == 0) {
        // columns per block: as many as leave every SM a block (the gates are made once a block)
        const long heads = (long)n_seqs * H, n_sm = bfi_sm_count();
        if (V > 64 && D <= 128 && heads * ((V + 127) / 128) >= n_sm) {
            if (D <= 64) BFI_MEM_STEP(4, 32, 8, true);
            else BFI_MEM_STEP(4, 32, 16, true);
        } else if (V > 32 && heads * ((V + 63) / 64) >= n_sm) {
            if (D <= 64) BFI_MEM_STEP(4, 16, 4, true);
            else if (D <= 128) BFI_MEM_STEP(4, 16, 8, true);
            else BFI_MEM_STEP(4, 16, 16, true);
        } else {
            if (D <= 64) BFI_MEM_STEP(4, 8, 2, true);
            else if (D <= 128) BFI_MEM_STEP(4, 8, 4, true);
            else BFI_MEM_STEP(4, 8, 8, true);
        }
        return;
    }
#define BFI_MEM_STEP_R(R)                     \
    do {                                      \
        if (vec) BFI_MEM_STEP(1, 32, R, true); \
        else BFI_MEM_STEP(1, 32, R, false);    \
    } while (0)
    if (D <= 32) BFI_MEM_STEP_R(4);
    else if (D <= 64) BFI_MEM_STEP_R(8);
    else if (D <= 128) BFI_MEM_STEP_R(16);
    else BFI_MEM_STEP_R(32);
#undef BFI_MEM_STEP_R
#undef BFI_MEM_STEP
}

// Returns 2 ("not taken") for heads of more than 256 key values; the caller then makes the gates' logits and
// runs bfi_mlstm_scan.
extern "C" int bfi_mlstm_step(const void* proj, int dtype, long stride, int q_off, int k_off, int v_off, const void* x, long x_stride,
                              const void* w_gate, int width, const float* bias_i, const float* bias_f, float cap, float q_scale, float* out,
                              long out_stride, float* state, float* tails, const int* cu_seqlens, const int* seq_slot, int n_seqs, int H,
                              int D, int V, cudaStream_t stream) {
    BFI_REQUIRE(dtype_ok(dtype), "mlstm_step: unknown dtype code %d", dtype);
    BFI_REQUIRE(H > 0 && D > 0 && V > 0 && width > 0, "mlstm_step: bad sizes heads=%d dim=%d vdim=%d width=%d", H, D, V, width);
    BFI_REQUIRE(cap > 0.0f, "mlstm_step: the gates' cap must be positive");
    BFI_REQUIRE(out_stride >= (long)H * V && x_stride >= width, "mlstm_step: a row stride is shorter than the row");
    if (n_seqs <= 0) return 0;
    if (D > MEM_STEP_MAX_D || n_seqs > 65535) return 2;
    const MemGates gp = {bias_i, bias_f, cap};
    if (dtype == BFI_F32)
        launch_mem_step<float>(proj, stride, q_off, k_off, v_off, x, x_stride, w_gate, width, gp, q_scale, out, out_stride, state, tails,
                               cu_seqlens, seq_slot, n_seqs, H, D, V, stream);
    else
        launch_mem_step<bf16>(proj, stride, q_off, k_off, v_off, x, x_stride, w_gate, width, gp, q_scale, out, out_stride, state, tails,
                              cu_seqlens, seq_slot, n_seqs, H, D, V, stream);
    return bfi_check_launch("mlstm_step");
}

BFI_TRACE_EXPORT(mlstm)
