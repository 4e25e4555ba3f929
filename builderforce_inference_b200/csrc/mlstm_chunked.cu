// The matrix memory (mlstm.cuh) over runs of new tokens, on the tensor cores: a chunk of 64 tokens at a
// time.  With S, n, m the state before the chunk, t and j counted inside it, F_t = f_0 + .. + f_t the sum
// of the log forget gates and M_t = F_t + max(m, max_{j <= t} (i_j - F_j)) the running maximum:
//     g_t    = exp(F_t + m - M_t)              A_tj = exp(F_t - F_j + i_j - M_t) (q_t . k_j)       j <= t
//     num_t  = g_t (q_t S) + sum_j A_tj v_j    den_t = g_t (q_t . n) + sum_j A_tj
//     S' = g_last S + sum_j w_j k_j v_j^T      n' = g_last n + sum_j w_j k_j        w_j = exp(F_last - F_j + i_j - M_last)
// No exponent is positive, whatever the gates.  q, k, v are the bfloat16 projections themselves (products
// of two bfloat16 values are exact in float32); gates, scores, sums and the state are float32.  Where a
// float32 matrix has to be a tensor-core operand (S, A, w v) it is a bfloat16 head and remainder.
//
// A block (16 warps) owns VB columns of one head of one sequence and walks its chunks in order, two
// phases and two barriers a chunk:
//   A  scores q k^T, decayed in registers and left as operands; q S into registers; q . n; w v split;
//      one warp scans the next chunk's gates; the next chunk's q, k, v travel by cp.async
//   B  num += A v, divided by its den and stored; S += k^T (w v) in registers, its split to shared memory; n
// Every warp keeps its tiles of S (float32) and of num in registers from chunk to chunk.
#include "chunk_tiles.cuh"
#include "mlstm.cuh"

#define MC 64              // tokens per chunk
#define MC_WARPS 16
#define MC_THREADS (MC_WARPS * 32)
#define MC_MAX_D 256

struct McSmem {
    int ldq, ldv, lda;
    size_t q, k, v, vhi, vlo, ahi, alo, shi, slo, n, nq, rs, gates, total;      // q, k, v: two buffers each
};
// per chunk parity: FM_t = F_t - M_t, IF_j = i_j - F_j, q_scale * g_t, w_j, exp(-M_t), then g_last and M_last
#define MC_GATE_FLOATS (5 * MC + 2)

static __host__ __device__ inline McSmem mc_layout(int D, int VB) {
    McSmem s;
    s.ldq = D + 8, s.ldv = VB + 8, s.lda = MC + 8;
    size_t o = 0;
    auto take = [&](size_t bytes) { size_t at = o; o += (bytes + 127) / 128 * 128; return at; };
    s.q = take((size_t)2 * MC * s.ldq * 2);
    s.k = take((size_t)2 * MC * s.ldq * 2);
    s.v = take((size_t)2 * MC * s.ldv * 2);
    s.vhi = take((size_t)MC * s.ldv * 2);
    s.vlo = take((size_t)MC * s.ldv * 2);
    s.ahi = take((size_t)MC * s.lda * 2);
    s.alo = take((size_t)MC * s.lda * 2);
    s.shi = take((size_t)D * s.ldv * 2);
    s.slo = take((size_t)D * s.ldv * 2);
    s.n = take((size_t)D * 4);
    s.nq = take((size_t)MC * 4);
    s.rs = take((size_t)4 * MC * 4);
    s.gates = take((size_t)2 * MC_GATE_FLOATS * 4);
    s.total = o;
    return s;
}

// 16 bytes to shared memory, zeros where there is no such row
__device__ __forceinline__ void mc_copy16(void* dst, const void* src, bool have) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(have ? 16 : 0));
}
__device__ __forceinline__ void mc_put_split(bf16* hi, bf16* lo, float a, float b) {
    const uint32_t h = pack_bf16(a, b);
    *reinterpret_cast<uint32_t*>(hi) = h;
    *reinterpret_cast<uint32_t*>(lo) = pack_bf16(a - bf16_lo(h), b - bf16_hi(h));
}

// DC: the head's key size when it is known at compile time (the products' loops are then unrolled), 0 for
// any multiple of 16 up to MC_MAX_D.
template <int VB, int DC>
__global__ void __launch_bounds__(MC_THREADS)
mlstm_chunk_kernel(const bf16* __restrict__ proj, long stride, int q_off, int k_off, int v_off, const float* __restrict__ gates,
                   long gate_stride, const MemGates gp, float q_scale, float* __restrict__ out, long out_stride,
                   float* __restrict__ state, float* __restrict__ tails, const int* __restrict__ cu_seqlens,
                   const int* __restrict__ seq_slot, int H, int V, int D_any, int v_blocks) {
    pdl_trigger();
    const int D = DC ? DC : D_any, DT = D / 16;
    constexpr int VT = VB / 16, CT = MC / 16;
    constexpr int NT = DC ? (DC / 16 * VT + MC_WARPS - 1) / MC_WARPS : VT;      // tiles of S a warp keeps
    extern __shared__ __align__(128) unsigned char mc_smem[];
    const McSmem L = mc_layout(D, VB);
    bf16* Vhi = reinterpret_cast<bf16*>(mc_smem + L.vhi);
    bf16* Vlo = reinterpret_cast<bf16*>(mc_smem + L.vlo);
    bf16* Ahi = reinterpret_cast<bf16*>(mc_smem + L.ahi);
    bf16* Alo = reinterpret_cast<bf16*>(mc_smem + L.alo);
    bf16* Shi = reinterpret_cast<bf16*>(mc_smem + L.shi);
    bf16* Slo = reinterpret_cast<bf16*>(mc_smem + L.slo);
    float* ns = reinterpret_cast<float*>(mc_smem + L.n);
    float* nqs = reinterpret_cast<float*>(mc_smem + L.nq);
    float* rs = reinterpret_cast<float*>(mc_smem + L.rs);                       // [CT][MC] row sums of A by key tile
    float* gate_smem = reinterpret_cast<float*>(mc_smem + L.gates);
    __shared__ int last_reader;

    const int seq = blockIdx.y;
    const int slot = seq_slot[seq];
    if (slot < 0) return;
    const int h = blockIdx.x / v_blocks;
    const int v0 = (blockIdx.x - h * v_blocks) * VB;
    const int t0 = cu_seqlens[seq], nt = cu_seqlens[seq + 1] - t0;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;

    // ---- the state earlier steps left (zero for a fresh slot): not written by this step's kernels
    float* sp = state + (((size_t)slot * H + h) * D) * V + v0;
    float* tail = tails + ((size_t)slot * H + h) * (D + 2);
    float S[NT][2][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) {
        const int job = warp + i * MC_WARPS, td = job / VT, tv = job - td * VT;
#pragma unroll
        for (int nb = 0; nb < 2; ++nb) {
            float2 lo = make_float2(0.0f, 0.0f), hi = lo;
            if (job < DT * VT) {
                const float* p = sp + (size_t)(td * 16 + g) * V + tv * 16 + nb * 8 + 2 * t4;
                lo = *reinterpret_cast<const float2*>(p);
                hi = *reinterpret_cast<const float2*>(p + (size_t)8 * V);
            }
            S[i][nb][0] = lo.x, S[i][nb][1] = lo.y, S[i][nb][2] = hi.x, S[i][nb][3] = hi.y;
        }
    }
    auto publish_state = [&]() {
#pragma unroll
        for (int i = 0; i < NT; ++i) {
            const int job = warp + i * MC_WARPS, td = job / VT, tv = job - td * VT;
            if (job >= DT * VT) continue;
            const int at = (td * 16 + g) * L.ldv + tv * 16 + 2 * t4;
#pragma unroll
            for (int nb = 0; nb < 2; ++nb) {
                mc_put_split(Shi + at + nb * 8, Slo + at + nb * 8, S[i][nb][0], S[i][nb][1]);
                mc_put_split(Shi + at + 8 * L.ldv + nb * 8, Slo + at + 8 * L.ldv + nb * 8, S[i][nb][2], S[i][nb][3]);
            }
        }
    };
    publish_state();
    // n: n_parts neighbouring threads share a row (and hold the same value)
    const int n_parts = D <= MC_THREADS / 4 ? 4 : 2;
    const int n_row = tid / n_parts, n_part = tid - n_row * n_parts;
    float n_reg = n_row < D ? tail[n_row] : 0.0f;
    if (n_row < D && n_part == 0) ns[n_row] = n_reg;
    float m = tail[D];                                    // used by the warp that scans the gates
    __syncthreads();
    if (tid == 0) last_reader = mem_last_reader(tail, D, v_blocks) ? 1 : 0;
    pdl_wait();

    // ---- the gates of a chunk: lane l of the last warp has tokens 2l and 2l + 1
    float zi[2], zf[2];
    auto fetch_gates = [&](int c0) {
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int t = c0 + 2 * lane + u;
            zi[u] = zf[u] = 0.0f;
            if (t < nt) {
                const float* row = gates + (size_t)(t0 + t) * gate_stride;
                zi[u] = row[h], zf[u] = row[H + h];
            }
        }
    };
    auto scan_gates = [&](int c0, float* gs) {
        // tokens past the end neither forget (f = 0) nor put (i = -inf)
        const int n = nt - c0;
        float gi[2], F[2];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const bool have = 2 * lane + u < n;
            gi[u] = have ? mem_log_input(gp, zi[u], h) : -INFINITY;
            F[u] = have ? mem_log_forget(gp, zf[u], h) : 0.0f;
        }
        F[1] += F[0];
        float before = F[1];                               // sum of the lanes up to this one
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float other = __shfl_up_sync(0xffffffffu, before, o);
            if (lane >= o) before += other;
        }
        const float base = before - F[1];
        F[0] += base, F[1] += base;
        const float d0 = gi[0] - F[0], d1 = gi[1] - F[1];
        float top = fmaxf(d0, d1);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float other = __shfl_up_sync(0xffffffffu, top, o);
            if (lane >= o) top = fmaxf(top, other);
        }
        const float top_before = __shfl_up_sync(0xffffffffu, top, 1);
        const float p0 = fmaxf(m, fmaxf(lane > 0 ? top_before : -INFINITY, d0)), p1 = fmaxf(m, top);
        const float M0 = F[0] + p0, M1 = F[1] + p1;        // F - M is -p: the large sum cancels exactly
        const float last_p = __shfl_sync(0xffffffffu, p1, 31);
        float* FM = gs;
        float* IF = gs + MC;
        *reinterpret_cast<float2*>(FM + 2 * lane) = make_float2(-p0, -p1);
        *reinterpret_cast<float2*>(IF + 2 * lane) = make_float2(d0, d1);
        *reinterpret_cast<float2*>(gs + 2 * MC + 2 * lane) = make_float2(q_scale * expf(m - p0), q_scale * expf(m - p1));
        *reinterpret_cast<float2*>(gs + 3 * MC + 2 * lane) = make_float2(expf(d0 - last_p), expf(d1 - last_p));
        *reinterpret_cast<float2*>(gs + 4 * MC + 2 * lane) = make_float2(expf(-M0), expf(-M1));
        const float M_last = __shfl_sync(0xffffffffu, M1, 31);
        if (lane == 31) gs[5 * MC] = expf(m - last_p), gs[5 * MC + 1] = M_last;
        m = M_last;
    };

    // ---- a chunk's q, k (all of the head) and v (this block's columns)
    auto fetch = [&](int c0, int buf) {
        bf16* Qs = reinterpret_cast<bf16*>(mc_smem + L.q) + (size_t)buf * MC * L.ldq;
        bf16* Ks = reinterpret_cast<bf16*>(mc_smem + L.k) + (size_t)buf * MC * L.ldq;
        bf16* Vs = reinterpret_cast<bf16*>(mc_smem + L.v) + (size_t)buf * MC * L.ldv;
        const int D8 = D >> 3;
        for (int idx = tid; idx < MC * D8; idx += MC_THREADS) {
            const int t = idx / D8, e = idx - t * D8;
            const bool have = c0 + t < nt;
            const bf16* row = proj + (size_t)(t0 + (have ? c0 + t : 0)) * stride + (size_t)h * D + e * 8;
            mc_copy16(Qs + t * L.ldq + e * 8, row + q_off, have);
            mc_copy16(Ks + t * L.ldq + e * 8, row + k_off, have);
        }
        constexpr int VB8 = VB / 8;
        for (int idx = tid; idx < MC * VB8; idx += MC_THREADS) {
            const int t = idx / VB8, e = idx - t * VB8;
            const bool have = c0 + t < nt;
            mc_copy16(Vs + t * L.ldv + e * 8, proj + (size_t)(t0 + (have ? c0 + t : 0)) * stride + v_off + (size_t)h * V + v0 + e * 8, have);
        }
        cp_async_commit();
    };
    fetch(0, 0);
    if (warp == MC_WARPS - 1) {
        fetch_gates(0);
        scan_gates(0, gate_smem);
        fetch_gates(MC);
    }
    cp_async_wait<0>();
    __syncthreads();

    int buf = 0;
    for (int c0 = 0; c0 < nt; c0 += MC, buf ^= 1) {
        const int n = min(MC, nt - c0);
        const bf16* Qs = reinterpret_cast<const bf16*>(mc_smem + L.q) + (size_t)buf * MC * L.ldq;
        const bf16* Ks = reinterpret_cast<const bf16*>(mc_smem + L.k) + (size_t)buf * MC * L.ldq;
        const bf16* Vs = reinterpret_cast<const bf16*>(mc_smem + L.v) + (size_t)buf * MC * L.ldv;
        const float* gs = gate_smem + buf * MC_GATE_FLOATS;
        const float* FM = gs;
        const float* IF = gs + MC;
        const float* qg = gs + 2 * MC;
        const float* wj = gs + 3 * MC;
        const float* floor_m = gs + 4 * MC;
        if (c0 + MC < nt) fetch(c0 + MC, buf ^ 1);

        // ================ phase A
        // q S: warp w < CT * VT owns tile (w / VT, w % VT) of the output from here to its store
        float acc[2][4] = {};
        const int o_ti = warp / VT, o_tv = warp - o_ti * VT;
        const bool o_mine = warp < CT * VT;
        if (o_mine) {
            float rest[2][4] = {};
#pragma unroll
            for (int kk = 0; kk < (DC ? DC / 16 : DT); ++kk) {
                uint32_t fa[4], fb[4];
                lc_a_rows(fa, Qs + o_ti * 16 * L.ldq + kk * 16, L.ldq);
                lc_b_rows(fb, Shi + kk * 16 * L.ldv + o_tv * 16, L.ldv);
                mma16816(acc[0], fa, fb[0], fb[1]);
                mma16816(acc[1], fa, fb[2], fb[3]);
                lc_b_rows(fb, Slo + kk * 16 * L.ldv + o_tv * 16, L.ldv);
                mma16816(rest[0], fa, fb[0], fb[1]);
                mma16816(rest[1], fa, fb[2], fb[3]);
            }
            const float s0 = qg[o_ti * 16 + g], s1 = qg[o_ti * 16 + g + 8];
#pragma unroll
            for (int nb = 0; nb < 2; ++nb) {
                acc[nb][0] = (acc[nb][0] + rest[nb][0]) * s0, acc[nb][1] = (acc[nb][1] + rest[nb][1]) * s0;
                acc[nb][2] = (acc[nb][2] + rest[nb][2]) * s1, acc[nb][3] = (acc[nb][3] + rest[nb][3]) * s1;
            }
        }
        // scores at or below the diagonal, dealt from the last warp down
        for (int job = MC_WARPS - 1 - warp; job < CT * (CT + 1) / 2; job += MC_WARPS) {
            int ti = 0, tj = job;
            while (tj > ti) tj -= ++ti;                    // job -> (ti, tj) with tj <= ti
            float a[2][4] = {};
#pragma unroll
            for (int kk = 0; kk < (DC ? DC / 16 : DT); ++kk) {
                uint32_t fa[4], fb[4];
                lc_a_rows(fa, Qs + ti * 16 * L.ldq + kk * 16, L.ldq);
                lc_b_cols(fb, Ks + tj * 16 * L.ldq + kk * 16, L.ldq);          // B[k = d][n = j] = k_j[d]
                mma16816(a[0], fa, fb[0], fb[1]);
                mma16816(a[1], fa, fb[2], fb[3]);
            }
            float sum[2] = {0.0f, 0.0f};
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                const int row = ti * 16 + g + r * 8;
                const float fm = FM[row];
#pragma unroll
                for (int nb = 0; nb < 2; ++nb) {
                    const int col = tj * 16 + nb * 8 + 2 * t4;
                    const float2 f = *reinterpret_cast<const float2*>(IF + col);
                    const float x = col <= row ? a[nb][2 * r] * q_scale * __expf(fm + f.x) : 0.0f;
                    const float y = col + 1 <= row ? a[nb][2 * r + 1] * q_scale * __expf(fm + f.y) : 0.0f;
                    sum[r] += x + y;
                    mc_put_split(Ahi + row * L.lda + col, Alo + row * L.lda + col, x, y);
                }
                sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 1);
                sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 2);
                if (t4 == 0) rs[tj * MC + row] = sum[r];
            }
        }
        // q . n: eight threads a token
        {
            const int tok = tid >> 3, part = tid & 7;
            float s = 0.0f;
            for (int p = part; p < (D >> 3); p += 8) {
                const uint4 raw = *reinterpret_cast<const uint4*>(Qs + tok * L.ldq + p * 8);
                const float4 a = *reinterpret_cast<const float4*>(ns + p * 8), b = *reinterpret_cast<const float4*>(ns + p * 8 + 4);
                s = fmaf(bf16_lo(raw.x), a.x, s), s = fmaf(bf16_hi(raw.x), a.y, s);
                s = fmaf(bf16_lo(raw.y), a.z, s), s = fmaf(bf16_hi(raw.y), a.w, s);
                s = fmaf(bf16_lo(raw.z), b.x, s), s = fmaf(bf16_hi(raw.z), b.y, s);
                s = fmaf(bf16_lo(raw.w), b.z, s), s = fmaf(bf16_hi(raw.w), b.w, s);
            }
            s += __shfl_xor_sync(0xffffffffu, s, 1);
            s += __shfl_xor_sync(0xffffffffu, s, 2);
            s += __shfl_xor_sync(0xffffffffu, s, 4);
            if (part == 0) nqs[tok] = s;
        }
        // w v
        for (int idx = tid; idx < MC * VB / 2; idx += MC_THREADS) {
            const int t = idx / (VB / 2), c = (idx - t * (VB / 2)) * 2;
            const uint32_t raw = *reinterpret_cast<const uint32_t*>(Vs + t * L.ldv + c);
            const float w = wj[t];
            mc_put_split(Vhi + t * L.ldv + c, Vlo + t * L.ldv + c, w * bf16_lo(raw), w * bf16_hi(raw));
        }
        if (warp == MC_WARPS - 1 && c0 + MC < nt) {
            scan_gates(c0 + MC, gate_smem + (buf ^ 1) * MC_GATE_FLOATS);
            fetch_gates(c0 + 2 * MC);
        }
        __syncthreads();

        // ================ phase B
        if (o_mine) {
#pragma unroll
            for (int kj = 0; kj < CT; ++kj) {
                if (kj > o_ti) break;
                uint32_t fa[4], fb[4];
                lc_b_rows(fb, Vs + kj * 16 * L.ldv + o_tv * 16, L.ldv);
                lc_a_rows(fa, Ahi + o_ti * 16 * L.lda + kj * 16, L.lda);
                mma16816(acc[0], fa, fb[0], fb[1]);
                mma16816(acc[1], fa, fb[2], fb[3]);
                lc_a_rows(fa, Alo + o_ti * 16 * L.lda + kj * 16, L.lda);
                mma16816(acc[0], fa, fb[0], fb[1]);
                mma16816(acc[1], fa, fb[2], fb[3]);
            }
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                const int row = o_ti * 16 + g + r * 8;
                float den = qg[row] * nqs[row];
                for (int tj = 0; tj <= o_ti; ++tj) den += rs[tj * MC + row];
                const float inv = 1.0f / (fmaxf(fabsf(den), floor_m[row]) + MEM_DEN_FLOOR);
                if (row < n) {
                    float* o = out + (size_t)(t0 + c0 + row) * out_stride + (size_t)h * V + v0 + o_tv * 16 + 2 * t4;
#pragma unroll
                    for (int nb = 0; nb < 2; ++nb)
                        *reinterpret_cast<float2*>(o + nb * 8) = make_float2(acc[nb][2 * r] * inv, acc[nb][2 * r + 1] * inv);
                }
            }
        }
        const float g_last = gs[5 * MC];
#pragma unroll
        for (int i = 0; i < NT; ++i) {
            const int job = warp + i * MC_WARPS, td = job / VT, tv = job - td * VT;
            if (job >= DT * VT) continue;
#pragma unroll
            for (int e = 0; e < 8; ++e) S[i][e >> 2][e & 3] *= g_last;
#pragma unroll
            for (int kj = 0; kj < CT; ++kj) {
                uint32_t fa[4], fb[4];
                lc_a_cols(fa, Ks + kj * 16 * L.ldq + td * 16, L.ldq);            // A[m = d][k = j] = k_j[d]
                lc_b_rows(fb, Vhi + kj * 16 * L.ldv + tv * 16, L.ldv);
                mma16816(S[i][0], fa, fb[0], fb[1]);
                mma16816(S[i][1], fa, fb[2], fb[3]);
                lc_b_rows(fb, Vlo + kj * 16 * L.ldv + tv * 16, L.ldv);
                mma16816(S[i][0], fa, fb[0], fb[1]);
                mma16816(S[i][1], fa, fb[2], fb[3]);
            }
        }
        publish_state();
        {
            float add = 0.0f;
            if (n_row < D) {
#pragma unroll 8
                for (int j = n_part; j < MC; j += n_parts) add = fmaf(wj[j], __bfloat162float(Ks[j * L.ldq + n_row]), add);
            }
            add += __shfl_xor_sync(0xffffffffu, add, 1);
            if (n_parts == 4) add += __shfl_xor_sync(0xffffffffu, add, 2);
            n_reg = fmaf(g_last, n_reg, add);
            if (n_row < D && n_part == 0) ns[n_row] = n_reg;
        }
        cp_async_wait<0>();
        __syncthreads();
    }

#pragma unroll
    for (int i = 0; i < NT; ++i) {
        const int job = warp + i * MC_WARPS, td = job / VT, tv = job - td * VT;
        if (job >= DT * VT) continue;
#pragma unroll
        for (int nb = 0; nb < 2; ++nb) {
            float* p = sp + (size_t)(td * 16 + g) * V + tv * 16 + nb * 8 + 2 * t4;
            *reinterpret_cast<float2*>(p) = make_float2(S[i][nb][0], S[i][nb][1]);
            *reinterpret_cast<float2*>(p + (size_t)8 * V) = make_float2(S[i][nb][2], S[i][nb][3]);
        }
    }
    if (last_reader && nt > 0) {
        if (n_row < D && n_part == 0) tail[n_row] = n_reg;
        if (tid == MC_THREADS - 1) tail[D] = m;            // the scanning warp's
    }
}

template <int VB, int DC>
static int launch_mem_chunks(const bf16* proj, long stride, int q_off, int k_off, int v_off, const float* gates, long gate_stride,
                             const MemGates& gp, float q_scale, float* out, long out_stride, float* state, float* tails,
                             const int* cu_seqlens, const int* seq_slot, int n_seqs, int H, int D, int V, cudaStream_t stream) {
    const McSmem L = mc_layout(D, VB);
    const int v_blocks = V / VB;
    auto kernel = mlstm_chunk_kernel<VB, DC>;
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)L.total);
    if (e != cudaSuccess) return bfi_fail("mlstm_chunks: cannot reserve %zu bytes of shared memory: %s", L.total, cudaGetErrorString(e));
    bfi_launch(kernel, dim3(H * v_blocks, n_seqs), dim3(MC_THREADS), L.total, stream, proj, stride, q_off, k_off, v_off, gates, gate_stride,
               gp, q_scale, out, out_stride, state, tails, cu_seqlens, seq_slot, H, V, D, v_blocks);
    return bfi_check_launch("mlstm_chunks");
}

// Returns 2 ("not taken") for sizes this kernel does not handle; the caller then runs bfi_mlstm_scan.
// `vb`: the columns per block (16, 32 or 64), 0 for the kernel's own choice.
extern "C" int bfi_mlstm_chunks_bf16(const void* proj, long stride, int q_off, int k_off, int v_off, const float* gates, long gate_stride,
                                     const float* bias_i, const float* bias_f, float cap, float q_scale, float* out, long out_stride,
                                     float* state, float* tails, const int* cu_seqlens, const int* seq_slot, int n_seqs, int H, int D,
                                     int V, int vb, cudaStream_t stream) {
    BFI_REQUIRE(H > 0 && D > 0 && V > 0, "mlstm_chunks: bad sizes heads=%d dim=%d vdim=%d", H, D, V);
    BFI_REQUIRE(cap > 0.0f, "mlstm_chunks: the gates' cap must be positive");
    BFI_REQUIRE(out_stride >= (long)H * V && gate_stride >= 2L * H, "mlstm_chunks: a row stride is shorter than the heads");
    if (n_seqs <= 0) return 0;
    if (D % 16 != 0 || D > MC_MAX_D || V % 16 != 0 || n_seqs > 65535) return 2;
    // q, k and v are read in 16-byte pieces, the state and the output in pieces of 8
    if (((uintptr_t)proj & 15) != 0 || stride % 8 != 0 || q_off % 8 != 0 || k_off % 8 != 0 || v_off % 8 != 0 || out_stride % 2 != 0 ||
        ((uintptr_t)out & 7) != 0 || ((uintptr_t)state & 7) != 0)
        return 2;
    const MemGates gp = {bias_i, bias_f, cap};
    // Columns per block: the time of a chunk times the rounds the blocks take on the GPU's SMs (one block per
    // SM, two where two fit), the cheapest product wins.
    const size_t limit = 227 * 1024;
    const int n_sm = bfi_sm_count();
    int best_vb = 0;
    double best = 0.0;
    for (int c = 0; c < 3; ++c) {
        const int cand = 64 >> c;
        const double per_chunk = c == 0 ? 3.6 : (c == 1 ? 2.8 : 2.4);
        if (V % cand != 0 || mc_layout(D, cand).total > limit || (vb > 0 && vb != cand)) continue;
        const long blocks = (long)n_seqs * H * (V / cand);
        const double cost = (double)((blocks + n_sm - 1) / n_sm) * per_chunk;
        if (best_vb == 0 || cost < best) best_vb = cand, best = cost;
    }
    if (best_vb == 0) return 2;
    const bf16* p = (const bf16*)proj;
#define BFI_MC(VBB, DCC)                                                                                                         \
    return launch_mem_chunks<VBB, DCC>(p, stride, q_off, k_off, v_off, gates, gate_stride, gp, q_scale, out, out_stride, state, tails, \
                                       cu_seqlens, seq_slot, n_seqs, H, D, V, stream)
#define BFI_MC_D(VBB)               \
    if (D == 64) BFI_MC(VBB, 64);   \
    if (D == 128) BFI_MC(VBB, 128); \
    if (D == 256) BFI_MC(VBB, 256); \
    BFI_MC(VBB, 0)
    if (best_vb == 64) {
        if (D == 64) BFI_MC(64, 64);
        if (D == 128) BFI_MC(64, 128);
        BFI_MC(64, 0);
    }
    if (best_vb == 32) { BFI_MC_D(32); }
    BFI_MC_D(16);
#undef BFI_MC_D
#undef BFI_MC
}

BFI_TRACE_EXPORT(mlstm_chunked)
