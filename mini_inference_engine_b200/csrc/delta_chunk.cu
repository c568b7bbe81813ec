// The gated delta rule with one decay per head over long portions, in chunks of 64 tokens (delta_rule.cu walks token by token).
//
// Within a chunk, with G_i the sum of the log decays up to token i, S the state in front of the chunk and
//   A_ij = beta_i exp(G_i - G_j) (k_i . k_j)  for j < i,      P_ij = exp(G_i - G_j) (q_i . k_j)  for j <= i,
// the recurrence S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q written out is
//   (I + A) U = diag(beta) (V - diag(e^G) K S),      O = diag(e^G) Q S + P U,      S <- e^{G_C} S + (diag(e^{G_C - G}) K)^T U,
// so a chunk is six small matrix products instead of 64 dependent steps.  Every exponent is a sum of log decays over a stretch of the
// chunk and never positive.  All of it is float32 on the CUDA cores (packed two to an instruction): the state is a 32-bit quantity, and
// the corrections that U holds cancel what earlier tokens wrote, which operands rounded for the tensor cores would not.
//
//   chunk_prep   a block per (chunk, key head): K K^T and Q K^T once, then for every head of the group the factors from its decays, the
//                inverse T of the unit triangular I + A (blocks of 16: each diagonal block by substitution, the rest by products),
//                and T diag(beta), P, e^G, e^{G_C - G} into scratch memory.
//   chunk_scan   a block per (row, head, 16 value columns) walks the row's chunks: its slice of the state stays in registers (and in shared
//                memory for the products that read it); keys and queries of the next chunk arrive by asynchronous copies while
//                this one is computed.
//
// Rows with fewer than `min_len` new tokens are left to delta_rule.cu.  Chunks count from the start of a row's portion.
#include "common.cuh"

#define CH 64                  // tokens a chunk
#define CHP 68                 // their stride in shared memory: rows of 64 and four words more, so that neighbouring rows lie four banks apart
#define COLS 16                // value columns a block of the scan

__device__ __forceinline__ void fma2(unsigned long long& d, unsigned long long a, unsigned long long b) {
    asm("fma.rn.f32x2 %0, %1, %2, %0;" : "+l"(d) : "l"(a), "l"(b));
}
__device__ __forceinline__ unsigned long long pack2(float lo, float hi) {
    unsigned long long r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ float2 unpack2(unsigned long long v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ float sum2(unsigned long long v) { const float2 f = unpack2(v); return f.x + f.y; }
struct Quad { unsigned long long lo, hi; };                    // four consecutive floats as two pairs
__device__ __forceinline__ Quad quad(const float* p) {
    const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(p);
    return Quad{v.x, v.y};
}
// 16 (or 4) bytes from global to shared memory; zeros where `on` is false (nothing is read then)
__device__ __forceinline__ void copy16(float* dst, const float* src, bool on) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(on ? 16 : 0) : "memory");
}
__device__ __forceinline__ void copy4(float* dst, const float* src, bool on) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(on ? 4 : 0) : "memory");
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void copy_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// 64 rows of up to DT entries (the rest zero) into rows of DT + 4; rows from `count` on are zero.
template <int DT>
__device__ __forceinline__ void copy_rows(float* dst, const float* src, int64_t stride, int D, int count) {
    for (int c = threadIdx.x; c < CH * (DT / 4); c += blockDim.x) {
        const int r = c / (DT / 4), d = (c - r * (DT / 4)) * 4;
        const bool on = r < count && d < D;
        copy16(dst + r * (DT + 4) + d, on ? src + r * stride + d : src, on);
    }
}

struct ChunkScratch {           // per (chunk, head): T diag(beta) [64, 64], P [64, 64], e^G [64], e^{G_C - G} [64]
    float* tb; float* p; float* eg; float* er;
    __device__ __forceinline__ ChunkScratch(float* base, int64_t item) {
        tb = base + item * (2 * CH * CH + 2 * CH);
        p = tb + CH * CH;
        eg = p + CH * CH;
        er = eg + CH;
    }
};

__device__ __forceinline__ int chunks_of(int n, int min_len) { return n >= min_len ? (n + CH - 1) / CH : 0; }

template <int DT>
__global__ void __launch_bounds__(256, 2) delta_chunk_prep_kernel(const float* __restrict__ qn, const float* __restrict__ kn,
                                                               const float* __restrict__ beta, const float* __restrict__ log_decay,
                                                               const int* __restrict__ row_q_start, const int* __restrict__ row_q_len,
                                                               int num_rows, int min_len, float* __restrict__ scratch, int H, int G, int D) {
    extern __shared__ __align__(16) float sm[];
    float* K = sm;                                             // [64][DT + 4]
    float* Q = K + CH * (DT + 4);
    float* KK = Q + CH * (DT + 4);                             // [64][68]: k_i . k_j
    float* QK = KK + CH * CHP;                                 // q_i . k_j
    float* X = QK + CH * CHP;                                  // products on the way to T [3][16][16]
    float* A = K;                                              // [64][68], and T: keys and queries are not read after the Gram matrices
    float* T = Q;
    __shared__ float lg[CH], be[CH];
    __shared__ int s_row, s_chunk;
    pdl_enter();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (warp == 0) {
        int within, items;
        const int r = warp_find_row(row_q_len, num_rows, (int)blockIdx.x, [&](int n) { return chunks_of(n, min_len); }, within, items);
        if (lane == 0) { s_row = r; s_chunk = within; }
    }
    __syncthreads();
    if (s_row < 0) return;
    const int g = blockIdx.y, row = s_row;
    const int t0 = row_q_start[row] + s_chunk * CH, count = min(CH, row_q_len[row] - s_chunk * CH);
    copy_rows<DT>(K, kn + ((int64_t)t0 * G + g) * D, (int64_t)G * D, D, count);
    copy_rows<DT>(Q, qn + ((int64_t)t0 * G + g) * D, (int64_t)G * D, D, count);
    copy_commit();
    copy_wait<0>();
    __syncthreads();
    {
        // four warps a Gram matrix, 32 x 32 entries a warp, 4 x 8 a lane (rows and columns interleaved over the lanes)
        const float* L = warp < 4 ? K : Q;
        float* out = warp < 4 ? KK : QK;
        const int rb = (warp & 1) * 32, cb = ((warp >> 1) & 1) * 32, r0 = rb + (lane >> 2), c0 = cb + (lane & 3);
        if (rb >= cb) {                                        // the block wholly above the diagonal is never read
            unsigned long long acc[4][8];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 8; ++j) acc[i][j] = 0ull;
#pragma unroll 2
            for (int d = 0; d < DT; d += 4) {
                Quad a[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) a[i] = quad(L + (r0 + 8 * i) * (DT + 4) + d);
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    const Quad b = quad(K + (c0 + 4 * j) * (DT + 4) + d);
#pragma unroll
                    for (int i = 0; i < 4; ++i) { fma2(acc[i][j], a[i].lo, b.lo); fma2(acc[i][j], a[i].hi, b.hi); }
                }
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 8; ++j) out[(r0 + 8 * i) * CHP + c0 + 4 * j] = sum2(acc[i][j]);
        }
    }
    for (int h = g * (H / G); h < (g + 1) * (H / G); ++h) {
        __syncthreads();                                       // the Gram matrices; and the head before is done with A, T, lg and be
        if (warp == 0) {
            // sums of the log decays: two tokens a lane (tokens beyond the row's end decay nothing and write nothing)
            const int i = 2 * lane;
            const int64_t at = (int64_t)(t0 + i) * H + h;
            const float a = i < count ? log_decay[at] : 0.f, b = i + 1 < count ? log_decay[at + H] : 0.f;
            float s = a + b;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) { const float up = __shfl_up_sync(0xffffffffu, s, o); if (lane >= o) s += up; }
            lg[i] = s - b;
            lg[i + 1] = s;
        } else if (warp == 1) {
#pragma unroll
            for (int k = 0; k < 2; ++k) { const int i = lane + 32 * k; be[i] = i < count ? beta[(int64_t)(t0 + i) * H + h] : 0.f; }
        }
        __syncthreads();
        const ChunkScratch out(scratch, (int64_t)blockIdx.x * H + h);
        if (threadIdx.x < CH) {
            out.eg[threadIdx.x] = expf(lg[threadIdx.x]);
            out.er[threadIdx.x] = expf(lg[CH - 1] - lg[threadIdx.x]);
        }
        for (int idx = threadIdx.x; idx < CH * CH; idx += blockDim.x) {
            const int i = idx >> 6, j = idx & 63;
            const float f = j <= i ? expf(lg[i] - lg[j]) : 0.f;
            out.p[idx] = j <= i ? f * QK[i * CHP + j] : 0.f;
            A[i * CHP + j] = j < i ? be[i] * f * KK[i * CHP + j] : 0.f;
        }
        __syncthreads();
        // diagonal blocks: a column of the inverse a thread, by substitution, in registers
        if (threadIdx.x < 64) {
            float t[16];
            const int db = (threadIdx.x >> 4) * 16, dc = threadIdx.x & 15;
#pragma unroll
            for (int i = 0; i < 16; ++i) {
                float v = i == dc ? 1.f : 0.f;
#pragma unroll
                for (int m = 0; m < i; ++m) v = fmaf(-A[(db + i) * CHP + db + m], t[m], v);
                t[i] = v;
                T[(db + i) * CHP + db + dc] = v;
            }
        }
        __syncthreads();
        // the blocks below: T_ij = -T_ii (sum over j <= m < i of A_im T_mj), one diagonal of blocks after the other
        for (int w = 1; w < 4; ++w) {
            const int n = (4 - w) * 256;                       // entries of the blocks (i, i - w)
            for (int idx = threadIdx.x; idx < n; idx += blockDim.x) {
                const int bi = w + (idx >> 8), bj = bi - w, r = (idx >> 4) & 15, c = idx & 15;
                float v = 0.f;
                for (int mb = bj * 16; mb < bi * 16; mb += 16) {
                    float part = 0.f;
#pragma unroll
                    for (int m = 0; m < 16; ++m) part = fmaf(A[(bi * 16 + r) * CHP + mb + m], T[(mb + m) * CHP + bj * 16 + c], part);
                    v += part;
                }
                X[idx] = v;
            }
            __syncthreads();
            for (int idx = threadIdx.x; idx < n; idx += blockDim.x) {
                const int bi = w + (idx >> 8), bj = bi - w, r = (idx >> 4) & 15, c = idx & 15;
                float v = 0.f;
#pragma unroll
                for (int m = 0; m < 16; ++m) v = fmaf(T[(bi * 16 + r) * CHP + bi * 16 + m], X[(idx & ~255) + m * 16 + c], v);
                T[(bi * 16 + r) * CHP + bj * 16 + c] = -v;
            }
            __syncthreads();
        }
        for (int idx = threadIdx.x; idx < CH * CH; idx += blockDim.x) {
            const int i = idx >> 6, j = idx & 63;
            out.tb[idx] = j <= i ? T[i * CHP + j] * be[j] : 0.f;
        }
    }
}

template <int DT>
__global__ void __launch_bounds__(256) delta_chunk_scan_kernel(const float* __restrict__ qn, const float* __restrict__ kn, const float* __restrict__ vn,
                                                               const int* __restrict__ row_q_start, const int* __restrict__ row_q_len,
                                                               const int* __restrict__ state_slots, int min_len, const float* __restrict__ scratch,
                                                               float* __restrict__ state, float* __restrict__ out, int H, int G, int D, int Dv) {
    constexpr int DP = DT + 4;
    extern __shared__ __align__(16) float sm[];
    float* KQ = sm;                                            // two stages of K [64][DP] | Q [64][DP] | V [64][16] | e^G [64] | e^{G_C - G} [64]
    constexpr int STAGE = 2 * CH * DP + CH * COLS + 2 * CH;
    float* TB = KQ + 2 * STAGE;                                // [64][68]
    float* P = TB + CH * CHP;                                  // [64][68]
    float* S = P + CH * CHP;                                   // the state's columns [16][DP]
    float* R = S + COLS * DP;                                  // V - e^G K S, column by column [16][68]
    float* U = R + COLS * CHP;                                 // [16][68]
    float* UE = U + COLS * CHP;                                // U with e^{G_C - G} [16][68]
    __shared__ int s_first;
    pdl_enter();
    const int row = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * COLS;
    const int n = row_q_len[row], chunks = chunks_of(n, min_len);
    if (chunks == 0) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (warp == 0) {                                           // where the row's chunks begin in the scratch memory
        int first = 0;
        for (int r = lane; r < row; r += 32) first += chunks_of(row_q_len[r], min_len);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) first += __shfl_xor_sync(0xffffffffu, first, o);
        if (lane == 0) s_first = first;
    }
    __syncthreads();
    const int t0 = row_q_start[row], g = h / (H / G);
    const int64_t first = s_first;
    float* sp = state + ((int64_t)state_slots[row] * H + h) * Dv * D;

    // the thread's part of the state, for warps 0 .. 3: entries d4 .. d4 + 3 of JT columns
    constexpr int JT = DT == 128 ? 4 : 2;
    const int d4 = (DT == 128 ? warp : warp & 1) * 32 + (lane & 7) * 4, jl = (lane >> 3) + (DT == 128 ? 0 : (warp >> 1) * 8);
    unsigned long long s_lo[JT], s_hi[JT];
    if (warp < 4) {
#pragma unroll
        for (int jj = 0; jj < JT; ++jj) {
            const int j = jl + 4 * jj;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (j0 + j < Dv && d4 < D) v = *reinterpret_cast<const float4*>(sp + (int64_t)(j0 + j) * D + d4);
            *reinterpret_cast<float4*>(S + j * DP + d4) = v;
            s_lo[jj] = pack2(v.x, v.y);
            s_hi[jj] = pack2(v.z, v.w);
        }
    }
    auto issue_keys = [&](int c) {                             // every thread commits one group, also an empty one
        if (c < chunks) {
            float* st = KQ + (c & 1) * STAGE;
            const int64_t tf = t0 + c * CH;
            const int count = min(CH, n - c * CH);
            copy_rows<DT>(st, kn + (tf * G + g) * D, (int64_t)G * D, D, count);
            copy_rows<DT>(st + CH * DP, qn + (tf * G + g) * D, (int64_t)G * D, D, count);
            float* v = st + 2 * CH * DP;
            for (int i = threadIdx.x; i < CH * COLS; i += 256) {
                const int t = i >> 4, j = i & 15;
                const bool on = t < count && j0 + j < Dv;
                copy4(v + i, on ? vn + ((tf + t) * H + h) * Dv + j0 + j : vn, on);
            }
            if (threadIdx.x < 32) {
                const float* eg = ChunkScratch(const_cast<float*>(scratch), (first + c) * H + h).eg;      // e^G and e^{G_C - G} lie side by side
                copy16(v + CH * COLS + threadIdx.x * 4, eg + threadIdx.x * 4, true);
            }
        }
        copy_commit();
    };
    auto issue_squares = [&](int c) {
        const ChunkScratch in(const_cast<float*>(scratch), (first + c) * H + h);
        for (int i = threadIdx.x; i < CH * CH / 4; i += 256) {
            const int r = i >> 4, m = (i & 15) * 4;
            copy16(TB + r * CHP + m, in.tb + i * 4, true);
            copy16(P + r * CHP + m, in.p + i * 4, true);
        }
        copy_commit();
    };
    issue_keys(0);
    // rows and columns of a lane: in the products with S four rows and two columns (warps 0 .. 3 the keys, 4 .. 7 the queries, 16 rows
    // a warp), in U two rows and two columns (8 rows a warp); always interleaved over the lanes
    const int half = warp >> 2, r1 = (warp & 3) * 16 + (lane >> 3), c1 = lane & 7;
    // (warps w and w + 4 share a scheduler: short and long rows of the triangle are dealt to them in pairs)
    const int rw = half ? 7 - (warp & 3) : (warp & 3), r2 = rw * 8 + (lane >> 3);
    for (int c = 0; c < chunks; ++c) {
        copy_wait<0>();                                        // keys and queries of this chunk
        __syncthreads();                                       // ... of every thread; S of the chunk before; TB and P are free
        issue_squares(c);
        issue_keys(c + 1);
        const float* st = KQ + (c & 1) * STAGE;
        const float* V = st + 2 * CH * DP;
        const float* eg = V + CH * COLS;
        const float* er = eg + CH;
        unsigned long long acc[4][2];
        float o[4][2];
        {
            const float* L = st + half * CH * DP;
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[i][0] = acc[i][1] = 0ull;
#pragma unroll 4
            for (int d = 0; d < DT; d += 4) {
                const Quad b0 = quad(S + c1 * DP + d), b1 = quad(S + (c1 + 8) * DP + d);
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const Quad a = quad(L + (r1 + 4 * i) * DP + d);
                    fma2(acc[i][0], a.lo, b0.lo); fma2(acc[i][0], a.hi, b0.hi);
                    fma2(acc[i][1], a.lo, b1.lo); fma2(acc[i][1], a.hi, b1.hi);
                }
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int r = r1 + 4 * i;
                const float e = eg[r];
#pragma unroll
                for (int k = 0; k < 2; ++k) {
                    o[i][k] = e * sum2(acc[i][k]);
                    if (half == 0) R[(c1 + 8 * k) * CHP + r] = V[r * COLS + c1 + 8 * k] - o[i][k];
                }
            }
        }
        copy_wait<1>();                                        // TB and P of this chunk
        __syncthreads();
        {
            unsigned long long u[2][2] = {{0ull, 0ull}, {0ull, 0ull}};
            const int end = rw * 8 + 8;                        // no row of the warp reads beyond its diagonal
#pragma unroll 2
            for (int m = 0; m < end; m += 4) {
                const Quad b0 = quad(R + c1 * CHP + m), b1 = quad(R + (c1 + 8) * CHP + m);
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const Quad a = quad(TB + (r2 + 4 * i) * CHP + m);
                    fma2(u[i][0], a.lo, b0.lo); fma2(u[i][0], a.hi, b0.hi);
                    fma2(u[i][1], a.lo, b1.lo); fma2(u[i][1], a.hi, b1.hi);
                }
            }
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int r = r2 + 4 * i;
                const float e = er[r];
#pragma unroll
                for (int k = 0; k < 2; ++k) {
                    const float v = sum2(u[i][k]);
                    U[(c1 + 8 * k) * CHP + r] = v;
                    UE[(c1 + 8 * k) * CHP + r] = e * v;
                }
            }
        }
        __syncthreads();
        if (half == 0) {
            // the state: its columns times the chunk's whole decay, plus keys times U
            const float total = eg[CH - 1];
            const unsigned long long tt = pack2(total, total);
            unsigned long long n_lo[JT], n_hi[JT];
#pragma unroll
            for (int jj = 0; jj < JT; ++jj) { n_lo[jj] = n_hi[jj] = 0ull; fma2(n_lo[jj], s_lo[jj], tt); fma2(n_hi[jj], s_hi[jj], tt); }
#pragma unroll 2
            for (int i = 0; i < CH; i += 4) {
                float4 u[JT];
#pragma unroll
                for (int jj = 0; jj < JT; ++jj) u[jj] = *reinterpret_cast<const float4*>(UE + (jl + 4 * jj) * CHP + i);
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    const Quad key = quad(st + (i + k) * DP + d4);
#pragma unroll
                    for (int jj = 0; jj < JT; ++jj) {
                        const float x = k == 0 ? u[jj].x : k == 1 ? u[jj].y : k == 2 ? u[jj].z : u[jj].w;
                        const unsigned long long xx = pack2(x, x);
                        fma2(n_lo[jj], key.lo, xx);
                        fma2(n_hi[jj], key.hi, xx);
                    }
                }
            }
#pragma unroll
            for (int jj = 0; jj < JT; ++jj) {
                s_lo[jj] = n_lo[jj];
                s_hi[jj] = n_hi[jj];
                *reinterpret_cast<ulonglong2*>(S + (jl + 4 * jj) * DP + d4) = make_ulonglong2(n_lo[jj], n_hi[jj]);
            }
        } else {
            // the outputs: what the state gave the queries, plus P U
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[i][0] = acc[i][1] = 0ull;
            const int end = (warp & 3) * 16 + 16;
#pragma unroll 2
            for (int m = 0; m < end; m += 4) {
                const Quad b0 = quad(U + c1 * CHP + m), b1 = quad(U + (c1 + 8) * CHP + m);
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const Quad a = quad(P + (r1 + 4 * i) * CHP + m);
                    fma2(acc[i][0], a.lo, b0.lo); fma2(acc[i][0], a.hi, b0.hi);
                    fma2(acc[i][1], a.lo, b1.lo); fma2(acc[i][1], a.hi, b1.hi);
                }
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int t = c * CH + r1 + 4 * i;
                if (t >= n) continue;
                float* dst = out + ((int64_t)(t0 + t) * H + h) * Dv + j0;
#pragma unroll
                for (int k = 0; k < 2; ++k)
                    if (j0 + c1 + 8 * k < Dv) dst[c1 + 8 * k] = o[i][k] + sum2(acc[i][k]);
            }
        }
    }
    if (warp < 4) {
#pragma unroll
        for (int jj = 0; jj < JT; ++jj) {
            const int j = jl + 4 * jj;
            if (j0 + j >= Dv || d4 >= D) continue;
            const float2 a = unpack2(s_lo[jj]), b = unpack2(s_hi[jj]);
            *reinterpret_cast<float4*>(sp + (int64_t)(j0 + j) * D + d4) = make_float4(a.x, a.y, b.x, b.y);
        }
    }
}

template <int DT>
static int launch_chunks(const float* qn, const float* kn, const float* vn, const float* beta, const float* log_decay, const int* row_q_start,
                         const int* row_q_len, const int* state_slots, float* state, float* out, float* scratch, int max_chunks, int num_rows,
                         int min_len, int H, int G, int D, int Dv, cudaStream_t stream) {
    const size_t prep = (size_t)(2 * CH * (DT + 4) + 2 * CH * CHP + 3 * 256) * sizeof(float);      // two blocks on an SM
    const size_t scan = (size_t)(2 * (2 * CH * (DT + 4) + CH * COLS + 2 * CH) + 2 * CH * CHP + COLS * (DT + 4) + 3 * COLS * CHP) * sizeof(float);
    cudaError_t e = cudaFuncSetAttribute(delta_chunk_prep_kernel<DT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)prep);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_chunk_scan_kernel<DT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)scan);
    if (e != cudaSuccess) return (int)e;
    const int rc = launch_kernel(delta_chunk_prep_kernel<DT>, dim3(max_chunks, G), dim3(256), prep, stream, qn, kn, beta, log_decay, row_q_start,
                                 row_q_len, num_rows, min_len, scratch, H, G, D);
    if (rc) return rc;
    return launch_kernel(delta_chunk_scan_kernel<DT>, dim3(num_rows, H, (Dv + COLS - 1) / COLS), dim3(256), scan, stream, qn, kn, vn, row_q_start,
                         row_q_len, state_slots, min_len, (const float*)scratch, state, out, H, G, D, Dv);
}

// Floats of scratch memory for one (chunk, head); tokens a chunk.
extern "C" int mie_delta_chunk_floats(void) { return 2 * CH * CH + 2 * CH; }
extern "C" int mie_delta_chunk_tokens(void) { return CH; }

// qn, kn: float32 [T, G, D]; vn, out: [T, H, Dv]; beta, log_decay (not positive): [T, H]; state [slots, H, Dv, D].  D a multiple of 4 up to
// 128, everything 16-byte aligned.  max_chunks: no fewer than the chunks of all rows with min_len tokens or more; scratch holds
// max_chunks * H times mie_delta_chunk_floats() floats.
extern "C" int mie_delta_chunks(const float* qn, const float* kn, const float* vn, const float* beta, const float* log_decay,
                                const int* row_q_start, const int* row_q_len, const int* state_slots, float* state, float* out, float* scratch,
                                int max_chunks, int num_rows, int min_len, int H, int G, int D, int Dv, cudaStream_t stream) {
    if (num_rows <= 0 || max_chunks <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || D <= 0 || D % 4 || Dv <= 0 || min_len < 1) return MIE_ERR_BAD_ARG;
    if (D > 128 || H > 65535) return MIE_ERR_TOO_LARGE;
    if ((reinterpret_cast<uintptr_t>(qn) | reinterpret_cast<uintptr_t>(kn) | reinterpret_cast<uintptr_t>(state) | reinterpret_cast<uintptr_t>(scratch)) & 15)
        return MIE_ERR_BAD_ARG;
    if (D <= 64)
        return launch_chunks<64>(qn, kn, vn, beta, log_decay, row_q_start, row_q_len, state_slots, state, out, scratch, max_chunks, num_rows, min_len, H, G, D, Dv, stream);
    return launch_chunks<128>(qn, kn, vn, beta, log_decay, row_q_start, row_q_len, state_slots, state, out, scratch, max_chunks, num_rows, min_len, H, G, D, Dv, stream);
}
