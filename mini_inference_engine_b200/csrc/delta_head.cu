// The gated delta rule with one decay per head: what surrounds the recurrence of portions (delta_rule.cu, delta_chunk.cu), and a single
// token's whole step.
//
// The input projection leaves float32 rows  proj[t] = [ q: G x D | k: G x D | v: H x Dv | gate: H x Dv | a: H | b: H | ... ].
//
//   prepare   per token: the short causal convolution over time of q, k and v and silu, q and k made unit vectors per head (q also scaled),
//             k . q per key head, beta = sigmoid(b), log g = -exp(A_log[h]) softplus(a + dt_bias) and g.  A warp takes a head of a few
//             consecutive tokens, four channels a lane, so that an input is read from memory once and its later uses hit the cache.
//   remember  the last inputs of every row's portion go into its convolution state.
//   step      rows of one new token: convolution, unit vectors, gates, S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q, the
//             head's norm and the output gate in one launch, a block per (row, head).  The head's state travels into shared memory while the
//             convolution is worked out, and is written back from registers.
//
// The convolution state is a ring: [slot, K, C] float32, entry (position mod K) holds the inputs at that position.  A token reads the K - 1
// entries before its own and writes its own, so a step needs no shift and no block waits for another's reads.  A fresh slot
// is zero, which is what stands in front of a sequence.  Slot 0 is scratch.  taps: [K, C], the last row for the token itself.
#include "common.cuh"

__device__ __forceinline__ float softplus_of(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float silu_of(float x) { return __fdividef(x, 1.0f + __expf(-fmaxf(x, -80.f))); }      // (the bound keeps the divisor in the fast division's range)

struct HeadParams {
    const float* proj; int64_t stride;
    const float* taps; float* ring;
    const int* positions; const int* token_row; const int* row_q_start; const int* row_q_len; const int* state_slots;
    const float* a_log; const float* dt_bias;
    int H, G, D, Dv, K; float q_scale, unit_eps;
};

template <int VEC> __device__ __forceinline__ void load_vec(float* v, const float* p) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(p);
    else v[0] = *p;
}
template <int VEC> __device__ __forceinline__ void store_vec(float* p, const float* v) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = *reinterpret_cast<const float4*>(v);
    else *p = v[0];
}

// VEC channels from c on of token t, `local` tokens into its row's portion, at position `pos`: the convolution's output behind silu.
// KT: the number of taps where it is known at compile time (all inputs are then asked for together), 0: p.K.
template <int VEC, int KT>
__device__ __forceinline__ void conv_silu(float* y, const HeadParams& p, const float* ring_slot, int t, int local, int pos, int c) {
    const int K = KT > 0 ? KT : p.K, C = 2 * p.G * p.D + p.H * p.Dv, m = K > 1 ? pos % K : 0;
#pragma unroll
    for (int e = 0; e < VEC; ++e) y[e] = 0.f;
    auto input = [&](float* x, int back) {
        int entry = m - back;
        if (entry < 0) entry += K;
        load_vec<VEC>(x, back <= local ? p.proj + (int64_t)(t - back) * p.stride + c : ring_slot + (int64_t)entry * C + c);
    };
    auto add = [&](const float* x, const float* w) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] = fmaf(w[e], x[e], y[e]);
    };
    if constexpr (KT > 0) {
        float x[KT][VEC], w[KT][VEC];
#pragma unroll
        for (int i = 0; i < KT; ++i) { input(x[i], KT - 1 - i); load_vec<VEC>(w[i], p.taps + (int64_t)i * C + c); }
#pragma unroll
        for (int i = 0; i < KT; ++i) add(x[i], w[i]);
    } else {
        for (int i = 0; i < K; ++i) {
            float x[VEC], w[VEC];
            input(x, K - 1 - i);
            load_vec<VEC>(w, p.taps + (int64_t)i * C + c);
            add(x, w);
        }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) y[e] = silu_of(y[e]);
}

// Work items of a token: G heads of q and k together, H heads of v, and one for the gates.  NCH: pieces of 32 * VEC channels a key head.
template <int VEC, int NCH, int KT>
__global__ void __launch_bounds__(256) delta_head_prepare_kernel(const HeadParams p, float* __restrict__ qn, float* __restrict__ kn, float* __restrict__ vn,
                                                                 float* __restrict__ beta, float* __restrict__ decay, float* __restrict__ log_decay,
                                                                 float* __restrict__ kq, int num_tokens, int tile) {
    pdl_enter();
    const int lane = threadIdx.x & 31, unit = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const int H = p.H, G = p.G, D = p.D, Dv = p.Dv, C = 2 * G * D + H * Dv;
    if (unit > G + H) return;
    const int end = min(num_tokens, ((int)blockIdx.x + 1) * tile);
    for (int t = blockIdx.x * tile; t < end; ++t) {
        if (unit == G + H) {                                   // decays and step sizes
            const float* z = p.proj + (int64_t)t * p.stride + C + H * Dv;
            for (int h = lane; h < H; h += 32) {
                const float ld = -expf(p.a_log[h]) * softplus_of(z[h] + p.dt_bias[h]);
                const int64_t at = (int64_t)t * H + h;
                decay[at] = expf(ld);
                log_decay[at] = fmaxf(ld, -100.f);             // (e^-100 is nothing in 32 bits; the bound keeps sums of these, and their differences, sharp)
                beta[at] = 1.0f / (1.0f + expf(-z[H + h]));
            }
            continue;
        }
        const int row = p.token_row[t], local = t - p.row_q_start[row], pos = p.positions[t];
        const float* ring_slot = p.ring + (int64_t)p.state_slots[row] * p.K * C;
        if (unit >= G) {
            const int h = unit - G;
            for (int d = lane * VEC; d < Dv; d += 32 * VEC) {
                float y[VEC];
                conv_silu<VEC, KT>(y, p, ring_slot, t, local, pos, 2 * G * D + h * Dv + d);
                store_vec<VEC>(vn + ((int64_t)t * H + h) * Dv + d, y);
            }
            continue;
        }
        float q[NCH][VEC], k[NCH][VEC], qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
        for (int n = 0; n < NCH; ++n) {
            const int d = (n * 32 + lane) * VEC;
#pragma unroll
            for (int e = 0; e < VEC; ++e) q[n][e] = k[n][e] = 0.f;
            if (d < D) {
                conv_silu<VEC, KT>(q[n], p, ring_slot, t, local, pos, unit * D + d);
                conv_silu<VEC, KT>(k[n], p, ring_slot, t, local, pos, (G + unit) * D + d);
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                qq = fmaf(q[n][e], q[n][e], qq);
                kk = fmaf(k[n][e], k[n][e], kk);
                qk = fmaf(q[n][e], k[n][e], qk);
            }
        }
        const float qs = p.q_scale / sqrtf(warp_sum(qq) + p.unit_eps), ks = 1.0f / sqrtf(warp_sum(kk) + p.unit_eps);
        qk = warp_sum(qk);
        const int64_t at = ((int64_t)t * G + unit) * D;
#pragma unroll
        for (int n = 0; n < NCH; ++n) {
            const int d = (n * 32 + lane) * VEC;
            if (d >= D) continue;
#pragma unroll
            for (int e = 0; e < VEC; ++e) { q[n][e] *= qs; k[n][e] *= ks; }
            store_vec<VEC>(qn + at + d, q[n]);
            store_vec<VEC>(kn + at + d, k[n]);
        }
        if (lane == 0) kq[(int64_t)t * G + unit] = qk * qs * ks;
    }
}

// The last min(n, K - 1) inputs of every row of n new tokens into its ring.
__global__ void delta_head_remember_kernel(const HeadParams p) {
    pdl_enter();
    const int row = blockIdx.y, n = p.row_q_len[row], t_end = p.row_q_start[row] + n, C = 2 * p.G * p.D + p.H * p.Dv;
    float* ring_slot = p.ring + (int64_t)p.state_slots[row] * p.K * C;
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= C) return;
    for (int t = max(t_end - n, t_end - (p.K - 1)); t < t_end; ++t)
        ring_slot[(int64_t)(p.positions[t] % p.K) * C + c] = p.proj[(int64_t)t * p.stride + c];
}

__device__ __forceinline__ void copy_async(float* dst, const float* src, int bytes16) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    if (bytes16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
    else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}

#define STEP_THREADS 256

// One new token a row.  VEC entries of a column of the state go together; eight lanes share a column, NM pieces each.
template <typename T, int VEC, int NM, int KT>
__global__ void __launch_bounds__(STEP_THREADS) delta_head_step_kernel(const HeadParams p, float* __restrict__ state, const float* __restrict__ norm,
                                                                       T* __restrict__ out, float eps) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[2][32];
    __shared__ float s_beta, s_decay, s_qs, s_ks, s_kq;
    pdl_enter();
    const int h = blockIdx.x, row = blockIdx.y;
    const int H = p.H, G = p.G, D = p.D, Dv = p.Dv, C = 2 * G * D + H * Dv, g = h / (H / G);
    if (p.row_q_len[row] != 1) return;
    const int Dp = (D + 3) / 4 * 4, Dvp = (Dv + 3) / 4 * 4;
    float* q = sm;                                             // [D], [D], [Dv], [Dv], then the head's state [Dv][D]
    float* k = q + Dp;
    float* v = k + Dp;
    float* o = v + Dvp;
    float* S = o + Dvp;
    const int t = p.row_q_start[row], pos = p.positions[t];
    const int64_t slot = p.state_slots[row];
    float* sp = state + (slot * H + h) * Dv * D;
    for (int i = threadIdx.x * VEC; i < Dv * D; i += STEP_THREADS * VEC) copy_async(S + i, sp + i, VEC == 4);
    asm volatile("cp.async.commit_group;" ::: "memory");
    float* ring_slot = p.ring + slot * p.K * C;
    const float* x = p.proj + (int64_t)t * p.stride;
    const bool keeps_keys = h % (H / G) == 0;                  // the first head of a group also remembers the group's q and k inputs
    for (int i = threadIdx.x * VEC; i < 2 * D + Dv; i += STEP_THREADS * VEC) {
        const int seg = i < D ? 0 : i < 2 * D ? 1 : 2;
        const int d = i - seg * D, c = seg == 0 ? g * D + d : seg == 1 ? (G + g) * D + d : 2 * G * D + h * Dv + d;
        float y[VEC], in[VEC];
        conv_silu<VEC, KT>(y, p, ring_slot, t, 0, pos, c);
        store_vec<VEC>((seg == 0 ? q : seg == 1 ? k : v) + d, y);
        if (p.K > 1 && (seg == 2 || keeps_keys)) {
            load_vec<VEC>(in, x + c);
            store_vec<VEC>(ring_slot + (int64_t)(pos % p.K) * C + c, in);
        }
    }
    if (threadIdx.x == STEP_THREADS - 1) {
        const float* z = x + C + H * Dv;
        s_decay = expf(-expf(p.a_log[h]) * softplus_of(z[h] + p.dt_bias[h]));
        s_beta = 1.0f / (1.0f + expf(-z[H + h]));
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (warp == 0) {
        float qq = 0.f, kk = 0.f, qk = 0.f;
        for (int d = lane; d < D; d += 32) { qq = fmaf(q[d], q[d], qq); kk = fmaf(k[d], k[d], kk); qk = fmaf(q[d], k[d], qk); }
        qq = warp_sum(qq); kk = warp_sum(kk); qk = warp_sum(qk);
        if (lane == 0) {
            s_qs = p.q_scale / sqrtf(qq + p.unit_eps);
            s_ks = 1.0f / sqrtf(kk + p.unit_eps);
            s_kq = qk * s_qs * s_ks;
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const float qs = s_qs, ks = s_ks, kq = s_kq, decay = s_decay, beta = s_beta;
    const int l = threadIdx.x & 7;
    float kr[NM][VEC], qr[NM][VEC];
#pragma unroll
    for (int m = 0; m < NM; ++m) {
        const int d = (l + 8 * m) * VEC;
#pragma unroll
        for (int e = 0; e < VEC; ++e) { kr[m][e] = d < D ? k[d + e] * ks : 0.f; qr[m][e] = d < D ? q[d + e] * qs : 0.f; }
    }
    float ss = 0.f;
    for (int base = 0; base < Dv; base += STEP_THREADS / 8) {  // every lane of a warp goes round equally often
        const int j = base + (threadIdx.x >> 3);
        float s[NM][VEC], r1 = 0.f, r2 = 0.f;
#pragma unroll
        for (int m = 0; m < NM; ++m) {
            const int d = (l + 8 * m) * VEC;
            if (j < Dv && d < D) load_vec<VEC>(s[m], S + j * D + d);
            else
#pragma unroll
                for (int e = 0; e < VEC; ++e) s[m][e] = 0.f;
#pragma unroll
            for (int e = 0; e < VEC; ++e) { r1 = fmaf(s[m][e], kr[m][e], r1); r2 = fmaf(s[m][e], qr[m][e], r2); }
        }
#pragma unroll
        for (int w = 4; w > 0; w >>= 1) { r1 += __shfl_xor_sync(0xffffffffu, r1, w); r2 += __shfl_xor_sync(0xffffffffu, r2, w); }
        if (j >= Dv) continue;
        const float u = beta * (v[j] - decay * r1), y = fmaf(u, kq, decay * r2);
#pragma unroll
        for (int m = 0; m < NM; ++m) {
            const int d = (l + 8 * m) * VEC;
            if (d >= D) continue;
#pragma unroll
            for (int e = 0; e < VEC; ++e) s[m][e] = fmaf(kr[m][e], u, decay * s[m][e]);
            store_vec<VEC>(sp + (int64_t)j * D + d, s[m]);
        }
        if (l == 0) { o[j] = y; ss = fmaf(y, y, ss); }
    }
    ss = warp_sum(ss);
    if (lane == 0) red[0][warp] = ss;
    __syncthreads();
    const float rs = 1.0f / sqrtf(warp_sum(lane < STEP_THREADS / 32 ? red[0][lane] : 0.f) / (float)Dv + eps);
    for (int j = threadIdx.x; j < Dv; j += STEP_THREADS)
        out[((int64_t)t * H + h) * Dv + j] = from_f32<T>(o[j] * rs * norm[j] * silu_of(x[C + h * Dv + j]));
}

static int head_params(HeadParams& p, const float* proj, long long stride, const float* taps, float* ring, const int* positions, const int* token_row,
                       const int* row_q_start, const int* row_q_len, const int* state_slots, const float* a_log, const float* dt_bias, int H, int G,
                       int D, int Dv, int K, float q_scale, float unit_eps) {
    if (H <= 0 || G <= 0 || H % G || D <= 0 || Dv <= 0 || K < 1) return MIE_ERR_BAD_ARG;
    if (D > 512) return MIE_ERR_TOO_LARGE;
    p = HeadParams{proj, (int64_t)stride, taps, ring, positions, token_row, row_q_start, row_q_len, state_slots, a_log, dt_bias, H, G, D, Dv, K, q_scale, unit_eps};
    return 0;
}
// whether every head starts at a whole 16-byte piece
static bool head_vec(const HeadParams& p) {
    return p.D % 4 == 0 && p.Dv % 4 == 0 && p.stride % 4 == 0 &&
           ((reinterpret_cast<uintptr_t>(p.proj) | reinterpret_cast<uintptr_t>(p.taps) | reinterpret_cast<uintptr_t>(p.ring)) & 15) == 0;
}

// All outputs float32: qn, kn [T, G, D], vn [T, H, Dv], beta, decay, log_decay [T, H], kq [T, G].
extern "C" int mie_delta_head_prepare(const float* proj, long long stride, const float* taps, float* ring, const int* positions, const int* token_row,
                                      const int* row_q_start, const int* state_slots, const float* a_log, const float* dt_bias, float* qn, float* kn,
                                      float* vn, float* beta, float* decay, float* log_decay, float* kq, int num_tokens, int H, int G, int D, int Dv,
                                      int K, float q_scale, float unit_eps, cudaStream_t stream) {
    if (num_tokens <= 0) return 0;
    HeadParams p;
    const int rc = head_params(p, proj, stride, taps, ring, positions, token_row, row_q_start, nullptr, state_slots, a_log, dt_bias, H, G, D, Dv, K, q_scale, unit_eps);
    if (rc) return rc;
    const int tile = num_tokens >= 512 ? 8 : num_tokens >= 128 ? 2 : 1;
    const dim3 grid((num_tokens + tile - 1) / tile, (G + H + 1 + 7) / 8);
#define PREPARE(VEC, NCH, KT) launch_kernel(delta_head_prepare_kernel<VEC, NCH, KT>, grid, dim3(256), 0, stream, p, qn, kn, vn, beta, decay, log_decay, kq, num_tokens, tile)
    const bool vec = head_vec(p) && ((reinterpret_cast<uintptr_t>(qn) | reinterpret_cast<uintptr_t>(kn) | reinterpret_cast<uintptr_t>(vn)) & 15) == 0;
    if (vec && D <= 128) return K == 4 ? PREPARE(4, 1, 4) : PREPARE(4, 1, 0);
    if (vec) return PREPARE(4, 4, 0);
    return D <= 128 ? PREPARE(1, 4, 0) : PREPARE(1, 16, 0);
#undef PREPARE
}

extern "C" int mie_delta_head_remember(const float* proj, long long stride, float* ring, const int* positions, const int* row_q_start, const int* row_q_len,
                                       const int* state_slots, int num_rows, int H, int G, int D, int Dv, int K, cudaStream_t stream) {
    if (num_rows <= 0 || K <= 1) return 0;
    if (num_rows > 65535) return MIE_ERR_TOO_LARGE;
    HeadParams p;
    const int rc = head_params(p, proj, stride, nullptr, ring, positions, nullptr, row_q_start, row_q_len, state_slots, nullptr, nullptr, H, G, D, Dv, K, 0.f, 0.f);
    if (rc) return rc;
    const int C = 2 * G * D + H * Dv;
    return launch_kernel(delta_head_remember_kernel, dim3((C + 127) / 128, num_rows), dim3(128), 0, stream, p);
}

// Bytes of shared memory the step needs for heads of this size (the caller asks before it chooses this path: at most 200 KB).
extern "C" int mie_delta_head_step_bytes(int D, int Dv) {
    return (int)(((int64_t)D * Dv + 2 * ((D + 3) / 4 * 4) + 2 * ((Dv + 3) / 4 * 4)) * (int64_t)sizeof(float));
}

// out [T, H, Dv] in the activation type; rows with another number of new tokens than one are left alone.  norm: float32 [Dv].
extern "C" int mie_delta_head_step(const float* proj, long long stride, const float* taps, float* ring, const int* positions, const int* row_q_start,
                                   const int* row_q_len, const int* state_slots, const float* a_log, const float* dt_bias, float* state,
                                   const float* norm, void* out, int tag, int num_rows, int H, int G, int D, int Dv, int K, float q_scale,
                                   float unit_eps, float eps, cudaStream_t stream) {
    if (num_rows <= 0) return 0;
    HeadParams p;
    const int rc = head_params(p, proj, stride, taps, ring, positions, nullptr, row_q_start, row_q_len, state_slots, a_log, dt_bias, H, G, D, Dv, K, q_scale, unit_eps);
    if (rc) return rc;
    const int smem = mie_delta_head_step_bytes(D, Dv);
    if ((int64_t)D * Dv > 51200 || smem > 200 * 1024 || num_rows > 65535) return MIE_ERR_TOO_LARGE;
    const bool vec = head_vec(p) && (reinterpret_cast<uintptr_t>(state) & 15) == 0;
#define STEP(T, VEC, NM, KT)                                                                                                                          \
    do {                                                                                                                                          \
        const cudaError_t e = cudaFuncSetAttribute(delta_head_step_kernel<T, VEC, NM, KT>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);         \
        if (e != cudaSuccess) return (int)e;                                                                                                      \
        return launch_kernel(delta_head_step_kernel<T, VEC, NM, KT>, dim3(H, num_rows), dim3(STEP_THREADS), (size_t)smem, stream, p, state, norm, (T*)out, eps); \
    } while (0)
#define STEPS(T)                                                                          \
    do {                                                                                  \
        if (vec && D <= 128 && K == 4) STEP(T, 4, 4, 4);                                  \
        if (vec && D <= 128) STEP(T, 4, 4, 0);                                            \
        if (vec) STEP(T, 4, 16, 0);                                                       \
        if (D <= 128) STEP(T, 1, 16, 0);                                                  \
        STEP(T, 1, 64, 0);                                                                   \
    } while (0)
    if (tag == MIE_F32) STEPS(float);
    if (tag == MIE_BF16) STEPS(bf16);
#undef STEPS
#undef STEP
    return MIE_ERR_BAD_ARG;
}
