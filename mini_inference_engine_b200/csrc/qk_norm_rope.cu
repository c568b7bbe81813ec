// What happens to a fused q|k|v projection between the product and attention, for mixers whose queries and keys
// are normed as whole projections and whose heads may be narrower than the pages that hold them:
//
//   qkv[t] = [ q: H x D | k: G x D | v: G x Dv | anything else ]         (row stride `qkv_stride`)
//   q <- q * rsqrt(mean over all H*D entries of q^2 + eps) * qw[:]       (if qw; the same for k with kw over G*D)
//   rotation (rotate-half pairing over the first `rot` dims of every head): with a = position * freq[i],
//       (x_i, x_{i + rot/2}) <- (x_i cos a - x_{i + rot/2} sin a,  x_{i + rot/2} cos a + x_i sin a)
//   q[h] <- q[h] * q_scale * temp[h]    (if temp: a per-head factor on the scores, folded into the query)
//   k    <- k * k_scale
//   q is written to q_out [T, H, DP], k and v to their cache slot [page, G, page_size, DP]; DP >= max(D, Dv), the tail of
//   every head is zero, so that kernels written for one head size serve heads whose key and value sizes differ.
//
// Options: `head_norm` -- the RMS statistics are per head (over its D entries) and qw / kw hold D weights shared by all heads, or
// are null (heads of unit root mean square; a statistic over whole pairs is the same before and after the rotation, which
// changes no pair's length, so this also serves designs that norm the rotated heads);
// `v_freq` (Dv/2 float32, or null) -- v is rotated too, over all its Dv entries in the same pairing, before it is stored;
// `v_cache` null -- there are no values of their own (the keys serve as values): rows hold q and k only, and only k is stored;
// `interleaved` -- the rotation pairs entry 2i with 2i + 1 instead of i with i + rot/2 (the same angle position * freq[i]);
// `temp_coef`, `temp_every` -- the query of position p is also multiplied by 1 + temp_coef * ln(floor((p + 1) / temp_every) + 1)
// (a temperature that grows with the position; temp_every <= 0: none).
//
// `freq` holds rot/2 float32 frequencies (the host computes them, with whatever rescaling the model asks for);
// angles, cosines and sines are float32 and computed here from the position (once per token, for all heads), so no
// table bounds the positions.
// Statistics and all arithmetic are float32; outputs are rounded to the activation type once.  One block per token.  bfloat16 rows
// whose sizes are whole 16-byte pieces take the second kernel below: a head is shared by 8, 16 or 32 lanes of eight entries each.
//
// turn_heads: what undoes the rotation of values on the attention's output: out[t, h, :Dv] = attn[t, h, :Dv] with every pair turned by
// -position * freq[i] (the padded tail is dropped).
#include "common.cuh"
#include "range_check.cuh"

#define MIE_K_QK_NORM_ROPE 10

template <typename T>
__global__ void qk_norm_rope_kernel(const T* __restrict__ qkv, int64_t qkv_stride, const int* __restrict__ positions,
                                    const int* __restrict__ slots, const float* __restrict__ freq,
                                    const void* __restrict__ qw, const void* __restrict__ kw, const void* __restrict__ temp,
                                    int w_tag, float eps, float q_scale, float k_scale, T* __restrict__ q_out,
                                    T* __restrict__ k_cache, T* __restrict__ v_cache, int H, int G, int D, int Dv, int DP,
                                    int rot, int page_size, int64_t num_pages, int write_cache, int* report, int head_norm,
                                    int interleaved, float temp_coef, int temp_every, const float* __restrict__ v_freq) {
    __shared__ float red[33];
    extern __shared__ float cs[];                 // cos [rot/2], sin [rot/2]: once per token, for all heads; cos and sin [Dv/2] for v
    pdl_enter();
    const int t = blockIdx.x;
    const T* q = qkv + (int64_t)t * qkv_stride;
    const T* k = q + H * D;
    const T* v = k + G * D;
    const float pos = (float)positions[t];
    float sq = 1.f, sk = 1.f;
    if (qw && !head_norm) {
        float ss = 0.f;
        for (int i = threadIdx.x; i < H * D; i += blockDim.x) { const float x = to_f32<T>(q[i]); ss += x * x; }
        sq = 1.0f / sqrtf(block_sum(ss, red) / (float)(H * D) + eps);
    }
    if (kw && !head_norm) {
        float ss = 0.f;
        for (int i = threadIdx.x; i < G * D; i += blockDim.x) { const float x = to_f32<T>(k[i]); ss += x * x; }
        sk = 1.0f / sqrtf(block_sum(ss, red) / (float)(G * D) + eps);
    }
    const int half = rot >> 1;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        const float a = pos * freq[i];
        cs[i] = cosf(a);
        cs[half + i] = sinf(a);
    }
    float* vcs = cs + rot;
    const int vhalf = v_freq ? Dv >> 1 : 0;
    for (int i = threadIdx.x; i < vhalf; i += blockDim.x) {
        const float a = pos * v_freq[i];
        vcs[i] = cosf(a);
        vcs[vhalf + i] = sinf(a);
    }
    __syncthreads();
    // one entry of a rotated projection: x normed, then turned with its partner
    auto entry = [&](const T* x, const void* w, float s, int h, int d) -> float {
        const int wb = head_norm ? 0 : h * D;                     // per-head norms share one weight vector
        float own = to_f32<T>(x[h * D + d]) * s;
        if (w) own *= load_tagged(w, wb + d, w_tag);
        if (d >= rot) return own;
        const bool first = interleaved ? !(d & 1) : d < half;    // the pair's first entry turns with a minus
        const int pd = interleaved ? (d ^ 1) : (d < half ? d + half : d - half);
        const int fi = interleaved ? (d >> 1) : (d < half ? d : d - half);
        float other = to_f32<T>(x[h * D + pd]) * s;
        if (w) other *= load_tagged(w, wb + pd, w_tag);
        const float c = cs[fi], sn = cs[half + fi];
        return first ? own * c - other * sn : own * c + other * sn;
    };
    // a head's own statistic, by the head's warp
    auto head_scale = [&](const T* x, int h, int lane) -> float {
        float ss = 0.f;
        for (int d = lane; d < D; d += 32) { const float v = to_f32<T>(x[h * D + d]); ss += v * v; }
        return 1.0f / sqrtf(warp_sum(ss) / (float)D + eps);
    };
    float pos_temp = 1.f;
    if (temp_every > 0) pos_temp = 1.0f + temp_coef * logf((float)((positions[t] + 1) / temp_every) + 1.0f);
    T* qo = q_out + (int64_t)t * H * DP;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    for (int h = warp; h < H; h += nw) {                      // a head a warp, a dimension a lane: no divisions
        const float hs = (temp ? q_scale * load_tagged(temp, h, w_tag) : q_scale) * pos_temp;
        const float s_h = head_norm ? head_scale(q, h, lane) : sq;
        for (int d = lane; d < DP; d += 32) qo[h * DP + d] = from_f32<T>(d < D ? entry(q, qw, s_h, h, d) * hs : 0.f);
    }
    if (!write_cache) return;
    const int slot = slots[t];
    if (range_slot(slot, num_pages, page_size) != MIE_RANGE_OK) {
        if (threadIdx.x == 0) range_report(report, MIE_RANGE_SLOT, MIE_K_QK_NORM_ROPE, t, slot);
        return;
    }
    const int page = slot / page_size, off = slot - page * page_size;
    for (int g = warp; g < G; g += nw) {
        const int64_t row = (((int64_t)page * G + g) * page_size + off) * DP;
        const float s_g = head_norm ? head_scale(k, g, lane) : sk;
        for (int d = lane; d < DP; d += 32) {
            k_cache[row + d] = from_f32<T>(d < D ? entry(k, kw, s_g, g, d) * k_scale : 0.f);
            if (!v_cache) continue;
            if (!v_freq || d >= Dv) {
                v_cache[row + d] = d < Dv ? v[g * Dv + d] : from_f32<T>(0.f);
                continue;
            }
            const bool first = interleaved ? !(d & 1) : d < vhalf;
            const int pd = interleaved ? (d ^ 1) : (first ? d + vhalf : d - vhalf), fi = interleaved ? (d >> 1) : (first ? d : d - vhalf);
            const float own = to_f32<T>(v[g * Dv + d]), other = to_f32<T>(v[g * Dv + pd]), c = vcs[fi], sn = vcs[vhalf + fi];
            v_cache[row + d] = from_f32<T>(first ? own * c - other * sn : own * c + other * sn);
        }
    }
}

__device__ __forceinline__ void unpack8(const uint4& u, float* f) {
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) { const float2 x = __bfloat1622float2(h[i]); f[2 * i] = x.x; f[2 * i + 1] = x.y; }
}
__device__ __forceinline__ uint4 pack8(const float* f) {
    uint4 u;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
    return u;
}

// Eight entries of a head (piece c of them) turned with their partners: `f` holds this lane's entries; in the "half" pairing the
// partners are another lane's of the same head (a shuffle within LANES lanes: every lane of the warp must come here).
// cs: cosines of the pairs, sn: sines (times `sign`: -1 turns back); n: entries that turn, a multiple of 16 (half) or 8.
template <int LANES>
__device__ __forceinline__ void turn8(float* f, int c, int n, const float* cs, const float* sn, float sign, bool interleaved) {
    if (interleaved) {
        if (c * 8 < n) {
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float co = cs[c * 4 + i], si = sign * sn[c * 4 + i], a = f[2 * i], b = f[2 * i + 1];
                f[2 * i] = a * co - b * si;
                f[2 * i + 1] = b * co + a * si;
            }
        }
        return;
    }
    const int hc = n >> 4;                                     // pieces in half of what turns
    const bool turns = c < 2 * hc, first = c < hc;
    const int from = turns ? (first ? c + hc : c - hc) : c, at = (first ? c : c - hc) * 8;
    float o[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) o[i] = __shfl_sync(0xffffffffu, f[i], from, LANES);
    if (turns) {
        const float s = first ? -sign : sign;
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] = f[i] * cs[at + i] + o[i] * (s * sn[at + i]);
    }
}

struct QkVec {
    const bf16* qkv; int64_t qkv_stride;
    const int* positions; const int* slots;
    const float* freq; const float* v_freq; const float* qw; const float* kw; const float* temp;
    float eps, q_scale, k_scale;
    bf16* q_out; bf16* k_cache; bf16* v_cache;
    int H, G, D, Dv, DP, rot, page_size; int64_t num_pages; int write_cache; int* report; int head_norm, interleaved;
    float temp_coef; int temp_every;
};

template <int LANES>
__global__ void qk_norm_rope_bf16x8_kernel(const QkVec p) {
    __shared__ float red[33];
    extern __shared__ __align__(16) float cs[];                // as above
    pdl_enter();
    const int t = blockIdx.x;
    const bf16* q = p.qkv + (int64_t)t * p.qkv_stride;
    const int lane = threadIdx.x % LANES, group = threadIdx.x / LANES, groups = blockDim.x / LANES;
    const int slot = p.write_cache ? p.slots[t] : 0;
    const bool stores = p.write_cache && range_slot(slot, p.num_pages, p.page_size) == MIE_RANGE_OK;
    if (p.write_cache && !stores && threadIdx.x == 0) range_report(p.report, MIE_RANGE_SLOT, MIE_K_QK_NORM_ROPE, t, slot);
    const int heads = p.H + (stores ? (p.v_cache ? 2 : 1) * p.G : 0), qk = p.H + p.G;
    // a head's entries lie side by side: q and k heads are D wide, v heads Dv
    auto load = [&](int hh) {
        const int width = hh < qk ? p.D : p.Dv;
        const bf16* src = q + (hh < qk ? hh * p.D : qk * p.D + (hh - qk) * p.Dv);
        return hh < heads && lane * 8 < width ? *reinterpret_cast<const uint4*>(src + lane * 8) : make_uint4(0, 0, 0, 0);
    };
    uint4 next = load(group);                                  // the first head's entries travel while angles are worked out
    const int position = p.positions[t];
    const float pos = (float)position;
    float sq = 1.f, sk = 1.f;
    if (!p.head_norm && (p.qw || p.kw)) {                      // statistics over whole projections
        float a = 0.f, b = 0.f, f[8];
        for (int i = threadIdx.x; i < (qk * p.D) >> 3; i += blockDim.x) {
            unpack8(*reinterpret_cast<const uint4*>(q + i * 8), f);
            float ss = 0.f;
#pragma unroll
            for (int j = 0; j < 8; ++j) ss += f[j] * f[j];
            if (i * 8 < p.H * p.D) a += ss; else b += ss;
        }
        if (p.qw) sq = 1.0f / sqrtf(block_sum(a, red) / (float)(p.H * p.D) + p.eps);
        if (p.kw) sk = 1.0f / sqrtf(block_sum(b, red) / (float)(p.G * p.D) + p.eps);
    }
    const int half = p.rot >> 1, vhalf = p.v_freq ? p.Dv >> 1 : 0;
    float* vcs = cs + p.rot;
    for (int i = threadIdx.x; i < half + vhalf; i += blockDim.x) {
        const bool of_v = i >= half;
        const int j = of_v ? i - half : i;
        float si, co;
        sincosf(pos * (of_v ? p.v_freq[j] : p.freq[j]), &si, &co);
        float* at = of_v ? vcs : cs;
        at[j] = co;
        at[(of_v ? vhalf : half) + j] = si;
    }
    __syncthreads();
    float pos_temp = 1.f;
    if (p.temp_every > 0) pos_temp = 1.0f + p.temp_coef * logf((float)((position + 1) / p.temp_every) + 1.0f);
    const int page = slot / p.page_size, off = slot - page * p.page_size;
    for (int base = 0; base < heads; base += groups) {         // every lane of a warp goes round equally often
        const int hh = base + group;
        float f[8];
        unpack8(next, f);
        if (base + groups < heads) next = load(hh + groups);
        const bool is_v = hh >= qk, is_k = hh >= p.H && !is_v;
        if (p.head_norm) {
            float ss = 0.f;
#pragma unroll
            for (int i = 0; i < 8; ++i) ss += f[i] * f[i];
#pragma unroll
            for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o, LANES);
            const float s = 1.0f / sqrtf(ss / (float)p.D + p.eps);
            if (!is_v) {
#pragma unroll
                for (int i = 0; i < 8; ++i) f[i] *= s;
            }
        } else if (!is_v) {
            const float s = is_k ? sk : sq;
#pragma unroll
            for (int i = 0; i < 8; ++i) f[i] *= s;
        }
        const float* w = is_v ? nullptr : is_k ? p.kw : p.qw;
        if (w && hh < heads && lane * 8 < p.D) {
            const float* wp = w + (p.head_norm ? 0 : (is_k ? hh - p.H : hh) * p.D) + lane * 8;
            const float4 w0 = *reinterpret_cast<const float4*>(wp), w1 = *reinterpret_cast<const float4*>(wp + 4);
            f[0] *= w0.x; f[1] *= w0.y; f[2] *= w0.z; f[3] *= w0.w; f[4] *= w1.x; f[5] *= w1.y; f[6] *= w1.z; f[7] *= w1.w;
        }
        turn8<LANES>(f, lane, is_v ? 2 * vhalf : p.rot, is_v ? vcs : cs, is_v ? vcs + vhalf : cs + half, 1.f, p.interleaved != 0);
        if (hh >= heads || lane * 8 >= p.DP) continue;
        if (!is_v) {
            const float s = is_k ? p.k_scale : (p.temp ? p.q_scale * p.temp[hh] : p.q_scale) * pos_temp;
#pragma unroll
            for (int i = 0; i < 8; ++i) f[i] *= s;
        }
        bf16* dst;
        if (hh < p.H) dst = p.q_out + ((int64_t)t * p.H + hh) * p.DP;
        else dst = (is_v ? p.v_cache : p.k_cache) + (((int64_t)page * p.G + (hh - p.H - (is_v ? p.G : 0))) * p.page_size + off) * p.DP;
        *reinterpret_cast<uint4*>(dst + lane * 8) = pack8(f);
    }
}

template <int LANES>
static int launch_qk_vec(const QkVec& p, int num_tokens, cudaStream_t stream) {
    const int pieces = (p.H + (p.v_cache ? 2 : 1) * p.G) * LANES;
    int threads = 64;
    while (threads < 256 && threads < pieces) threads <<= 1;
    return launch_kernel(qk_norm_rope_bf16x8_kernel<LANES>, dim3(num_tokens), dim3(threads),
                         (size_t)(p.rot + (p.v_freq ? p.Dv : 0)) * sizeof(float), stream, p);
}

template <typename T>
__global__ void turn_heads_kernel(const T* __restrict__ attn, const int* __restrict__ positions, const float* __restrict__ freq,
                                  T* __restrict__ out, int H, int Dv, int DP, int interleaved) {
    extern __shared__ float cs[];
    pdl_enter();
    const int t = blockIdx.x, half = Dv >> 1;
    const float pos = (float)positions[t];
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        const float a = pos * freq[i];
        cs[i] = cosf(a);
        cs[half + i] = sinf(a);
    }
    __syncthreads();
    for (int idx = threadIdx.x; idx < H * Dv; idx += blockDim.x) {
        const int h = idx / Dv, d = idx - h * Dv;
        const T* x = attn + ((int64_t)t * H + h) * DP;
        const bool first = interleaved ? !(d & 1) : d < half;
        const int pd = interleaved ? (d ^ 1) : (first ? d + half : d - half), fi = interleaved ? (d >> 1) : (first ? d : d - half);
        const float own = to_f32<T>(x[d]), other = to_f32<T>(x[pd]), c = cs[fi], sn = cs[half + fi];
        out[(int64_t)t * H * Dv + idx] = from_f32<T>(first ? own * c + other * sn : own * c - other * sn);
    }
}

template <int LANES>
__global__ void turn_heads_bf16x8_kernel(const bf16* __restrict__ attn, const int* __restrict__ positions, const float* __restrict__ freq,
                                         bf16* __restrict__ out, int H, int Dv, int DP, int interleaved) {
    extern __shared__ __align__(16) float cs[];
    pdl_enter();
    const int t = blockIdx.x, half = Dv >> 1;
    const int lane = threadIdx.x % LANES, group = threadIdx.x / LANES, groups = blockDim.x / LANES;
    auto load = [&](int h) {
        return h < H && lane * 8 < Dv ? *reinterpret_cast<const uint4*>(attn + ((int64_t)t * H + h) * DP + lane * 8) : make_uint4(0, 0, 0, 0);
    };
    uint4 next = load(group);
    const float pos = (float)positions[t];
    for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf(pos * freq[i], &cs[half + i], &cs[i]);
    __syncthreads();
    for (int base = 0; base < H; base += groups) {
        const int h = base + group;
        float f[8];
        unpack8(next, f);
        if (base + groups < H) next = load(h + groups);
        turn8<LANES>(f, lane, Dv, cs, cs + half, -1.f, interleaved != 0);
        if (h < H && lane * 8 < Dv) *reinterpret_cast<uint4*>(out + ((int64_t)t * H + h) * Dv + lane * 8) = pack8(f);
    }
}

template <int LANES>
static int launch_turn_vec(const bf16* attn, const int* positions, const float* freq, bf16* out, int num_tokens, int H, int Dv, int DP,
                           int interleaved, cudaStream_t stream) {
    int threads = 64;
    while (threads < 256 && threads < H * LANES) threads <<= 1;
    return launch_kernel(turn_heads_bf16x8_kernel<LANES>, dim3(num_tokens), dim3(threads), (size_t)Dv * sizeof(float), stream, attn,
                         positions, freq, out, H, Dv, DP, interleaved);
}

// attn [T, H, DP] (heads of Dv entries, padded), out [T, H, Dv]; freq holds Dv / 2 frequencies.
extern "C" int mie_turn_heads(const void* attn, int tag, const int* positions, const float* freq, void* out, int num_tokens, int H, int Dv,
                              int DP, int interleaved, cudaStream_t stream) {
    if (num_tokens <= 0) return 0;
    if (H <= 0 || Dv <= 0 || (Dv & 1) || DP < Dv) return MIE_ERR_BAD_ARG;
    const size_t smem = (size_t)Dv * sizeof(float);
    if (tag == MIE_F32)
        return launch_kernel(turn_heads_kernel<float>, dim3(num_tokens), dim3(256), smem, stream, (const float*)attn, positions, freq,
                             (float*)out, H, Dv, DP, interleaved);
    if (tag != MIE_BF16) return MIE_ERR_BAD_ARG;
    const bool vec = Dv % (interleaved ? 8 : 16) == 0 && DP % 8 == 0 && Dv <= 256 &&
                     (reinterpret_cast<uintptr_t>(attn) | reinterpret_cast<uintptr_t>(out)) % 16 == 0;
    if (vec) {
        if (Dv <= 64) return launch_turn_vec<8>((const bf16*)attn, positions, freq, (bf16*)out, num_tokens, H, Dv, DP, interleaved, stream);
        if (Dv <= 128) return launch_turn_vec<16>((const bf16*)attn, positions, freq, (bf16*)out, num_tokens, H, Dv, DP, interleaved, stream);
        return launch_turn_vec<32>((const bf16*)attn, positions, freq, (bf16*)out, num_tokens, H, Dv, DP, interleaved, stream);
    }
    return launch_kernel(turn_heads_kernel<bf16>, dim3(num_tokens), dim3(256), smem, stream, (const bf16*)attn, positions, freq, (bf16*)out,
                         H, Dv, DP, interleaved);
}

extern "C" int mie_qk_norm_rope(const void* qkv, int tag, long long qkv_stride, const int* positions, const int* slots,
                                const float* freq, const void* qw, const void* kw, const void* temp, int w_tag, float eps,
                                float q_scale, float k_scale, void* q_out, void* k_cache, void* v_cache, int num_tokens, int H,
                                int G, int D, int Dv, int DP, int rot, int page_size, long long num_pages, int write_cache,
                                int head_norm, int interleaved, float temp_coef, int temp_every, const float* v_freq,
                                cudaStream_t stream) {
    if (num_tokens <= 0) return 0;
    if (H <= 0 || G <= 0 || D <= 0 || Dv <= 0 || DP < D || DP < Dv || rot < 0 || rot > D || (rot & 1) || page_size <= 0)
        return MIE_ERR_BAD_ARG;
    if (v_freq && (Dv & 1)) return MIE_ERR_BAD_ARG;
    const auto aligned = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
    const int step = interleaved ? 8 : 16;
    if (tag == MIE_BF16 && DP <= 256 && D % 8 == 0 && Dv % 8 == 0 && DP % 8 == 0 && rot % step == 0 && (!v_freq || Dv % step == 0) &&
        qkv_stride % 8 == 0 && (w_tag == MIE_F32 || (!qw && !kw && !temp)) && aligned(qkv) && aligned(q_out) && aligned(k_cache) &&
        aligned(v_cache) && aligned(qw) && aligned(kw)) {
        const QkVec p{(const bf16*)qkv, (int64_t)qkv_stride, positions, slots, freq, v_freq, (const float*)qw, (const float*)kw,
                      (const float*)temp, eps, q_scale, k_scale, (bf16*)q_out, (bf16*)k_cache, (bf16*)v_cache, H, G, D, Dv, DP, rot,
                      page_size, (int64_t)num_pages, write_cache, g_range_report, head_norm, interleaved, temp_coef, temp_every};
        if (DP <= 64) return launch_qk_vec<8>(p, num_tokens, stream);
        if (DP <= 128) return launch_qk_vec<16>(p, num_tokens, stream);
        return launch_qk_vec<32>(p, num_tokens, stream);
    }
    const int threads = H * DP >= 2048 ? 256 : 128;
    const size_t smem = (size_t)(rot + (v_freq ? Dv : 0)) * sizeof(float);
    if (tag == MIE_F32)
        return launch_kernel(qk_norm_rope_kernel<float>, dim3(num_tokens), dim3(threads), smem, stream, (const float*)qkv,
                             (int64_t)qkv_stride, positions, slots, freq, qw, kw, temp, w_tag, eps, q_scale, k_scale,
                             (float*)q_out, (float*)k_cache, (float*)v_cache, H, G, D, Dv, DP, rot, page_size,
                             (int64_t)num_pages, write_cache, g_range_report, head_norm, interleaved, temp_coef, temp_every, v_freq);
    else if (tag == MIE_BF16)
        return launch_kernel(qk_norm_rope_kernel<bf16>, dim3(num_tokens), dim3(threads), smem, stream, (const bf16*)qkv,
                             (int64_t)qkv_stride, positions, slots, freq, qw, kw, temp, w_tag, eps, q_scale, k_scale,
                             (bf16*)q_out, (bf16*)k_cache, (bf16*)v_cache, H, G, D, Dv, DP, rot, page_size,
                             (int64_t)num_pages, write_cache, g_range_report, head_norm, interleaved, temp_coef, temp_every, v_freq);
    return MIE_ERR_BAD_ARG;
}
