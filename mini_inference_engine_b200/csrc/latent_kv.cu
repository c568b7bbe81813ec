// Latent attention: queries and keys/values that go through low-rank latents, with one rotated key part shared by all heads.
//
//   down[t] = [ dq: Rq | dkv: C + R | anything else ]        one product of the mixer's input (row stride `stride`)
//   cq = rms(dq) wq          (RMS over the Rq entries, eps inside the root)         -> the up-projection of the queries
//   c  = rms(dkv[:C]) wc                                                          -> the up-projections of keys and values
//   kr = rotate(dkv[C:])     (the shared key part; not normed)
//
// (Rq 0: the queries have no latent.)  And, after the up-projections  qu[t] = [H x (D + R)] (row stride `qu_stride`: it may be part of a
// wider product),  kvu[t] = [k: H x D | v: H x Dv]:
//
//   q[h] = [ qu[h, :D] | rotate(qu[h, D:]) | 0 ]       -> q_out [T, H, DP]
//   k[h] = [ kvu.k[h]  | kr               | 0 ]       -> the cache slot of the token, head h
//   v[h] = [ kvu.v[h]  | 0 ]                           -> the cache slot
//
// so that the paged attention kernels, written for one head size DP >= max(D + R, Dv), serve it with H key/value heads.
// Rotation runs over the first `rot` entries of the rotated part and pairs entry 2i with 2i + 1 (`interleaved`) or i with
// i + rot/2; the angle is position x freq[i], computed here in float32 from the position (no table bounds the positions), and cos
// and sin are multiplied by `gain` (1, or what a frequency rescaling asks for).  Norm statistics and the rotation are float32;
// outputs are rounded once to the activation type.  One block per token; bfloat16 rows of whole 16-byte pieces are read
// and written eight entries at a time.
#include "common.cuh"
#include "range_check.cuh"

#define MIE_K_LATENT_KV 12

// entry i of a rotated part: the other entry of its pair, the pair's frequency, and whether it is the pair's first (which turns with a minus)
struct Pair { int partner, freq; bool first; };
__device__ __forceinline__ Pair pair_of(int i, int rot, int interleaved) {
    const int half = rot >> 1;
    if (interleaved) return {i ^ 1, i >> 1, (i & 1) == 0};
    return i < half ? Pair{i + half, i, true} : Pair{i - half, i - half, false};
}

template <typename T>
__global__ void latent_norm_rope_kernel(const T* __restrict__ down, int64_t stride, const int* __restrict__ positions,
                                        const float* __restrict__ freq, const float* __restrict__ wq, const float* __restrict__ wc,
                                        float eps, T* __restrict__ cq, T* __restrict__ c, float* __restrict__ kr, int Rq, int C, int R,
                                        int rot, int interleaved, float gain) {
    __shared__ float red[33];
    pdl_enter();
    const int t = blockIdx.x;
    const T* dq = down + (int64_t)t * stride;
    const T* dkv = dq + Rq;
    float ss = 0.f, sq = 1.f;
    if (Rq > 0) {
        for (int i = threadIdx.x; i < Rq; i += blockDim.x) { const float x = to_f32<T>(dq[i]); ss += x * x; }
        sq = 1.0f / sqrtf(block_sum(ss, red) / (float)Rq + eps);
    }
    ss = 0.f;
    for (int i = threadIdx.x; i < C; i += blockDim.x) { const float x = to_f32<T>(dkv[i]); ss += x * x; }
    const float sc = 1.0f / sqrtf(block_sum(ss, red) / (float)C + eps);
    for (int i = threadIdx.x; i < Rq; i += blockDim.x) cq[(int64_t)t * Rq + i] = from_f32<T>(to_f32<T>(dq[i]) * sq * wq[i]);
    for (int i = threadIdx.x; i < C; i += blockDim.x) c[(int64_t)t * C + i] = from_f32<T>(to_f32<T>(dkv[i]) * sc * wc[i]);
    const float pos = (float)positions[t];
    for (int i = threadIdx.x; i < R; i += blockDim.x) {
        float v = to_f32<T>(dkv[C + i]);
        if (i < rot) {
            const Pair p = pair_of(i, rot, interleaved);
            const float a = pos * freq[p.freq];
            const float cs = gain * cosf(a), sn = gain * sinf(a);
            const float other = to_f32<T>(dkv[C + p.partner]);
            v = p.first ? v * cs - other * sn : v * cs + other * sn;
        }
        kr[(int64_t)t * R + i] = v;
    }
}

template <typename T>
__global__ void latent_assemble_kernel(const T* __restrict__ qu, const T* __restrict__ kvu, const float* __restrict__ kr,
                                       const int* __restrict__ positions, const int* __restrict__ slots,
                                       const float* __restrict__ freq, T* __restrict__ q_out, T* __restrict__ k_cache,
                                       T* __restrict__ v_cache, int H, int D, int R, int Dv, int DP, int rot, int page_size,
                                       int64_t num_pages, int write_cache, int* report, int64_t qu_stride, int interleaved, float gain) {
    extern __shared__ float cs[];                 // cos [rot/2], sin [rot/2]
    pdl_enter();
    const int t = blockIdx.x;
    const int half = rot >> 1;
    const float pos = (float)positions[t];
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        const float a = pos * freq[i];
        cs[i] = gain * cosf(a);
        cs[half + i] = gain * sinf(a);
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    const T* q = qu + (int64_t)t * qu_stride;
    T* qo = q_out + (int64_t)t * H * DP;
    for (int h = warp; h < H; h += nw) {
        const T* qh = q + h * (D + R);
        for (int d = lane; d < DP; d += 32) {
            float v = 0.f;
            if (d < D) v = to_f32<T>(qh[d]);
            else if (d < D + R) {
                const int i = d - D;
                v = to_f32<T>(qh[d]);
                if (i < rot) {
                    const Pair p = pair_of(i, rot, interleaved);
                    const float other = to_f32<T>(qh[D + p.partner]);
                    const float c = cs[p.freq], s = cs[half + p.freq];
                    v = p.first ? v * c - other * s : v * c + other * s;
                }
            }
            qo[h * DP + d] = from_f32<T>(v);
        }
    }
    if (!write_cache) return;
    const int slot = slots[t];
    if (range_slot(slot, num_pages, page_size) != MIE_RANGE_OK) {
        if (threadIdx.x == 0) range_report(report, MIE_RANGE_SLOT, MIE_K_LATENT_KV, t, slot);
        return;
    }
    const int page = slot / page_size, off = slot - page * page_size;
    const T* kp = kvu + (int64_t)t * H * (D + Dv);
    const T* vp = kp + H * D;
    const float* krt = kr + (int64_t)t * R;
    for (int h = warp; h < H; h += nw) {
        const int64_t row = (((int64_t)page * H + h) * page_size + off) * DP;
        for (int d = lane; d < DP; d += 32) {
            k_cache[row + d] = d < D ? kp[h * D + d] : from_f32<T>(d < D + R ? krt[d - D] : 0.f);
            v_cache[row + d] = d < Dv ? vp[h * Dv + d] : from_f32<T>(0.f);
        }
    }
}

// The same for bfloat16 in pieces of eight entries (D, Dv, DP and the strides multiples of 8, R and rot of 16 with the "half" pairing, of
// 8 else).  A unit of work is one piece of one head of q_out, of k or of v; a piece of the rotated part reads its partner piece
// itself (two 16-byte loads instead of a shuffle: no unit depends on another lane).
__global__ void latent_assemble_bf16x8_kernel(const bf16* __restrict__ qu, int64_t qu_stride, const bf16* __restrict__ kvu,
                                              const float* __restrict__ kr, const int* __restrict__ positions, const int* __restrict__ slots,
                                              const float* __restrict__ freq, bf16* __restrict__ q_out, bf16* __restrict__ k_cache,
                                              bf16* __restrict__ v_cache, int H, int D, int R, int Dv, int DP, int rot, int page_size,
                                              int64_t num_pages, int write_cache, int* report, int interleaved, float gain) {
    extern __shared__ __align__(16) float cs[];                 // cos [rot/2], sin [rot/2], times gain
    pdl_enter();
    const int t = blockIdx.x;
    const int half = rot >> 1;
    const float pos = (float)positions[t];
    const int slot = write_cache ? slots[t] : 0;
    const bool stores = write_cache && range_slot(slot, num_pages, page_size) == MIE_RANGE_OK;
    if (write_cache && !stores && threadIdx.x == 0) range_report(report, MIE_RANGE_SLOT, MIE_K_LATENT_KV, t, slot);
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float si, co;
        sincosf(pos * freq[i], &si, &co);
        cs[i] = gain * co;
        cs[half + i] = gain * si;
    }
    __syncthreads();
    const int P = DP >> 3, D8 = D >> 3, R8 = R >> 3, V8 = Dv >> 3, half8 = half >> 3;
    const int page = slot / page_size, off = slot - page * page_size;
    const bf16* q = qu + (int64_t)t * qu_stride;
    const bf16* kp = kvu + (int64_t)t * H * (D + Dv);
    const bf16* vp = kp + H * D;
    const float* krt = kr + (int64_t)t * R;
    // units: q heads, then k heads, then v heads; a thread keeps its place within a head while it goes round by whole heads where
    // the block is a multiple of P, so the division runs once
    const int total = (stores ? 3 : 1) * H * P;
    int hh = threadIdx.x / P, c = threadIdx.x - hh * P;
    const int step_h = blockDim.x / P, step_c = blockDim.x - step_h * P;
    for (int u = threadIdx.x; u < total; u += blockDim.x, hh += step_h, c += step_c) {
        if (c >= P) { c -= P; ++hh; }
        uint4 o = make_uint4(0, 0, 0, 0);
        bf16* dst;
        if (hh < H) {
            const bf16* qh = q + hh * (D + R);
            dst = q_out + ((int64_t)t * H + hh) * DP;
            if (c < D8 || (c < D8 + R8 && (c - D8) * 8 >= rot)) {
                o = *reinterpret_cast<const uint4*>(qh + c * 8);
            } else if (c < D8 + R8) {
                const int i8 = c - D8;
                const uint4 own = *reinterpret_cast<const uint4*>(qh + c * 8);
                const __nv_bfloat162* ho = reinterpret_cast<const __nv_bfloat162*>(&own);
                __nv_bfloat162* hd = reinterpret_cast<__nv_bfloat162*>(&o);
                if (interleaved) {
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        const float2 x = __bfloat1622float2(ho[j]);
                        const float co = cs[i8 * 4 + j], si = cs[half + i8 * 4 + j];
                        hd[j] = __floats2bfloat162_rn(x.x * co - x.y * si, x.y * co + x.x * si);
                    }
                } else {
                    const bool first = i8 < half8;
                    const int at = (first ? i8 : i8 - half8) * 8;
                    const uint4 oth = *reinterpret_cast<const uint4*>(qh + (first ? c + half8 : c - half8) * 8);
                    const __nv_bfloat162* hx = reinterpret_cast<const __nv_bfloat162*>(&oth);
                    const float sign = first ? -1.f : 1.f;
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        const float2 x = __bfloat1622float2(ho[j]), y = __bfloat1622float2(hx[j]);
                        hd[j] = __floats2bfloat162_rn(x.x * cs[at + 2 * j] + sign * y.x * cs[half + at + 2 * j],
                                                      x.y * cs[at + 2 * j + 1] + sign * y.y * cs[half + at + 2 * j + 1]);
                    }
                }
            }
        } else if (hh < 2 * H) {
            const int h = hh - H;
            dst = k_cache + (((int64_t)page * H + h) * page_size + off) * DP;
            if (c < D8) {
                o = *reinterpret_cast<const uint4*>(kp + h * D + c * 8);
            } else if (c < D8 + R8) {
                const float4 a = *reinterpret_cast<const float4*>(krt + (c - D8) * 8), b = *reinterpret_cast<const float4*>(krt + (c - D8) * 8 + 4);
                __nv_bfloat162* hd = reinterpret_cast<__nv_bfloat162*>(&o);
                hd[0] = __floats2bfloat162_rn(a.x, a.y); hd[1] = __floats2bfloat162_rn(a.z, a.w);
                hd[2] = __floats2bfloat162_rn(b.x, b.y); hd[3] = __floats2bfloat162_rn(b.z, b.w);
            }
        } else {
            const int h = hh - 2 * H;
            dst = v_cache + (((int64_t)page * H + h) * page_size + off) * DP;
            if (c < V8) o = *reinterpret_cast<const uint4*>(vp + h * Dv + c * 8);
        }
        *reinterpret_cast<uint4*>(dst + c * 8) = o;
    }
}

// A warp a token: norms of the latents and the shared key part, in pieces of eight entries (every size a multiple of 8); eight tokens a block.
__global__ void latent_norm_rope_bf16x8_kernel(const bf16* __restrict__ down, int64_t stride, const int* __restrict__ positions,
                                               const float* __restrict__ freq, const float* __restrict__ wq, const float* __restrict__ wc,
                                               float eps, bf16* __restrict__ cq, bf16* __restrict__ c, float* __restrict__ kr, int Rq, int C,
                                               int R, int rot, int interleaved, float gain, int num_tokens) {
    pdl_enter();
    const int t = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (t >= num_tokens) return;
    const bf16* dkv = down + (int64_t)t * stride + Rq;
    auto normed = [&](const bf16* x, const float* w, bf16* out, int n) {
        constexpr int KEEP = 4;                                 // pieces a lane keeps in registers (rows of up to 1,024 entries); longer rows are read twice
        uint4 kept[KEEP];
        float ss = 0.f;
        auto square = [&](const uint4& u) {
            const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
            for (int j = 0; j < 4; ++j) { const float2 f = __bfloat1622float2(h[j]); ss += f.x * f.x + f.y * f.y; }
        };
#pragma unroll
        for (int k = 0; k < KEEP; ++k) {
            const int i = (lane + 32 * k) * 8;
            kept[k] = i < n ? *reinterpret_cast<const uint4*>(x + i) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
        for (int k = 0; k < KEEP; ++k) square(kept[k]);
        for (int i = (lane + 32 * KEEP) * 8; i < n; i += 256) square(*reinterpret_cast<const uint4*>(x + i));
        const float s = 1.0f / sqrtf(warp_sum(ss) / (float)n + eps);
        auto emit = [&](const uint4& u, int i) {
            const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
            const float4 a = *reinterpret_cast<const float4*>(w + i), b = *reinterpret_cast<const float4*>(w + i + 4);
            const float ww[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
            uint4 o;
            __nv_bfloat162* ho = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
            for (int j = 0; j < 4; ++j) { const float2 f = __bfloat1622float2(h[j]); ho[j] = __floats2bfloat162_rn(f.x * s * ww[2 * j], f.y * s * ww[2 * j + 1]); }
            *reinterpret_cast<uint4*>(out + i) = o;
        };
#pragma unroll
        for (int k = 0; k < KEEP; ++k) { const int i = (lane + 32 * k) * 8; if (i < n) emit(kept[k], i); }
        for (int i = (lane + 32 * KEEP) * 8; i < n; i += 256) emit(*reinterpret_cast<const uint4*>(x + i), i);
    };
    if (Rq > 0) normed(dkv - Rq, wq, cq + (int64_t)t * Rq, Rq);
    normed(dkv, wc, c + (int64_t)t * C, C);
    const float pos = (float)positions[t];
    for (int i = lane; i < R; i += 32) {
        float v = __bfloat162float(dkv[C + i]);
        if (i < rot) {
            const Pair p = pair_of(i, rot, interleaved);
            float si, co;
            sincosf(pos * freq[p.freq], &si, &co);
            const float other = __bfloat162float(dkv[C + p.partner]);
            v = gain * (p.first ? v * co - other * si : v * co + other * si);
        }
        kr[(int64_t)t * R + i] = v;
    }
}

extern "C" int mie_latent_norm_rope(const void* down, int tag, long long stride, const int* positions, const float* freq,
                                    const float* wq, const float* wc, float eps, void* cq, void* c, float* kr, int num_tokens,
                                    int Rq, int C, int R, int rot, int interleaved, float gain, cudaStream_t stream) {
    if (num_tokens <= 0) return 0;
    if (Rq < 0 || C <= 0 || R < 0 || rot < 0 || rot > R || (rot & 1)) return MIE_ERR_BAD_ARG;
    const auto aligned = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
    if (tag == MIE_BF16 && Rq % 8 == 0 && C % 8 == 0 && stride % 8 == 0 && aligned(down) && aligned(wc) && aligned(c) &&
        (Rq == 0 || (aligned(wq) && aligned(cq)))) {
        const int warps = num_tokens >= 1024 ? 8 : num_tokens >= 256 ? 2 : 1;
        return launch_kernel(latent_norm_rope_bf16x8_kernel, dim3((num_tokens + warps - 1) / warps), dim3(32 * warps), 0, stream, (const bf16*)down,
                             (int64_t)stride, positions, freq, wq, wc, eps, (bf16*)cq, (bf16*)c, kr, Rq, C, R, rot, interleaved, gain, num_tokens);
    }
    const int threads = (Rq + C) >= 1024 ? 256 : 128;
    if (tag == MIE_F32)
        return launch_kernel(latent_norm_rope_kernel<float>, dim3(num_tokens), dim3(threads), 0, stream, (const float*)down,
                             (int64_t)stride, positions, freq, wq, wc, eps, (float*)cq, (float*)c, kr, Rq, C, R, rot, interleaved, gain);
    else if (tag == MIE_BF16)
        return launch_kernel(latent_norm_rope_kernel<bf16>, dim3(num_tokens), dim3(threads), 0, stream, (const bf16*)down,
                             (int64_t)stride, positions, freq, wq, wc, eps, (bf16*)cq, (bf16*)c, kr, Rq, C, R, rot, interleaved, gain);
    return MIE_ERR_BAD_ARG;
}

extern "C" int mie_latent_assemble(const void* qu, long long qu_stride, const void* kvu, int tag, const float* kr, const int* positions, const int* slots,
                                   const float* freq, void* q_out, void* k_cache, void* v_cache, int num_tokens, int H, int D,
                                   int R, int Dv, int DP, int rot, int page_size, long long num_pages, int write_cache, int interleaved,
                                   float gain, cudaStream_t stream) {
    if (num_tokens <= 0) return 0;
    if (H <= 0 || D < 0 || R < 0 || Dv <= 0 || DP < D + R || DP < Dv || rot < 0 || rot > R || (rot & 1) || page_size <= 0)
        return MIE_ERR_BAD_ARG;
    const auto aligned = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
    const int step = interleaved ? 8 : 16;
    if (tag == MIE_BF16 && D % 8 == 0 && R % 8 == 0 && Dv % 8 == 0 && DP % 8 == 0 && rot % step == 0 && qu_stride % 8 == 0 && aligned(qu) &&
        aligned(kvu) && aligned(kr) && aligned(q_out) && aligned(k_cache) && aligned(v_cache)) {
        int threads = 64;
        while (threads < 256 && threads < 3 * H * (DP / 8)) threads <<= 1;
        return launch_kernel(latent_assemble_bf16x8_kernel, dim3(num_tokens), dim3(threads), (size_t)rot * sizeof(float), stream,
                             (const bf16*)qu, (int64_t)qu_stride, (const bf16*)kvu, kr, positions, slots, freq, (bf16*)q_out, (bf16*)k_cache,
                             (bf16*)v_cache, H, D, R, Dv, DP, rot, page_size, (int64_t)num_pages, write_cache, g_range_report, interleaved, gain);
    }
    const int threads = H * DP >= 2048 ? 256 : 128;
    if (tag == MIE_F32)
        return launch_kernel(latent_assemble_kernel<float>, dim3(num_tokens), dim3(threads), (size_t)rot * sizeof(float), stream,
                             (const float*)qu, (const float*)kvu, kr, positions, slots, freq, (float*)q_out, (float*)k_cache,
                             (float*)v_cache, H, D, R, Dv, DP, rot, page_size, (int64_t)num_pages, write_cache, g_range_report,
                             (int64_t)qu_stride, interleaved, gain);
    else if (tag == MIE_BF16)
        return launch_kernel(latent_assemble_kernel<bf16>, dim3(num_tokens), dim3(threads), (size_t)rot * sizeof(float), stream,
                             (const bf16*)qu, (const bf16*)kvu, kr, positions, slots, freq, (bf16*)q_out, (bf16*)k_cache,
                             (bf16*)v_cache, H, D, R, Dv, DP, rot, page_size, (int64_t)num_pages, write_cache, g_range_report,
                             (int64_t)qu_stride, interleaved, gain);
    return MIE_ERR_BAD_ARG;
}
