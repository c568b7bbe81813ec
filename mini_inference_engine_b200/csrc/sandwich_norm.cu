// The stream's update between two sublayers of a layer that norms both a sublayer's input and its output:
//
//   y[r, :]   = c0 * d0[r, :] + c1 * d1[r, :]                                   the output of the sublayer before (one or two branches)
//   x[r, :]   = res[r, :] + y / sqrt(mean(y^2) + eps) * pw[:]  + extra[r, :] + shift[:]
//   out[r, :] = x / sqrt(mean(x^2) + eps) * w[:]                                the next sublayer's input
//
// and res <- x.  Everything but res is optional: without d0 nothing is normed and added, `extra` (float32 [rows, n]) and `shift`
// (float32 [n]) are added where a model does so between two layers, without `out` the stream is updated only.  pw and w are the
// norms' weights as factors (a weight stored around zero, or a constant on the branch, is folded in when they are bound).
// `rows` (optional) gathers: output row b comes from input row rows[b] and the stream is left untouched (the selection in
// front of the output head).  One block per row; a thread keeps its pieces of the row in registers from the first load to the
// last store, so every input is read once; sums, statistics and the stream are float32, only `out` is rounded.
#include "common.cuh"
#include "range_check.cuh"

#define MIE_K_SANDWICH_NORM 13

struct SandwichParams {
    float* res;
    const void* d0; const void* d1; int tag0, tag1; float c0, c1;
    const float* pw; const float* extra; const float* shift; const float* w;
    void* out;
    const int* rows; int n, num_in_rows; float eps; int* report;
};

// Sum over the block, the same in every thread; `red` is 32 floats that nothing else uses.
__device__ __forceinline__ float sum_over_block(float v, float* red) {
    v = warp_sum(v);
    if (blockDim.x <= 32) return v;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    if (lane == 0) red[warp] = v;
    __syncthreads();
    return warp_sum(lane < (int)(blockDim.x >> 5) ? red[lane] : 0.f);
}

__device__ __forceinline__ float4 load4(const void* p, int tag, int64_t i) {       // entries i .. i+3, i a multiple of 4
    if (tag == MIE_F32) return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + i);
    const uint2 u = *reinterpret_cast<const uint2*>(reinterpret_cast<const bf16*>(p) + i);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, const float4& v) {
    uint2 o;
    *reinterpret_cast<__nv_bfloat162*>(&o.x) = __floats2bfloat162_rn(v.x, v.y);
    *reinterpret_cast<__nv_bfloat162*>(&o.y) = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = o;
}
__device__ __forceinline__ void add4(float4& a, const float4& b) { a.x += b.x; a.y += b.y; a.z += b.z; a.w += b.w; }
__device__ __forceinline__ float dot4(const float4& a) { return (a.x * a.x + a.y * a.y) + (a.z * a.z + a.w * a.w); }

// NV: pieces of four entries a thread.
template <typename TO, int NV>
__global__ void sandwich_norm_vec_kernel(const SandwichParams p) {
    __shared__ float red[2][32];
    pdl_enter();
    const int b = blockIdx.x;
    const int64_t r = p.rows ? p.rows[b] : b;
    if (p.rows && range_row(r, p.num_in_rows) != MIE_RANGE_OK) {
        if (threadIdx.x == 0) range_report(p.report, MIE_RANGE_ROW, MIE_K_SANDWICH_NORM, b, (int)r);
        return;
    }
    const int n = p.n;
    const int64_t base = r * n;
    float4 x[NV], y[NV];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = (threadIdx.x + k * blockDim.x) * 4;
        x[k] = y[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i >= n) continue;
        x[k] = *reinterpret_cast<const float4*>(p.res + base + i);
        if (p.d0) {
            const float4 a = load4(p.d0, p.tag0, base + i);
            y[k] = make_float4(p.c0 * a.x, p.c0 * a.y, p.c0 * a.z, p.c0 * a.w);
        }
        if (p.d1) {
            const float4 a = load4(p.d1, p.tag1, base + i);
            y[k].x = fmaf(p.c1, a.x, y[k].x); y[k].y = fmaf(p.c1, a.y, y[k].y); y[k].z = fmaf(p.c1, a.z, y[k].z); y[k].w = fmaf(p.c1, a.w, y[k].w);
        }
        if (p.extra) add4(x[k], *reinterpret_cast<const float4*>(p.extra + base + i));
        if (p.shift) add4(x[k], *reinterpret_cast<const float4*>(p.shift + i));
        ss += dot4(y[k]);
    }
    if (p.d0) {
        const float s = 1.0f / sqrtf(sum_over_block(ss, red[0]) / (float)n + p.eps);
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int i = (threadIdx.x + k * blockDim.x) * 4;
            if (i >= n) continue;
            const float4 w = *reinterpret_cast<const float4*>(p.pw + i);
            x[k].x = fmaf(y[k].x * s, w.x, x[k].x); x[k].y = fmaf(y[k].y * s, w.y, x[k].y);
            x[k].z = fmaf(y[k].z * s, w.z, x[k].z); x[k].w = fmaf(y[k].w * s, w.w, x[k].w);
        }
    }
    const bool stores = !p.rows && (p.d0 || p.extra || p.shift);
    ss = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = (threadIdx.x + k * blockDim.x) * 4;
        if (stores && i < n) *reinterpret_cast<float4*>(p.res + base + i) = x[k];
        ss += dot4(x[k]);
    }
    if (!p.out) return;
    const float s = 1.0f / sqrtf(sum_over_block(ss, red[1]) / (float)n + p.eps);
    TO* o = reinterpret_cast<TO*>(p.out) + (int64_t)b * n;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = (threadIdx.x + k * blockDim.x) * 4;
        if (i >= n) continue;
        const float4 w = *reinterpret_cast<const float4*>(p.w + i);
        store4(o + i, make_float4(x[k].x * s * w.x, x[k].y * s * w.y, x[k].z * s * w.z, x[k].w * s * w.w));
    }
}

// Rows that are no whole pieces of 16 bytes, and very long ones: y and x lie in shared memory between the passes.
template <typename TO>
__global__ void sandwich_norm_kernel(const SandwichParams p) {
    extern __shared__ float cache[];
    __shared__ float red[2][32];
    pdl_enter();
    const int b = blockIdx.x;
    const int64_t r = p.rows ? p.rows[b] : b;
    if (p.rows && range_row(r, p.num_in_rows) != MIE_RANGE_OK) {
        if (threadIdx.x == 0) range_report(p.report, MIE_RANGE_ROW, MIE_K_SANDWICH_NORM, b, (int)r);
        return;
    }
    const int n = p.n;
    const int64_t base = r * n;
    float ss = 0.f;
    if (p.d0)
        for (int i = threadIdx.x; i < n; i += blockDim.x) {
            float v = p.c0 * load_tagged(p.d0, base + i, p.tag0);
            if (p.d1) v = fmaf(p.c1, load_tagged(p.d1, base + i, p.tag1), v);
            cache[i] = v;
            ss += v * v;
        }
    float s = p.d0 ? 1.0f / sqrtf(sum_over_block(ss, red[0]) / (float)n + p.eps) : 0.f;
    const bool stores = !p.rows && (p.d0 || p.extra || p.shift);
    ss = 0.f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) {             // a thread reads back only what it has written itself
        float v = p.res[base + i];
        if (p.extra) v += p.extra[base + i];
        if (p.shift) v += p.shift[i];
        if (p.d0) v = fmaf(cache[i] * s, p.pw[i], v);
        if (stores) p.res[base + i] = v;
        cache[i] = v;
        ss += v * v;
    }
    if (!p.out) return;
    s = 1.0f / sqrtf(sum_over_block(ss, red[1]) / (float)n + p.eps);
    TO* o = reinterpret_cast<TO*>(p.out) + (int64_t)b * n;
    for (int i = threadIdx.x; i < n; i += blockDim.x) o[i] = from_f32<TO>(cache[i] * s * p.w[i]);
}

template <typename TO>
static int launch_sandwich(const SandwichParams& p, int num_rows, cudaStream_t stream) {
    const auto aligned = [](const void* q, uintptr_t a) { return (reinterpret_cast<uintptr_t>(q) & (a - 1)) == 0; };
    const bool vec = p.n % 4 == 0 && p.n <= 16384 && aligned(p.res, 16) && aligned(p.d0, p.tag0 == MIE_F32 ? 16 : 8) &&
                     aligned(p.d1, p.tag1 == MIE_F32 ? 16 : 8) && aligned(p.pw, 16) && aligned(p.extra, 16) && aligned(p.shift, 16) &&
                     aligned(p.w, 16) && aligned(p.out, 16);
    if (!vec) {
        const size_t smem = (size_t)p.n * sizeof(float);
        if (smem > 200 * 1024) return MIE_ERR_TOO_LARGE;
        if (smem > 48 * 1024) {
            const cudaError_t e = cudaFuncSetAttribute(sandwich_norm_kernel<TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            if (e != cudaSuccess) return (int)e;
        }
        int threads = 32;
        while (threads < 512 && threads < p.n) threads <<= 1;
        return launch_kernel(sandwich_norm_kernel<TO>, dim3(num_rows), dim3(threads), smem, stream, p);
    }
    // pieces a thread: one where few rows leave the GPU to themselves (the shortest chain), else two, more for wide rows
    const int pieces = p.n / 4;
    int nv = num_rows <= device_sm_count() && pieces <= 1024 ? 1 : 2;
    while (nv < 8 && (pieces + nv - 1) / nv > (nv < 4 ? 1024 : 512)) nv <<= 1;
    const int threads = ((pieces + nv - 1) / nv + 31) / 32 * 32;
    const dim3 grid(num_rows), block(threads);
    switch (nv) {
        case 1: return launch_kernel(sandwich_norm_vec_kernel<TO, 1>, grid, block, 0, stream, p);
        case 2: return launch_kernel(sandwich_norm_vec_kernel<TO, 2>, grid, block, 0, stream, p);
        case 4: return launch_kernel(sandwich_norm_vec_kernel<TO, 4>, grid, block, 0, stream, p);
        default: return launch_kernel(sandwich_norm_vec_kernel<TO, 8>, grid, block, 0, stream, p);
    }
}

// d0 / d1 (may be null): float32 or bfloat16 by tag; pw, shift, w: float32 [n]; extra: float32, rows as res.  out_tag: type of out.
extern "C" int mie_sandwich_norm(float* res, const void* d0, int tag0, float c0, const void* d1, int tag1, float c1, const float* pw,
                                 const float* extra, const float* shift, const float* w, void* out, int out_tag, const int* rows,
                                 int num_rows, int n, float eps, int num_in_rows, cudaStream_t stream) {
    if (num_rows <= 0) return 0;
    if (n <= 0 || (d1 && !d0) || (d0 && !pw) || (out && !w)) return MIE_ERR_BAD_ARG;
    const SandwichParams p{res, d0, d1, tag0, tag1, c0, c1, pw, extra, shift, w, out, rows, n, num_in_rows, eps, g_range_report};
    if (out_tag == MIE_F32) return launch_sandwich<float>(p, num_rows, stream);
    if (out_tag == MIE_BF16) return launch_sandwich<bf16>(p, num_rows, stream);
    return MIE_ERR_BAD_ARG;
}
