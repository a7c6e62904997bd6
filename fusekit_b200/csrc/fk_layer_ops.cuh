// Device functions shared by the layered decoders' kernels.
#pragma once
#include "fk_common.cuh"
#include <math.h>

#define FKL_MAX_EXPERTS 1024
#define FKL_MAX_TOP 64
#define FKL_GV_MAX_GROUPS 1024        // groups of a mixer's output norm
#define FKL_ERR_TOKEN 0x20000u
#define FKL_ERR_CAPACITY 0x100000u
#define FKL_ERR_TC_WAIT 0x200000u

enum { FKL_ACT_NONE = 0, FKL_ACT_RELU2 = 2, FKL_ACT_SILU = 3 };

__device__ __forceinline__ float ldT(const uint16_t *p) { return bf2f(*p); }
__device__ __forceinline__ float ldT(const float *p) { return *p; }
__device__ __forceinline__ void stT(uint16_t *p, float v) { *p = f2bf(v); }
__device__ __forceinline__ void stT(float *p, float v) { *p = v; }
__device__ __forceinline__ float inv_rms(float ss, int n, float eps) { return __fdiv_rn(1.0f, __fsqrt_rn(ss / (float)n + eps)); }
__device__ __forceinline__ float sigmoid_f(float z) { return __fdiv_rn(1.0f, 1.0f + expf(-z)); }
__device__ __forceinline__ float act_apply(float v, int act) {
    if (act == FKL_ACT_RELU2) { v = fmaxf(v, 0.0f); v *= v; }
    else if (act == FKL_ACT_SILU) v *= sigmoid_f(v);
    return v;
}
// one value of a clamped gated feed-forward from its gate and up products
__device__ __forceinline__ float clamped_glu(float g, float u, float limit) {
    g = fminf(g, limit); u = fminf(fmaxf(u, -limit), limit);
    return g * sigmoid_f(1.702f * g) * (u + 1.0f);
}
// two sums of a block at once (red: 66 floats)
__device__ __forceinline__ float2 block_sum2(float a, float b, float *red) {
    const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
    a = warp_sum(a); b = warp_sum(b);
    __syncthreads();
    if (lane == 0) { red[wid] = a; red[33 + wid] = b; }
    __syncthreads();
    if (wid == 0) {
        const float u = warp_sum(lane < nw ? red[lane] : 0.0f), v = warp_sum(lane < nw ? red[33 + lane] : 0.0f);
        if (lane == 0) { red[32] = u; red[65] = v; }
    }
    __syncthreads();
    return make_float2(red[32], red[65]);
}
// The keys a position sees: all up to itself, or with a window the newest `window` of them and the first `keep`.  They are counted
// 0 .. n - 1 in order (the position itself is n - 1).
struct Visible { int kept, lo, n; __device__ __forceinline__ int key(int i) const { return i < kept ? i : lo + i - kept; } };
__device__ __forceinline__ Visible visible_keys(int pos, int window, int keep) {
    const int lo = window > 0 ? max(0, pos - window + 1) : 0, kept = min(keep, lo);
    return Visible{kept, lo, kept + pos - lo + 1};
}
// dimension i of a head after rotation by a position's table row (cos, sin of pair 0, of pair 1, ..); v: the value, other: its pair's
__device__ __forceinline__ float rotate_dim(float v, float other, int i, int dims, const float *row) {
    if (i >= dims) return v;
    const float2 cs = reinterpret_cast<const float2 *>(row)[i >> 1];
    return (i & 1) ? fmaf(v, cs.x, other * cs.y) : fmaf(v, cs.x, -(other * cs.y));
}
__device__ __forceinline__ void unpack8f(uint4 v, float (&f)[8]) {
    f[0] = bf_lo(v.x); f[1] = bf_hi(v.x); f[2] = bf_lo(v.y); f[3] = bf_hi(v.y); f[4] = bf_lo(v.z); f[5] = bf_hi(v.z); f[6] = bf_lo(v.w); f[7] = bf_hi(v.w);
}
__device__ __forceinline__ void load8(const uint16_t *p, float (&f)[8]) { unpack8f(__ldcg(reinterpret_cast<const uint4 *>(p)), f); }
__device__ __forceinline__ void load8(const float *p, float (&f)[8]) {
    const float4 a = __ldcg(reinterpret_cast<const float4 *>(p)), b = __ldcg(reinterpret_cast<const float4 *>(p) + 1);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ float4 ld4(const uint16_t *p) { const uint2 v = __ldcg(reinterpret_cast<const uint2 *>(p)); return make_float4(bf_lo(v.x), bf_hi(v.x), bf_lo(v.y), bf_hi(v.y)); }
__device__ __forceinline__ float4 ld4(const float *p) { return __ldcg(reinterpret_cast<const float4 *>(p)); }
__device__ __forceinline__ void st4(uint16_t *p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2 *>(p) = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
}
__device__ __forceinline__ void st4(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void cp16_zfill(uint32_t dst, const void *src, bool valid) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
