// Causal attention of M positions on the tensor cores (mma.m16n8k16, bf16 operands, fp32 accumulation), with one or two
// query/key maps per head over the same values.
//
// A block owns 64 positions of one query head.  Four warps per map, 16 positions each; both maps walk the keys together, 64 at a
// time, through a double-buffered shared-memory tile (cp.async) of the maps' keys and the one set of values.  Scores and the
// online softmax are fp32; a weight enters the value product as two bf16 terms (hi + lo), which keeps it at fp32 grade.  At the
// end the second map's warps hand their result over in shared memory and the first map's apply a1 - lambda a2, the unit rms, the
// factor 1 - diff and the output gate.  KD / VD: head sizes padded to the instance (zero columns).  With a window the block walks the
// tiles of the kept first keys and those from the oldest key its first position sees; a tile may hide all of a row's keys.
#pragma once
#include "fk_layers.cuh"

struct FlashArgs { const uint16_t *q, *ck, *cv, *gate; uint16_t *out; int H, G, maps, vdim, dpad, vpad, cap, ldo, ldg, rows; float scale, lambda, diff, eps; int window, keep; };
template <int KD, int VD> __host__ __device__ constexpr size_t flash_stage_bytes(int maps) { return (size_t)64 * 2 * ((size_t)maps * (KD + 8) + (VD + 8)); }
template <int KD, int VD> __host__ __device__ constexpr size_t flash_smem_bytes(int maps) {
    return 2 * flash_stage_bytes<KD, VD>(maps) > (size_t)64 * (VD + 2) * 4 ? 2 * flash_stage_bytes<KD, VD>(maps) : (size_t)64 * (VD + 2) * 4;
}
__device__ __forceinline__ void fl_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void fl_ldsm(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void fl_ldsm_t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void fl_copy16(uint32_t dst, const void *src, bool valid) {        // 16 bytes, zeros when not valid
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ uint32_t fl_pack(float lo, float hi) { const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi); return *reinterpret_cast<const uint32_t *>(&h); }

template <int KD, int VD, bool WIN>
__global__ void __launch_bounds__(256, VD <= 128 && KD <= 64 ? 2 : 1) k_flash_rows(FkState *st, FlashArgs a) {
    extern __shared__ __align__(128) unsigned char fl_smem[];
    constexpr int KS = KD + 8, VS = VD + 8;             // row strides in elements: odd multiples of 16 bytes, so ldmatrix has no conflicts
    const int tid = threadIdx.x, lane = tid & 31, wid = tid >> 5, g8 = lane >> 2, t4 = lane & 3, map = wid >> 2, nt = blockDim.x;
    const int head = blockIdx.x, g = head / (a.H / a.G), row0 = ((int)gridDim.y - 1 - (int)blockIdx.y) * 64, wrow = row0 + (wid & 3) * 16;
    pdl_launch_dependents(); pdl_wait();
    const int off = (int)st->offset;
    const int last = off + min(row0 + 63, a.rows - 1);  // newest position of the block
    if (off + a.rows > a.cap) return;                   // reported by the cache store that came before
    const int wtile = WIN ? max(0, off + row0 - a.window + 1) / 64 : 0, kept = WIN ? min((a.keep + 63) / 64, wtile) : 0, ntiles = kept + last / 64 - wtile + 1;
    auto place = [&](int i) { return i < kept ? i : wtile + i - kept; };
    const uint32_t sbase = (uint32_t)__cvta_generic_to_shared(fl_smem), stage = (uint32_t)flash_stage_bytes<KD, VD>(a.maps);
    const uint16_t *ck = a.ck + (size_t)g * a.maps * a.cap * a.dpad, *cv = a.cv + (size_t)g * a.cap * a.vpad;
    auto fetch = [&](int tile, int s) {
        const uint32_t kb = sbase + s * stage, vb = kb + (uint32_t)(a.maps * 64 * KS * 2);
        for (int i = tid; i < a.maps * 64 * (KD / 8); i += nt) {
            const int r = i / (KD / 8), c = (i - r * (KD / 8)) * 8, key = tile * 64 + (r & 63);
            const bool v = c < a.dpad && key <= last;
            fl_copy16(kb + (uint32_t)((r * KS + c) * 2), v ? ck + ((size_t)(r >> 6) * a.cap + key) * a.dpad + c : ck, v);
        }
        for (int i = tid; i < 64 * (VD / 8); i += nt) {
            const int r = i / (VD / 8), c = (i - r * (VD / 8)) * 8, key = tile * 64 + r;
            const bool v = c < a.vpad && key <= last;
            fl_copy16(vb + (uint32_t)((r * VS + c) * 2), v ? cv + (size_t)key * a.vpad + c : cv, v);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(place(0), 0);
    // the warp's query rows as A fragments
    uint32_t qf[KD / 16][4];
    {
        const int r0 = min(wrow + g8, a.rows - 1), r1 = min(wrow + g8 + 8, a.rows - 1);
        const uint16_t *q0 = a.q + ((size_t)r0 * a.H * a.maps + head * a.maps + map) * a.dpad, *q1 = a.q + ((size_t)r1 * a.H * a.maps + head * a.maps + map) * a.dpad;
#pragma unroll
        for (int k = 0; k < KD / 16; ++k) {
            const int c = k * 16 + t4 * 2;
            qf[k][0] = c < a.dpad ? *reinterpret_cast<const uint32_t *>(q0 + c) : 0u; qf[k][1] = c < a.dpad ? *reinterpret_cast<const uint32_t *>(q1 + c) : 0u;
            qf[k][2] = c + 8 < a.dpad ? *reinterpret_cast<const uint32_t *>(q0 + c + 8) : 0u; qf[k][3] = c + 8 < a.dpad ? *reinterpret_cast<const uint32_t *>(q1 + c + 8) : 0u;
        }
    }
    float o[VD / 8][4];
#pragma unroll
    for (int i = 0; i < VD / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.0f, l1 = 0.0f;
    const float sc = a.scale * 1.44269504088896341f;     // scores in base-2 exponents
    const int pos0 = off + wrow + g8, pos1 = pos0 + 8;
    for (int it = 0; it < ntiles; ++it) {
        const int tile = place(it);
        if (it + 1 < ntiles) { fetch(place(it + 1), (it + 1) & 1); asm volatile("cp.async.wait_group 1;" ::: "memory"); }
        else asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        const uint32_t kb = sbase + (it & 1) * stage + (uint32_t)(map * 64 * KS * 2), vb = sbase + (it & 1) * stage + (uint32_t)(a.maps * 64 * KS * 2);
        // 32 keys at a time, as far as some key is visible to some row of the warp
#pragma unroll 1
        for (int h0 = 0; h0 < 64 && tile * 64 + h0 <= off + wrow + 15; h0 += 32) {
            if (WIN && tile * 64 + h0 >= a.keep && tile * 64 + h0 + 31 <= off + wrow - a.window) continue;
            float s[4][4];
#pragma unroll
            for (int i = 0; i < 4; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
#pragma unroll
            for (int k = 0; k < KD / 16; ++k)
#pragma unroll
                for (int n = 0; n < 2; ++n) {           // 16 keys: matrices (keys 0-7, k 0-7), (keys 0-7, k 8-15), (keys 8-15, ..) x 2
                    uint32_t b[4];
                    fl_ldsm(b, kb + (uint32_t)(((h0 + n * 16 + (lane & 7) + ((lane >> 4) << 3)) * KS + k * 16 + ((lane >> 3) & 1) * 8) * 2));
                    fl_mma(s[2 * n], qf[k], b[0], b[1]); fl_mma(s[2 * n + 1], qf[k], b[2], b[3]);
                }
            const bool edge = tile * 64 + h0 + 31 > off + wrow || (WIN && tile * 64 + h0 <= off + wrow + 15 - a.window);
            auto hidden = [&](int k, int p) { return k > p || (WIN && p - k >= a.window && k >= a.keep); };
            float x0 = -INFINITY, x1 = -INFINITY;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int key = tile * 64 + h0 + i * 8 + t4 * 2;
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    s[i][j] = edge && hidden(key + j, pos0) ? -INFINITY : s[i][j] * sc;
                    s[i][2 + j] = edge && hidden(key + j, pos1) ? -INFINITY : s[i][2 + j] * sc;
                    x0 = fmaxf(x0, s[i][j]); x1 = fmaxf(x1, s[i][2 + j]);
                }
            }
            x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 1)); x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 2));
            x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 1)); x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 2));
            const float n0 = fmaxf(m0, x0), n1 = fmaxf(m1, x1);
            const float e0 = WIN && n0 == -INFINITY ? 0.0f : n0, e1 = WIN && n1 == -INFINITY ? 0.0f : n1;       // no key seen yet: every factor is 0
            if (__any_sync(0xffffffffu, n0 > m0 || n1 > m1)) {          // a new maximum somewhere in the warp
                const float c0 = exp2f(m0 - e0), c1 = exp2f(m1 - e1);
                m0 = n0; m1 = n1; l0 *= c0; l1 *= c1;
#pragma unroll
                for (int i = 0; i < VD / 8; ++i) { o[i][0] *= c0; o[i][1] *= c0; o[i][2] *= c1; o[i][3] *= c1; }
            }
#pragma unroll
            for (int k = 0; k < 2; ++k) {               // 16 keys at a time: weights as hi + lo, times the values
                uint32_t ph[4], pl[4];
#pragma unroll
                for (int h = 0; h < 2; ++h) {
                    const int i = 2 * k + h;
                    const float p0 = exp2f(s[i][0] - e0), p1 = exp2f(s[i][1] - e0), p2 = exp2f(s[i][2] - e1), p3 = exp2f(s[i][3] - e1);
                    l0 += p0 + p1; l1 += p2 + p3;
                    ph[2 * h] = fl_pack(p0, p1); ph[2 * h + 1] = fl_pack(p2, p3);
                    pl[2 * h] = fl_pack(p0 - bf_lo(ph[2 * h]), p1 - bf_hi(ph[2 * h])); pl[2 * h + 1] = fl_pack(p2 - bf_lo(ph[2 * h + 1]), p3 - bf_hi(ph[2 * h + 1]));
                }
#pragma unroll
                for (int n = 0; n < VD / 16; ++n) {     // 16 value columns: matrices (keys 0-7 / 8-15) x (columns 0-7 / 8-15), transposed
                    uint32_t b[4];
                    fl_ldsm_t(b, vb + (uint32_t)(((h0 + k * 16 + (lane & 15)) * VS + n * 16 + (lane >> 4) * 8) * 2));
                    fl_mma(o[2 * n], ph, b[0], b[1]); fl_mma(o[2 * n + 1], ph, b[2], b[3]);
                    fl_mma(o[2 * n], pl, b[0], b[1]); fl_mma(o[2 * n + 1], pl, b[2], b[3]);
                }
            }
        }
        __syncthreads();
    }
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1); l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1); l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    const float i0 = 1.0f / l0, i1 = 1.0f / l1;
#pragma unroll
    for (int i = 0; i < VD / 8; ++i) { o[i][0] *= i0; o[i][1] *= i0; o[i][2] *= i1; o[i][3] *= i1; }
    const int lr = (wid & 3) * 16 + g8;
    float f0 = 1.0f, f1 = 1.0f;
    if (a.maps == 2) {
        float *x = reinterpret_cast<float *>(fl_smem);
        if (map == 1) {
#pragma unroll
            for (int i = 0; i < VD / 8; ++i) {
                *reinterpret_cast<float2 *>(x + lr * (VD + 2) + i * 8 + t4 * 2) = make_float2(o[i][0], o[i][1]);
                *reinterpret_cast<float2 *>(x + (lr + 8) * (VD + 2) + i * 8 + t4 * 2) = make_float2(o[i][2], o[i][3]);
            }
        }
        __syncthreads();
        if (map == 1) return;
        float s0 = 0.0f, s1 = 0.0f;
#pragma unroll
        for (int i = 0; i < VD / 8; ++i) {
            const float2 a0 = *reinterpret_cast<const float2 *>(x + lr * (VD + 2) + i * 8 + t4 * 2), a1 = *reinterpret_cast<const float2 *>(x + (lr + 8) * (VD + 2) + i * 8 + t4 * 2);
            o[i][0] -= a.lambda * a0.x; o[i][1] -= a.lambda * a0.y; o[i][2] -= a.lambda * a1.x; o[i][3] -= a.lambda * a1.y;
            s0 = fmaf(o[i][0], o[i][0], fmaf(o[i][1], o[i][1], s0)); s1 = fmaf(o[i][2], o[i][2], fmaf(o[i][3], o[i][3], s1));
        }
        s0 += __shfl_xor_sync(0xffffffffu, s0, 1); s0 += __shfl_xor_sync(0xffffffffu, s0, 2);
        s1 += __shfl_xor_sync(0xffffffffu, s1, 1); s1 += __shfl_xor_sync(0xffffffffu, s1, 2);
        f0 = inv_rms(s0, a.vdim, a.eps) * (1.0f - a.diff); f1 = inv_rms(s1, a.vdim, a.eps) * (1.0f - a.diff);
    }
    const int r0 = row0 + lr, r1 = r0 + 8;
    if (a.gate) {
        if (r0 < a.rows) f0 *= sigmoid_f(bf2f(a.gate[(size_t)r0 * a.ldg + head]));
        if (r1 < a.rows) f1 *= sigmoid_f(bf2f(a.gate[(size_t)r1 * a.ldg + head]));
    }
    const bool pairs = (a.vdim & 1) == 0;
#pragma unroll
    for (int i = 0; i < VD / 8; ++i) {
        const int d = i * 8 + t4 * 2;
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int r = h ? r1 : r0; const float f = h ? f1 : f0;
            if (r >= a.rows || d >= a.vdim) continue;
            uint16_t *y = a.out + (size_t)r * a.ldo + head * a.vdim + d;
            if (pairs) *reinterpret_cast<uint32_t *>(y) = fl_pack(o[i][2 * h] * f, o[i][2 * h + 1] * f);
            else { y[0] = f2bf(o[i][2 * h] * f); if (d + 1 < a.vdim) y[1] = f2bf(o[i][2 * h + 1] * f); }
        }
    }
}
