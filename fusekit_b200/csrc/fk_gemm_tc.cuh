// Matrix product on the 5th-generation tensor cores: Y[m, n] = act(sum_k X[m, k] W[row0 + n, k]), bf16 operands, fp32
// accumulation, optionally grouped by expert (the rows of X between offsets[e] and offsets[e + 1] use the weight rows e * N ..).
//
// Persistent, warp-specialised, one CTA per SM.  A tile is 128 rows of X by BN rows of W.  Warp 0 fetches K slices of 64 by
// TMA (128-byte swizzle) into a ring of shared-memory stages, one thread of warp 1 issues tcgen05.mma (cta_group::1, M = 128,
// N = BN, K = 16) into one of two accumulators in tensor memory, warps 4 .. 7 read finished accumulators back and store them
// while the next tile is being multiplied.  Rows past the end of a tile's range are multiplied and not stored (past the end of
// the tensor TMA delivers zeros).  Every wait is bounded: when one runs out the kernel sets an error bit, waits (bounded) for
// its copies in flight, frees its tensor memory and returns.
#pragma once
#include "fk_layers.cuh"
#include <cuda.h>

#define FKL_TC_BK 64
#define FKL_TC_THREADS 256
#define FKL_TC_SPIN (1u << 21)
template <int BN> struct TcTile {
    static constexpr int STAGES = BN == 256 ? 4 : BN == 128 ? 6 : 8;
    static constexpr int A_BYTES = 128 * FKL_TC_BK * 2, B_BYTES = BN * FKL_TC_BK * 2, STAGE = A_BYTES + B_BYTES, COLS = 2 * BN;
    static constexpr size_t SMEM = (size_t)STAGES * STAGE + 1024;
};
struct TcGemmArgs { void *y; const int *offsets; int m, n, kblocks, row0, ldy, act, out_f32, experts; float scale; BlockCols b; };       // b: BLOCK form

__device__ __forceinline__ uint32_t tcg_smem(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void tcg_init(uint32_t bar, uint32_t count) { asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar), "r"(count) : "memory"); }
__device__ __forceinline__ void tcg_arrive(uint32_t bar) { asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar) : "memory"); }
__device__ __forceinline__ bool tcg_wait(uint32_t bar, uint32_t parity) {
    for (uint32_t i = 0; i < FKL_TC_SPIN; ++i) {
        uint32_t ok;
        asm volatile("{\n\t.reg .pred p;\n\tmbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\tselp.u32 %0, 1, 0, p;\n\t}" : "=r"(ok) : "r"(bar), "r"(parity) : "memory");
        if (ok) return true;
    }
    return false;
}
__device__ __forceinline__ void tcg_load(uint32_t dst, const CUtensorMap *map, int k, int row, uint32_t bar) {
    asm volatile("cp.async.bulk.tensor.2d.shared::cta.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];"
                 ::"r"(dst), "l"(map), "r"(k), "r"(row), "r"(bar) : "memory");
}
// K-major operand with 128-byte swizzle: rows of 128 bytes, groups of 8 rows 1024 bytes apart
__device__ __forceinline__ uint64_t tcg_desc(uint32_t addr) {
    return (uint64_t)((addr >> 4) & 0x3FFFu) | (1ull << 16) | ((uint64_t)(1024 >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
template <int BN, bool BLOCK>
__global__ void __launch_bounds__(FKL_TC_THREADS, 1) k_gemm_tc(FkState *st, const __grid_constant__ CUtensorMap mx, const __grid_constant__ CUtensorMap mw, TcGemmArgs a) {
    using T = TcTile<BN>;
    constexpr int S = T::STAGES;
    extern __shared__ unsigned char smem_raw[];
    __shared__ __align__(8) uint64_t bars[2 * S + 4];
    __shared__ uint32_t tmem_slot;
    __shared__ int first[FKL_MAX_EXPERTS + 1];          // grouped: first 128-row tile of every expert
    __shared__ int wsum[8];
    const int tid = threadIdx.x, lane = tid & 31, wid = tid >> 5;
    const uint32_t base = (tcg_smem(smem_raw) + 1023u) & ~1023u;
    const uint32_t full = tcg_smem(bars), empty = full + 8 * S, afull = empty + 8 * S, aempty = afull + 16;
    pdl_launch_dependents();
    if (tid == 0) {
        for (int s = 0; s < S; ++s) { tcg_init(full + 8 * s, 1); tcg_init(empty + 8 * s, 1); }
        for (int s = 0; s < 2; ++s) { tcg_init(afull + 8 * s, 1); tcg_init(aempty + 8 * s, 4); }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (wid == 2) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(tcg_smem(&tmem_slot)), "r"((uint32_t)T::COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    pdl_wait();
    const int ntn = (a.n + BN - 1) / BN;
    int mtiles = (a.m + 127) / 128;
    if (a.offsets) {
        int carry = 0;
        for (int b = 0; b < a.experts; b += FKL_TC_THREADS) {
            const int e = b + tid, c = e < a.experts ? (a.offsets[e + 1] - a.offsets[e] + 127) / 128 : 0;
            int v = c;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) { const int t = __shfl_up_sync(0xffffffffu, v, o); if (lane >= o) v += t; }
            if (lane == 31) wsum[wid] = v;
            __syncthreads();
            int before = carry, total = 0;
            for (int w = 0; w < 8; ++w) { if (w < wid) before += wsum[w]; total += wsum[w]; }
            if (e < a.experts) first[e] = before + v - c;
            carry += total;
            __syncthreads();
        }
        if (tid == 0) first[a.experts] = carry;
        mtiles = carry;
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = tmem_slot;
    const int total = mtiles * ntn;
    // tile -> first row of X, end of its rows, first weight row, first column: neighbours share the weight tile (plain) or the
    // rows of X (grouped, where an expert has few rows)
    auto place = [&](int t, int &m0, int &mend, int &wrow, int &n0) {
        if (!a.offsets) { const int nt = t / mtiles; m0 = (t - nt * mtiles) * 128; mend = a.m; n0 = nt * BN; wrow = a.row0 + n0; return; }
        const int mt = t / ntn; n0 = (t - mt * ntn) * BN;
        int lo = 0, hi = a.experts;                     // last expert whose first tile is <= mt
        while (hi - lo > 1) { const int mid = (lo + hi) >> 1; if (first[mid] <= mt) lo = mid; else hi = mid; }
        m0 = a.offsets[lo] + (mt - first[lo]) * 128; mend = a.offsets[lo + 1]; wrow = lo * a.n + n0;
    };
    bool ok = true;
    if (wid == 0) {
        if (lane == 0) {
            int it = 0;
            for (int t = blockIdx.x; t < total && ok; t += gridDim.x) {
                int m0, mend, wrow, n0; place(t, m0, mend, wrow, n0);
                for (int kb = 0; kb < a.kblocks; ++kb, ++it) {
                    const int s = it % S;
                    if (it >= S && !tcg_wait(empty + 8 * s, (uint32_t)(it / S - 1) & 1u)) { ok = false; break; }
                    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(full + 8 * s), "r"((uint32_t)T::STAGE) : "memory");
                    tcg_load(base + s * T::STAGE, &mx, kb * FKL_TC_BK, m0, full + 8 * s);
                    tcg_load(base + s * T::STAGE + T::A_BYTES, &mw, kb * FKL_TC_BK, wrow, full + 8 * s);
                }
            }
            // the last stages are multiplied (or at least have landed) before the block may leave
            for (int j = it > S ? it - S : 0; j < it; ++j) if (!tcg_wait((ok ? empty : full) + 8 * (j % S), (uint32_t)(j / S) & 1u)) ok = false;
            if (!ok) atomicOr(&st->error, FKL_ERR_TC_WAIT);
        }
    } else if (wid == 1) {
        if (lane == 0) {
            const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BN >> 3) << 17) | ((128u >> 4) << 24);
            int it = 0, j = 0;
            for (int t = blockIdx.x; t < total && ok; t += gridDim.x, ++j) {
                const int b = j & 1;
                if (j >= 2 && !tcg_wait(aempty + 8 * b, (uint32_t)(j / 2 - 1) & 1u)) { ok = false; break; }
                for (int kb = 0; kb < a.kblocks; ++kb, ++it) {
                    const int s = it % S;
                    if (!tcg_wait(full + 8 * s, (uint32_t)(it / S) & 1u)) { ok = false; break; }
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    const uint64_t da = tcg_desc(base + s * T::STAGE), db = tcg_desc(base + s * T::STAGE + T::A_BYTES);
#pragma unroll
                    for (int k = 0; k < FKL_TC_BK / 16; ++k)
                        asm volatile("{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\ttcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
                                     ::"r"(tmem + (uint32_t)(b * BN)), "l"(da + (uint64_t)(k * 2)), "l"(db + (uint64_t)(k * 2)), "r"(idesc), "r"(kb | k) : "memory");
                    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(empty + 8 * s) : "memory");
                }
                if (ok) asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(afull + 8 * b) : "memory");
            }
            // the last commits have arrived before tensor memory is freed: the epilogue waits for every accumulator
            if (!ok) atomicOr(&st->error, FKL_ERR_TC_WAIT);
        }
    } else if (wid >= 4) {
        const int q = wid - 4;
        int j = 0;
        for (int t = blockIdx.x; t < total && ok; t += gridDim.x, ++j) {
            int m0, mend, wrow, n0; place(t, m0, mend, wrow, n0);
            const int b = j & 1, row = m0 + q * 32 + lane;
            if (!tcg_wait(afull + 8 * b, (uint32_t)(j / 2) & 1u)) { ok = false; break; }
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll 1
            for (int c = 0; c < BN; c += 32) {
                __syncwarp();
                uint32_t d[32];
                asm volatile("tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
                             : "=r"(d[0]), "=r"(d[1]), "=r"(d[2]), "=r"(d[3]), "=r"(d[4]), "=r"(d[5]), "=r"(d[6]), "=r"(d[7]), "=r"(d[8]), "=r"(d[9]), "=r"(d[10]),
                               "=r"(d[11]), "=r"(d[12]), "=r"(d[13]), "=r"(d[14]), "=r"(d[15]), "=r"(d[16]), "=r"(d[17]), "=r"(d[18]), "=r"(d[19]), "=r"(d[20]), "=r"(d[21]),
                               "=r"(d[22]), "=r"(d[23]), "=r"(d[24]), "=r"(d[25]), "=r"(d[26]), "=r"(d[27]), "=r"(d[28]), "=r"(d[29]), "=r"(d[30]), "=r"(d[31])
                             : "r"(tmem + ((uint32_t)(q * 32) << 16) + (uint32_t)(b * BN + c)));
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                const int col = n0 + c;
                if (row >= mend || col >= a.n) continue;
                if (BLOCK && col >= a.b.exact) {            // 16 (gate, up) pairs
                    uint16_t *y = (uint16_t *)a.b.y3 + (size_t)row * a.b.ld3 + (col - a.b.exact) / 2;
                    float v[16];
#pragma unroll
                    for (int i = 0; i < 16; ++i) v[i] = clamped_glu(__uint_as_float(d[2 * i]), __uint_as_float(d[2 * i + 1]), a.b.limit);
                    if (col + 32 <= a.n) {
#pragma unroll
                        for (int i = 0; i < 4; ++i) st4(y + 4 * i, make_float4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]));
                    } else {
#pragma unroll
                        for (int i = 0; i < 16; ++i) if (col + 2 * i < a.n) y[i] = f2bf(v[i]);
                    }
                    continue;
                }
                if (BLOCK) {
                    if (col < a.b.silu) {
#pragma unroll
                        for (int i = 0; i < 32; ++i) if (col + i < a.b.silu) d[i] = __float_as_uint(act_apply(__uint_as_float(d[i]), FKL_ACT_SILU));
                    }
                } else {
#pragma unroll
                    for (int i = 0; i < 32; ++i) d[i] = __float_as_uint(act_apply(__uint_as_float(d[i]), a.act) * a.scale);
                }
                const bool whole = col + 32 <= a.n, exact = BLOCK && col >= a.b.plain;
                if (a.out_f32 || exact) {
                    const int ld = exact ? a.b.exact - a.b.plain : a.ldy;
                    float *y = exact ? a.b.y2 + (size_t)row * ld + col - a.b.plain : (float *)a.y + (size_t)row * ld + col;
                    if (whole && (ld & 3) == 0) {
#pragma unroll
                        for (int i = 0; i < 8; ++i) reinterpret_cast<uint4 *>(y)[i] = make_uint4(d[4 * i], d[4 * i + 1], d[4 * i + 2], d[4 * i + 3]);
                    } else {
#pragma unroll
                        for (int i = 0; i < 32; ++i) if (col + i < a.n) y[i] = __uint_as_float(d[i]);
                    }
                } else {
                    uint16_t *y = (uint16_t *)a.y + (size_t)row * a.ldy + col;
                    if (whole && (a.ldy & 7) == 0) {
#pragma unroll
                        for (int i = 0; i < 4; ++i) {
                            uint32_t w[4];
#pragma unroll
                            for (int p = 0; p < 4; ++p) {
                                const __nv_bfloat162 h = __floats2bfloat162_rn(__uint_as_float(d[8 * i + 2 * p]), __uint_as_float(d[8 * i + 2 * p + 1]));
                                w[p] = *reinterpret_cast<const uint32_t *>(&h);
                            }
                            reinterpret_cast<uint4 *>(y)[i] = make_uint4(w[0], w[1], w[2], w[3]);
                        }
                    } else {
#pragma unroll
                        for (int i = 0; i < 32; ++i) if (col + i < a.n) y[i] = f2bf(__uint_as_float(d[i]));
                    }
                }
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) tcg_arrive(aempty + 8 * b);
        }
        if (!ok && lane == 0) atomicOr(&st->error, FKL_ERR_TC_WAIT);
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    if (wid == 2) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"((uint32_t)T::COLS) : "memory");
}
