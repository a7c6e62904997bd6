// Kernels of the parallel blocks beside the products and the attention: the residual add with a layer norm, joint q/k norm with
// rotation and cache store, linear recurrences (a decayed sum of k v^T; a matrix memory with exponential gates), norm and gate.
//
// A recurrence's state belongs to a (head, slice of 64 value columns): S [dim][64] in fp32, for the matrix memory followed by its
// normaliser n [dim] and running maximum m (every slice keeps its own copy, so slices never read what another one writes).  At
// position 0 the stored state is not read: a sequence starts from zeros whoever had the slot before.
#pragma once
#include "fk_layer_ops.cuh"

// ---------------------------------------------------------------- residual add, then a layer norm (or RMS norm) per row
// x <- x + scale * sum_{p < nnorm} norm(y_p) * post_p + the other y_p;  h <- norm(x) * w (+ b, then a layer norm)
struct BlockNormArgs {
    const float *x; const void *y[3]; const uint16_t *post; float *x_out; const uint16_t *w, *b; void *h; const uint32_t *index;
    int d, ldh, ldy, np, nnorm; float eps, scale;
};
// four values as they are stored
template <typename T> struct Raw4;
template <> struct Raw4<uint16_t> {
    uint2 v;
    __device__ __forceinline__ void load(const uint16_t *p) { v = __ldcg(reinterpret_cast<const uint2 *>(p)); }
    __device__ __forceinline__ void zero() { v = make_uint2(0, 0); }
    __device__ __forceinline__ float4 get() const { return make_float4(bf_lo(v.x), bf_hi(v.x), bf_lo(v.y), bf_hi(v.y)); }
};
template <> struct Raw4<float> {
    float4 v;
    __device__ __forceinline__ void load(const float *p) { v = __ldcg(reinterpret_cast<const float4 *>(p)); }
    __device__ __forceinline__ void zero() { v = make_float4(0.0f, 0.0f, 0.0f, 0.0f); }
    __device__ __forceinline__ float4 get() const { return v; }
};
// sums over a block of up to 32 warps with one barrier: every warp adds up all warps' parts.  Each call of a kernel has buffers of its own.
template <int N> __device__ __forceinline__ void block_sums(float (&v)[N], float (*buf)[32]) {
    const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = blockDim.x >> 5;
#pragma unroll
    for (int i = 0; i < N; ++i) { v[i] = warp_sum(v[i]); if (lane == 0) buf[i][wid] = v[i]; }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] = warp_sum(lane < nw ? buf[i][lane] : 0.0f);
}
__device__ __forceinline__ float4 bf4(uint2 v) { return make_float4(bf_lo(v.x), bf_hi(v.x), bf_lo(v.y), bf_hi(v.y)); }
// rows of a multiple of 4 and at most NV * 4 * blockDim.x values: everything in registers, one round of loads, weights ahead of the sums
template <typename T, int NV, int NT, int BLOCKS>
__global__ void __launch_bounds__(NT, BLOCKS) k_block_norm_rows4(const FkState *st, BlockNormArgs a) {
    __shared__ float red[5][32];
    const int tid = threadIdx.x, nt = blockDim.x;
    pdl_wait(); pdl_launch_dependents();
    const size_t row = a.index ? a.index[blockIdx.x] : blockIdx.x;
    float4 x[NV];
    Raw4<T> y[3][NV];
    uint2 w0[NV], w1[NV];                               // post weights, then the norm's weights
#pragma unroll
    for (int v = 0; v < NV; ++v) {
        const int i = (v * nt + tid) * 4;
        x[v] = i < a.d ? ld4(a.x + row * a.d + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
        for (int p = 0; p < 3; ++p) { if (p < a.np && i < a.d) y[p][v].load((const T *)a.y[p] + row * a.ldy + i); else y[p][v].zero(); }
        w0[v] = a.nnorm > 0 && i < a.d ? __ldg(reinterpret_cast<const uint2 *>(a.post + i)) : make_uint2(0, 0);
        w1[v] = a.nnorm > 1 && i < a.d ? __ldg(reinterpret_cast<const uint2 *>(a.post + a.d + i)) : make_uint2(0, 0);
    }
    if (a.nnorm > 0) {
        float f[3] = {};
#pragma unroll
        for (int p = 0; p < 3; ++p)
#pragma unroll
            for (int v = 0; v < NV; ++v) { const float4 e = y[p][v].get(); f[p] = fmaf(e.x, e.x, fmaf(e.y, e.y, fmaf(e.z, e.z, fmaf(e.w, e.w, f[p])))); }
        block_sums(f, red);
#pragma unroll
        for (int p = 0; p < 3; ++p) {
            const float s = a.scale * inv_rms(f[p], a.d, a.eps);
#pragma unroll
            for (int v = 0; v < NV; ++v) {
                const int i = (v * nt + tid) * 4;
                if (p >= a.nnorm || i >= a.d) continue;
                const float4 e = y[p][v].get(), w = p == 0 ? bf4(w0[v]) : p == 1 ? bf4(w1[v]) : ld4(a.post + (size_t)2 * a.d + i);
                x[v].x = fmaf(e.x * s, w.x, x[v].x); x[v].y = fmaf(e.y * s, w.y, x[v].y); x[v].z = fmaf(e.z * s, w.z, x[v].z); x[v].w = fmaf(e.w * s, w.w, x[v].w);
            }
        }
    }
    float sum[1] = {0.0f};
#pragma unroll
    for (int v = 0; v < NV; ++v) {
        const int i = (v * nt + tid) * 4;
#pragma unroll
        for (int p = 0; p < 3; ++p) if (p >= a.nnorm && p < a.np) { const float4 e = y[p][v].get(); x[v].x += e.x; x[v].y += e.y; x[v].z += e.z; x[v].w += e.w; }
        sum[0] += (x[v].x + x[v].y) + (x[v].z + x[v].w);
        if (a.x_out && i < a.d) st4(a.x_out + row * a.d + i, x[v]);
        w0[v] = i < a.d ? __ldg(reinterpret_cast<const uint2 *>(a.w + i)) : make_uint2(0, 0);
        w1[v] = a.b && i < a.d ? __ldg(reinterpret_cast<const uint2 *>(a.b + i)) : make_uint2(0, 0);
    }
    float mean = 0.0f;
    if (a.b) { block_sums(sum, red + 3); mean = sum[0] / (float)a.d; }
    float ss[1] = {0.0f};
#pragma unroll
    for (int v = 0; v < NV; ++v) if ((v * nt + tid) * 4 < a.d) {
        const float d0 = x[v].x - mean, d1 = x[v].y - mean, d2 = x[v].z - mean, d3 = x[v].w - mean;
        ss[0] = fmaf(d0, d0, fmaf(d1, d1, fmaf(d2, d2, fmaf(d3, d3, ss[0]))));
    }
    block_sums(ss, red + 4);
    const float r = inv_rms(ss[0], a.d, a.eps);
#pragma unroll
    for (int v = 0; v < NV; ++v) {
        const int i = (v * nt + tid) * 4;
        if (i >= a.d) continue;
        const float4 w = bf4(w0[v]), b = bf4(w1[v]);
        st4((T *)a.h + (size_t)blockIdx.x * a.ldh + i, make_float4(fmaf((x[v].x - mean) * r, w.x, b.x), fmaf((x[v].y - mean) * r, w.y, b.y),
                                                                   fmaf((x[v].z - mean) * r, w.z, b.z), fmaf((x[v].w - mean) * r, w.w, b.w)));
    }
}
template <typename T>
__global__ void __launch_bounds__(256) k_block_norm_rows(const FkState *st, BlockNormArgs a) {      // any width
    extern __shared__ float xs[];                       // [d]
    __shared__ float red[40];
    pdl_wait(); pdl_launch_dependents();
    const size_t row = a.index ? a.index[blockIdx.x] : blockIdx.x;
    float f[3] = {1.0f, 1.0f, 1.0f};
    for (int p = 0; p < a.nnorm; ++p) {
        float ss = 0.0f;
        for (int i = threadIdx.x; i < a.d; i += blockDim.x) { const float v = ldT((const T *)a.y[p] + row * a.ldy + i); ss = fmaf(v, v, ss); }
        f[p] = a.scale * inv_rms(block_sum(ss, red), a.d, a.eps);
    }
    float sum = 0.0f;
    for (int i = threadIdx.x; i < a.d; i += blockDim.x) {
        float v = a.x[row * a.d + i];
        for (int p = 0; p < a.np; ++p) v = fmaf(ldT((const T *)a.y[p] + row * a.ldy + i) * f[p], p < a.nnorm ? bf2f(a.post[(size_t)p * a.d + i]) : 1.0f, v);
        xs[i] = v; sum += v;
        if (a.x_out) a.x_out[row * a.d + i] = v;
    }
    const float mean = a.b ? block_sum(sum, red) / (float)a.d : 0.0f;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < a.d; i += blockDim.x) { const float v = xs[i] - mean; ss = fmaf(v, v, ss); }
    const float r = inv_rms(block_sum(ss, red), a.d, a.eps);
    T *h = (T *)a.h + (size_t)blockIdx.x * a.ldh;
    for (int i = threadIdx.x; i < a.d; i += blockDim.x) stT(h + i, fmaf((xs[i] - mean) * r, bf2f(a.w[i]), a.b ? bf2f(a.b[i]) : 0.0f));
}

// ---------------------------------------------------------------- joint q/k norm, rotation and the cache store of M positions
// One block per position.  q (all heads) and k (all heads) are each divided by their root mean square over all rows, scaled, rotated
// by the position's table row; q goes to a buffer of its own, k and v into the caches (layouts as in k_qk_norm_store_rows).
struct RotaryStoreArgs { const void *qkv; const uint16_t *qn, *kn; void *q, *ck, *cv; const float *rot; int H, G, dim, vdim, dpad, vpad, cap, ld, rot_dims; float eps; };
template <typename T>
__global__ void __launch_bounds__(256) k_rotary_store_rows(FkState *st, RotaryStoreArgs a) {
    __shared__ float red[66];
    pdl_wait(); pdl_launch_dependents();
    const int tid = threadIdx.x, row = blockIdx.x, nq = a.H * a.dim, nk = a.G * a.dim, nv = a.G * a.vdim;
    const uint32_t pos = st->offset + (uint32_t)row;
    if (pos >= (uint32_t)a.cap) { if (tid == 0) atomicOr(&st->error, FKL_ERR_CAPACITY); return; }
    const T *src = (const T *)a.qkv + (size_t)row * a.ld;
    float sq = 0.0f, sk = 0.0f;
    for (int i = tid; i < nq; i += 256) { const float v = ldT(src + i); sq = fmaf(v, v, sq); }
    for (int i = tid; i < nk; i += 256) { const float v = ldT(src + nq + i); sk = fmaf(v, v, sk); }
    const float2 s = block_sum2(sq, sk, red);
    const float rq = inv_rms(s.x, nq, a.eps), rk = inv_rms(s.y, nk, a.eps);
    const float *rot = a.rot ? a.rot + (size_t)pos * a.rot_dims : nullptr;
    for (int i = tid; i < nq + nk; i += 256) {
        const bool isq = i < nq;
        const int j = isq ? i : i - nq, head = j / a.dim, d = j - head * a.dim;
        const uint16_t *w = isq ? a.qn : a.kn; const float r = isq ? rq : rk;
        float v = ldT(src + i) * r * bf2f(w[j]);
        if (rot && d < a.rot_dims) {
            const int o = (d & 1) ? -1 : 1;             // the pair's other dimension
            v = rotate_dim(v, ldT(src + i + o) * r * bf2f(w[j + o]), d, a.rot_dims, rot);
        }
        stT(isq ? (T *)a.q + ((size_t)row * a.H + head) * a.dpad + d : (T *)a.ck + ((size_t)head * a.cap + pos) * a.dpad + d, v);
    }
    for (int i = tid; i < nv; i += 256) { const int g = i / a.vdim; ((T *)a.cv)[((size_t)g * a.cap + pos) * a.vpad + i - g * a.vdim] = src[nq + nk + i]; }
}

// ---------------------------------------------------------------- a mixer's joined heads: RMS norm in groups, scale, gate
struct NormGateArgs { const void *o; const uint16_t *w; const void *gate; void *out; int n, group, ldo, ldg, ld; float eps; };
template <typename T>
__global__ void __launch_bounds__(256) k_norm_gate_rows(const FkState *st, NormGateArgs a) {
    __shared__ float red[40], inv[FKL_GV_MAX_GROUPS];
    pdl_wait(); pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, wid = tid >> 5, ng = a.n / a.group;
    const T *o = (const T *)a.o + (size_t)blockIdx.x * a.ldo, *gate = (const T *)a.gate + (size_t)blockIdx.x * a.ldg;
    if (ng == 1) {
        float ss = 0.0f;
        for (int i = tid; i < a.n; i += 256) { const float v = ldT(o + i); ss = fmaf(v, v, ss); }
        ss = block_sum(ss, red);
        if (tid == 0) inv[0] = inv_rms(ss, a.n, a.eps);
    } else for (int q = wid; q < ng; q += 8) {
        float ss = 0.0f;
        for (int i = lane; i < a.group; i += 32) { const float v = ldT(o + q * a.group + i); ss = fmaf(v, v, ss); }
        ss = warp_sum(ss);
        if (lane == 0) inv[q] = inv_rms(ss, a.group, a.eps);
    }
    __syncthreads();
    T *out = (T *)a.out + (size_t)blockIdx.x * a.ld;
    for (int i = tid; i < a.n; i += 256) stT(out + i, ldT(o + i) * inv[i / a.group] * bf2f(a.w[i]) * sigmoid_f(ldT(gate + i)));
}

// ---------------------------------------------------------------- linear recurrences, position by position
// S_t = keep_t S_(t-1) + add_t k_t v_t^T, o_t = S_t^T (qscale q_t).  Decay form (log_decay set: the heads' logarithms, then the decays themselves): keep = decay, add = 1.  Matrix
// memory (MEM): log gates i = cap tanh((zi + bi) / cap), f = log sigmoid(cap tanh((zf + bf) / cap)), m_t = max(f + m_(t-1), i),
// keep = exp(f + m_(t-1) - m_t), add = exp(i - m_t), n_t like S with k alone, and o_t over max(|n_t . q_t|, exp(-m_t)) + 1e-6.
// One block per (slice of 64 value columns, head); a thread holds RPT rows of one column in registers through all positions.
#define FKL_RC_COLS 64
#define FKL_RC_PARTS 8
#define FKL_RC_THREADS (FKL_RC_COLS * FKL_RC_PARTS)
struct RecArgs {
    const void *q, *k, *v; const float *logits; const uint16_t *bias; const float *log_decay; float *state; void *out;
    int heads, dim, vdim, rows, ld, ldl, ldo, sstride; float qscale, cap;
    float *seg; int segments, per;                       // chunk form: scratch, runs of chunks that are worked on side by side, chunks of a run
};
__host__ __device__ inline int rec_state_stride(int dim, bool mem) { return dim * FKL_RC_COLS + (mem ? (dim + 1 + 3) / 4 * 4 : 0); }
__device__ __forceinline__ float log_sigmoid_f(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float soft_cap_f(float z, float cap) { return cap * tanhf(z / cap); }

template <typename T, bool MEM, int RPT>
__global__ void __launch_bounds__(FKL_RC_THREADS) k_recurrence(FkState *st, RecArgs a) {
    constexpr int DIM = RPT * FKL_RC_PARTS;
    __shared__ __align__(16) float qs[2][DIM], ks[2][DIM];
    __shared__ float po[2][FKL_RC_PARTS][FKL_RC_COLS], pn[2][FKL_RC_THREADS / 32];
    const int tid = threadIdx.x, c = tid & 63, part = tid >> 6, head = blockIdx.y, col = blockIdx.x * FKL_RC_COLS + c;
    float *S = a.state + ((size_t)head * gridDim.x + blockIdx.x) * a.sstride;
    const bool fresh = st->offset == 0;                 // advanced by the head of the token before, long since finished
    float s[RPT], n = 0.0f, m = 0.0f;
#pragma unroll
    for (int j = 0; j < RPT; ++j) { const int d = part * RPT + j; s[j] = !fresh && d < a.dim ? __ldcg(S + d * FKL_RC_COLS + c) : 0.0f; }
    const bool own_n = MEM && c < RPT && part * RPT + c < a.dim;         // this thread keeps row part * RPT + c of the normaliser
    if (MEM && !fresh) { if (own_n) n = __ldcg(S + a.dim * FKL_RC_COLS + part * RPT + c); m = __ldcg(S + a.dim * FKL_RC_COLS + a.dim); }
    const float bi = MEM ? bf2f(a.bias[head]) : 0.0f, bf = MEM ? bf2f(a.bias[a.heads + head]) : 0.0f, decay = MEM ? 0.0f : a.log_decay[a.heads + head];
    pdl_wait(); pdl_launch_dependents();
    const T *q = (const T *)a.q + head * a.dim, *k = (const T *)a.k + head * a.dim, *v = (const T *)a.v + head * a.vdim;
    float rq = 0.0f, rk = 0.0f, rv = 0.0f, ri = 0.0f, rf = 0.0f;
    auto request = [&](int t) {
        if (t >= a.rows) return;
        if (tid < a.dim) { rq = ldT(q + (size_t)t * a.ld + tid); rk = ldT(k + (size_t)t * a.ld + tid); }
        rv = col < a.vdim ? ldT(v + (size_t)t * a.ld + col) : 0.0f;
        if (MEM) { ri = a.logits[(size_t)t * a.ldl + head]; rf = a.logits[(size_t)t * a.ldl + a.heads + head]; }
    };
    float floor_ = 0.0f;                                // exp(-m) of the position whose sums are being folded
    auto finish = [&](int t) {                          // fold the parts of position t
        if (tid >= FKL_RC_COLS || col >= a.vdim) return;
        const int p = t & 1;
        float o = 0.0f;
#pragma unroll
        for (int i = 0; i < FKL_RC_PARTS; ++i) o += po[p][i][c];
        if (MEM) {
            float d = 0.0f;
#pragma unroll
            for (int i = 0; i < FKL_RC_THREADS / 32; ++i) d += pn[p][i];
            o /= fmaxf(fabsf(d), floor_) + 1e-6f;
        }
        stT((T *)a.out + (size_t)t * a.ldo + head * a.vdim + col, o);
    };
    request(0);
    for (int t = 0; t < a.rows; ++t) {
        const int p = t & 1;
        if (tid < DIM) { qs[p][tid] = tid < a.dim ? rq * a.qscale : 0.0f; ks[p][tid] = tid < a.dim ? rk : 0.0f; }
        const float vv = rv; float keep = decay, add = 1.0f, fl = 0.0f;
        if (MEM) {
            const float i = soft_cap_f(ri + bi, a.cap), f = log_sigmoid_f(soft_cap_f(rf + bf, a.cap)), mn = fmaxf(f + m, i);
            keep = expf(f + m - mn); add = expf(i - mn); m = mn; fl = expf(-mn);
        }
        __syncthreads();
        request(t + 1);
        if (t > 0) finish(t - 1);
        floor_ = fl;
        const float x = add * vv;
        float o = 0.0f;
#pragma unroll
        for (int j = 0; j < RPT; j += 4) {
            const float4 kk = *reinterpret_cast<const float4 *>(&ks[p][part * RPT + j]), qq = *reinterpret_cast<const float4 *>(&qs[p][part * RPT + j]);
            s[j] = fmaf(keep, s[j], kk.x * x); o = fmaf(s[j], qq.x, o); s[j + 1] = fmaf(keep, s[j + 1], kk.y * x); o = fmaf(s[j + 1], qq.y, o);
            s[j + 2] = fmaf(keep, s[j + 2], kk.z * x); o = fmaf(s[j + 2], qq.z, o); s[j + 3] = fmaf(keep, s[j + 3], kk.w * x); o = fmaf(s[j + 3], qq.w, o);
        }
        po[p][part][c] = o;
        if (MEM) {
            float d = 0.0f;
            if (own_n) { n = fmaf(keep, n, add * ks[p][part * RPT + c]); d = n * qs[p][part * RPT + c]; }
            d = warp_sum(d);
            if ((tid & 31) == 0) pn[p][tid >> 5] = d;
        }
    }
    __syncthreads();
    finish(a.rows - 1);
#pragma unroll
    for (int j = 0; j < RPT; ++j) { const int d = part * RPT + j; if (d < a.dim) S[d * FKL_RC_COLS + c] = s[j]; }
    if (MEM) { if (own_n) S[a.dim * FKL_RC_COLS + part * RPT + c] = n; if (tid == 0) S[a.dim * FKL_RC_COLS + a.dim] = m; }
}

// ---------------------------------------------------------------- linear recurrences, 64 positions at a time (bf16 rows)
// Inside a chunk, with F the running sum of the log keeps from the chunk's start (inclusive), a_s = i_s - F_s and
// M_t = max(m_0, max_{s <= t} a_s), position s enters position t with weight exp(a_s - M_t) and the state before the chunk with
// exp(m_0 - M_t); m_t = F_t + M_t.  The decay form is the same with i = 0 and M_t = -F_t (no maximum: m stays 0).  So
//   o_t = exp(m_0 - M_t) S_0^T q_t + sum_{s <= t} exp(a_s - M_t) (q_t . k_s) v_s,      S_end = exp(m_0 - M_end) S_0 + sum_s exp(a_s - M_end) k_s v_s^T
// are four small matrix products on the tensor cores (mma.m16n8k16).  fp32 factors (scores, weighted keys, the state) enter as two bf16 terms
// (hi + lo); the state itself stays in fp32 accumulators.
//
// The normaliser rides along as one more value column that is always 1.  exp(a_s - M_t) needs only F, a and the running maximum of a inside the
// chunk besides m_0, so the gates of several chunks are worked out at once, a warp each.
//
// One block per (slice of 64 value columns, head, run of chunks), two to an SM up to keys of 128.  With several runs, a first pass
// (OUT = false) leaves each run's own end state in scratch and the second starts every run from the fold of those before it.
#define FKL_CH 64
#define FKL_CH_THREADS 256
#define FKL_CH_GATES 4                // chunks whose gates are worked out together
template <int KD> struct ChunkSmem {
    static constexpr int KS = KD + 8, VS = FKL_RC_COLS + 8;
    static constexpr int K = FKL_CH * KS * 2, V = FKL_CH * VS * 2, Q = 2 * (K + V), SHI = Q + K, SLO = SHI + KD * VS * 2, TOTAL = SLO + KD * VS * 2;
};
__device__ __forceinline__ void ch_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ch_ldsm(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ch_ldsm_t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ uint32_t ch_pack(float lo, float hi) { const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi); return *reinterpret_cast<const uint32_t *>(&h); }
// two fp32 values as bf16 pairs hi + lo
__device__ __forceinline__ void ch_split(float x, float y, uint32_t &hi, uint32_t &lo) { hi = ch_pack(x, y); lo = ch_pack(x - bf_lo(hi), y - bf_hi(hi)); }

template <int KD, bool MEM, bool OUT>
__global__ void __launch_bounds__(FKL_CH_THREADS, KD <= 128 ? 2 : 1) k_recurrence_chunks(FkState *st, RecArgs a) {
    using L = ChunkSmem<KD>;
    constexpr int KS = L::KS, VS = L::VS, GR = FKL_CH_GATES;
    // state tiles of 16 rows: with fewer tiles than warps several warps share one, some columns each
    constexpr int TILES = KD / 16, MT = TILES > 8 ? TILES / 8 : 1, SHARE = TILES >= 8 ? 1 : 8 / TILES, NT = 8 / SHARE;
    extern __shared__ __align__(128) unsigned char ch_smem[];
    __shared__ float sF[GR][FKL_CH], sa[GR][FKL_CH], sX[GR][FKL_CH];      // F, a, running maximum of a inside the chunk
    const int tid = threadIdx.x, lane = tid & 31, wid = tid >> 5, g8 = lane >> 2, t4 = lane & 3;
    const int slice = blockIdx.x, head = blockIdx.y, run = blockIdx.z, col0 = slice * FKL_RC_COLS;
    const int chunk0 = run * a.per, nchunk = min((a.rows + FKL_CH - 1) / FKL_CH - chunk0, a.per);
    const size_t cell = (size_t)head * gridDim.x + slice, cells = (size_t)a.heads * gridDim.x;
    float *S = a.state + cell * a.sstride;
    const bool fresh = st->offset == 0;
    const float lgd = MEM ? 0.0f : a.log_decay[head], bi = MEM ? bf2f(a.bias[head]) : 0.0f, bf = MEM ? bf2f(a.bias[a.heads + head]) : 0.0f;
    pdl_wait(); pdl_launch_dependents();
    const uint32_t sbase = (uint32_t)__cvta_generic_to_shared(ch_smem), qb = sbase + L::Q, shi = sbase + L::SHI, slo = sbase + L::SLO;
    const uint16_t *gq = (const uint16_t *)a.q + head * a.dim, *gk = (const uint16_t *)a.k + head * a.dim, *gv = (const uint16_t *)a.v + head * a.vdim + col0;
    const int vcols = min(FKL_RC_COLS, a.vdim - col0);
    // rows of chunk c of this run; past the end and in padding columns zeros
    auto fetch_rows = [&](const uint16_t *g, uint32_t dst, int c) {
        const int r0 = (chunk0 + c) * FKL_CH;
        for (int i = tid; i < FKL_CH * (KD / 8); i += FKL_CH_THREADS) {
            const int r = i / (KD / 8), cc = (i - r * (KD / 8)) * 8; const bool v = r0 + r < a.rows && cc < a.dim;
            cp16_zfill(dst + (uint32_t)((r * KS + cc) * 2), v ? g + (size_t)(r0 + r) * a.ld + cc : g, v);
        }
    };
    auto fetch_kv = [&](int c) {
        const uint32_t kb = sbase + (uint32_t)((c & 1) * (L::K + L::V)), vb = kb + L::K;
        const int r0 = (chunk0 + c) * FKL_CH;
        fetch_rows(gk, kb, c);
        for (int i = tid; i < FKL_CH * (FKL_RC_COLS / 8); i += FKL_CH_THREADS) {
            const int r = i >> 3, cc = (i & 7) * 8; const bool v = r0 + r < a.rows && cc < vcols;
            cp16_zfill(vb + (uint32_t)((r * VS + cc) * 2), v ? gv + (size_t)(r0 + r) * a.ld + cc : gv, v);
        }
    };
    fetch_kv(0);
    if (OUT) fetch_rows(gq, qb, 0);
    asm volatile("cp.async.commit_group;" ::: "memory");
    auto gates = [&](int c) {                           // this warp: F, a and X of chunk c, two positions per lane
        const int r0 = (chunk0 + c) * FKL_CH + 2 * lane, p = c % GR;
        float f[2], i2[2];
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const bool v = r0 + j < a.rows;
            if (MEM) {
                const float zi = v ? a.logits[(size_t)(r0 + j) * a.ldl + head] : 0.0f, zf = v ? a.logits[(size_t)(r0 + j) * a.ldl + a.heads + head] : 0.0f;
                f[j] = v ? log_sigmoid_f(soft_cap_f(zf + bf, a.cap)) : 0.0f; i2[j] = v ? soft_cap_f(zi + bi, a.cap) : -INFINITY;
            } else { f[j] = v ? lgd : 0.0f; i2[j] = v ? 0.0f : -INFINITY; }
        }
        float F = f[0] + f[1];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) { const float t = __shfl_up_sync(0xffffffffu, F, o); if (lane >= o) F += t; }
        const float F0 = F - f[1], a0 = i2[0] - F0, a1 = i2[1] - F;
        sF[p][2 * lane] = F0; sF[p][2 * lane + 1] = F; sa[p][2 * lane] = a0; sa[p][2 * lane + 1] = a1;
        if (MEM) {
            float x = fmaxf(a0, a1);
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) { const float t = __shfl_up_sync(0xffffffffu, x, o); if (lane >= o) x = fmaxf(x, t); }
            const float before = __shfl_up_sync(0xffffffffu, x, 1);
            sX[p][2 * lane] = lane == 0 ? a0 : fmaxf(before, a0); sX[p][2 * lane + 1] = x;
        }
    };
    // ---- the state before the run: tile rows (16 of dim) x columns in accumulators; the normaliser in column 0 of a tile of its own
    const int tile0 = SHARE > 1 ? wid / SHARE : wid * MT, n0 = SHARE > 1 ? (wid % SHARE) * NT : 0;
    const uint32_t ones = g8 == 0 ? 0x3f803f80u : 0u;   // B fragment whose column 0 is 1
    float acc[MT][NT][4], accn[MEM ? MT : 1][4];
#pragma unroll
    for (int i = 0; i < MT; ++i) {
#pragma unroll
        for (int j = 0; j < NT; ++j) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.0f;
        if (MEM) accn[i][0] = accn[i][1] = accn[i][2] = accn[i][3] = 0.0f;
    }
    float m0 = 0.0f;
    auto add_state = [&](const float *src, float fa, float fb) {         // acc <- fa acc + fb src, the same for n
#pragma unroll
        for (int i = 0; i < MT; ++i)
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                const int d = (tile0 + i) * 16 + g8 + h * 8;
                if (d >= a.dim) continue;
#pragma unroll
                for (int j = 0; j < NT; ++j) {
                    const float2 v = __ldcg(reinterpret_cast<const float2 *>(src + d * FKL_RC_COLS + (n0 + j) * 8 + t4 * 2));
                    acc[i][j][2 * h] = fmaf(fa, acc[i][j][2 * h], fb * v.x); acc[i][j][2 * h + 1] = fmaf(fa, acc[i][j][2 * h + 1], fb * v.y);
                }
                if (MEM && t4 == 0) accn[i][2 * h] = fmaf(fa, accn[i][2 * h], fb * __ldcg(src + a.dim * FKL_RC_COLS + d));
            }
    };
    auto put_state = [&](float *dst, float m) {
#pragma unroll
        for (int i = 0; i < MT; ++i)
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                const int d = (tile0 + i) * 16 + g8 + h * 8;
                if (d >= a.dim) continue;
#pragma unroll
                for (int j = 0; j < NT; ++j) *reinterpret_cast<float2 *>(dst + d * FKL_RC_COLS + (n0 + j) * 8 + t4 * 2) = make_float2(acc[i][j][2 * h], acc[i][j][2 * h + 1]);
                if (MEM && n0 == 0 && t4 == 0) dst[a.dim * FKL_RC_COLS + d] = accn[i][2 * h];
            }
        if (MEM && tid == 0) dst[a.dim * FKL_RC_COLS + a.dim] = m;
    };
    // scratch: [runs + 1][cells][sstride], entry 0 the stored state, entry r + 1 what run r leaves (run 0: from the stored state); then
    // [runs][cells] sums of log keeps
    float *fsum = a.seg + (size_t)(a.segments + 1) * cells * a.sstride;
    auto seg = [&](int r) { return a.seg + ((size_t)r * cells + cell) * a.sstride; };
    if (a.segments == 1) {
        if (!fresh) { add_state(S, 0.0f, 1.0f); if (MEM) m0 = __ldcg(S + a.dim * FKL_RC_COLS + a.dim); }
    } else if (!OUT) {
        if (run == 0) {
            if (!fresh) { add_state(S, 0.0f, 1.0f); if (MEM) m0 = __ldcg(S + a.dim * FKL_RC_COLS + a.dim); }
            put_state(seg(0), m0);
        } else if (MEM) m0 = -INFINITY;                 // nothing seen yet
    } else if (run == 0) {
        add_state(seg(0), 0.0f, 1.0f);
        if (MEM) m0 = __ldcg(seg(0) + a.dim * FKL_RC_COLS + a.dim);
    } else {
        add_state(seg(1), 0.0f, 1.0f);
        if (MEM) m0 = __ldcg(seg(1) + a.dim * FKL_RC_COLS + a.dim);
        for (int r = 1; r < run; ++r) {
            const float F = __ldcg(fsum + (size_t)r * cells + cell);
            float fa = expf(F), fb = 1.0f;
            if (MEM) {
                const float ml = __ldcg(seg(r + 1) + a.dim * FKL_RC_COLS + a.dim), mn = fmaxf(F + m0, ml);
                fa = expf(F + m0 - mn); fb = expf(ml - mn); m0 = mn;
            }
            add_state(seg(r + 1), fa, fb);
        }
    }
    float Ftotal = 0.0f;
    for (int c = 0; c < nchunk; ++c) {
        const int p = c % GR;
        if (p == 0) {
            if (c > 0) __syncthreads();                 // the last chunks' gates have been read
            if (wid < GR && c + wid < nchunk) gates(c + wid);
        }
        if (OUT) {                                      // the state before this chunk as hi + lo
#pragma unroll
            for (int i = 0; i < MT; ++i)
#pragma unroll
                for (int h = 0; h < 2; ++h) {
                    const uint32_t row = (uint32_t)(((tile0 + i) * 16 + g8 + h * 8) * VS * 2);
                    uint32_t hi, lo;
#pragma unroll
                    for (int j = 0; j < NT; ++j) {
                        ch_split(acc[i][j][2 * h], acc[i][j][2 * h + 1], hi, lo);
                        const uint32_t at = row + (uint32_t)(((n0 + j) * 8 + t4 * 2) * 2);
                        asm volatile("st.shared.b32 [%0], %1;" ::"r"(shi + at), "r"(hi) : "memory");
                        asm volatile("st.shared.b32 [%0], %1;" ::"r"(slo + at), "r"(lo) : "memory");
                    }
                    if (MEM && n0 == 0) {               // columns 64 .. 71 (row padding): the normaliser and zeros
                        ch_split(accn[i][2 * h], 0.0f, hi, lo);
                        const uint32_t at = row + (uint32_t)((FKL_RC_COLS + t4 * 2) * 2);
                        asm volatile("st.shared.b32 [%0], %1;" ::"r"(shi + at), "r"(hi) : "memory");
                        asm volatile("st.shared.b32 [%0], %1;" ::"r"(slo + at), "r"(lo) : "memory");
                    }
                }
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        if (c + 1 < nchunk) { fetch_kv(c + 1); asm volatile("cp.async.commit_group;" ::: "memory"); }      // its stage was read a chunk ago
        const uint32_t kb = sbase + (uint32_t)((c & 1) * (L::K + L::V)), vb = kb + L::K;
        const float Fe = sF[p][FKL_CH - 1], Me = MEM ? fmaxf(m0, sX[p][FKL_CH - 1]) : -Fe;
        if (OUT) {
            // 16 positions x 32 columns of this warp; later positions have more to do, so the two warps of a scheduler take opposite ends
            const int hc = wid >> 2, wr = hc ? 3 - (wid & 3) : wid & 3, row0 = wr * 16;
            float s[8][4], o[4][4], nd[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
            for (int i = 0; i < 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
#pragma unroll
            for (int i = 0; i < 4; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
#pragma unroll 2
            for (int k = 0; k < KD / 16; ++k) {
                uint32_t q[4], b[4];
                ch_ldsm(q, qb + (uint32_t)(((row0 + (lane & 15)) * KS + k * 16 + (lane >> 4) * 8) * 2));
#pragma unroll
                for (int n = 0; n < 4; ++n) if (n <= wr) {
                    ch_ldsm(b, kb + (uint32_t)(((n * 16 + (lane & 7) + ((lane >> 4) << 3)) * KS + k * 16 + ((lane >> 3) & 1) * 8) * 2));
                    ch_mma(s[2 * n], q, b[0], b[1]); ch_mma(s[2 * n + 1], q, b[2], b[3]);
                }
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    const uint32_t at = (uint32_t)(((k * 16 + (lane & 15)) * VS + hc * 32 + n * 16 + (lane >> 4) * 8) * 2);
                    ch_ldsm_t(b, shi + at); ch_mma(o[2 * n], q, b[0], b[1]); ch_mma(o[2 * n + 1], q, b[2], b[3]);
                    ch_ldsm_t(b, slo + at); ch_mma(o[2 * n], q, b[0], b[1]); ch_mma(o[2 * n + 1], q, b[2], b[3]);
                }
                if (MEM) {                              // n . q: hi in the first two matrices, lo in the others
                    const uint32_t at = (uint32_t)(((k * 16 + (lane & 15)) * VS + FKL_RC_COLS) * 2);
                    ch_ldsm_t(b, (lane < 16 ? shi : slo) + at); ch_mma(nd, q, b[0], b[1]); ch_mma(nd, q, b[2], b[3]);
                }
            }
            const int ra = row0 + g8, rb = ra + 8;
            const float Ma = MEM ? fmaxf(m0, sX[p][ra]) : -sF[p][ra], Mb = MEM ? fmaxf(m0, sX[p][rb]) : -sF[p][rb], fa = expf(m0 - Ma) * a.qscale, fb = expf(m0 - Mb) * a.qscale;
#pragma unroll
            for (int i = 0; i < 4; ++i) { o[i][0] *= fa; o[i][1] *= fa; o[i][2] *= fb; o[i][3] *= fb; }
            float da = 0.0f, db = 0.0f;
#pragma unroll
            for (int n = 0; n < 4; ++n) if (n <= wr) {  // 16 positions s: weighted scores as hi + lo, times their values
                uint32_t ph[4], pl[4];
#pragma unroll
                for (int h = 0; h < 2; ++h) {
                    const int i = 2 * n + h, ka = i * 8 + t4 * 2;
                    const float a0 = sa[p][ka], a1 = sa[p][ka + 1];
                    const float x0 = ka <= ra ? s[i][0] * a.qscale * expf(a0 - Ma) : 0.0f, x1 = ka + 1 <= ra ? s[i][1] * a.qscale * expf(a1 - Ma) : 0.0f;
                    const float x2 = ka <= rb ? s[i][2] * a.qscale * expf(a0 - Mb) : 0.0f, x3 = ka + 1 <= rb ? s[i][3] * a.qscale * expf(a1 - Mb) : 0.0f;
                    da += x0 + x1; db += x2 + x3;
                    ch_split(x0, x1, ph[2 * h], pl[2 * h]); ch_split(x2, x3, ph[2 * h + 1], pl[2 * h + 1]);
                }
#pragma unroll
                for (int v = 0; v < 2; ++v) {
                    uint32_t b[4];
                    ch_ldsm_t(b, vb + (uint32_t)(((n * 16 + (lane & 15)) * VS + hc * 32 + v * 16 + (lane >> 4) * 8) * 2));
                    ch_mma(o[2 * v], ph, b[0], b[1]); ch_mma(o[2 * v + 1], ph, b[2], b[3]);
                    ch_mma(o[2 * v], pl, b[0], b[1]); ch_mma(o[2 * v + 1], pl, b[2], b[3]);
                }
            }
            __syncthreads();                            // q and the shared copy of the state have been read
            if (c + 1 < nchunk) { fetch_rows(gq, qb, c + 1); asm volatile("cp.async.commit_group;" ::: "memory"); }
            float na = 1.0f, nb = 1.0f;
            if (MEM) {
                da += __shfl_xor_sync(0xffffffffu, da, 1); da += __shfl_xor_sync(0xffffffffu, da, 2);
                db += __shfl_xor_sync(0xffffffffu, db, 1); db += __shfl_xor_sync(0xffffffffu, db, 2);
                da = fmaf(fa, __shfl_sync(0xffffffffu, nd[0], lane & 28), da); db = fmaf(fb, __shfl_sync(0xffffffffu, nd[2], lane & 28), db);
                na = 1.0f / (fmaxf(fabsf(da), expf(-(sF[p][ra] + Ma))) + 1e-6f); nb = 1.0f / (fmaxf(fabsf(db), expf(-(sF[p][rb] + Mb))) + 1e-6f);
            }
            const int r0 = (chunk0 + c) * FKL_CH;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int cc = hc * 32 + i * 8 + t4 * 2;
                if (cc >= vcols) continue;
                uint16_t *y = (uint16_t *)a.out + head * a.vdim + col0 + cc;
                if (r0 + ra < a.rows) *reinterpret_cast<uint32_t *>(y + (size_t)(r0 + ra) * a.ldo) = ch_pack(o[i][0] * na, o[i][1] * na);
                if (r0 + rb < a.rows) *reinterpret_cast<uint32_t *>(y + (size_t)(r0 + rb) * a.ldo) = ch_pack(o[i][2] * nb, o[i][3] * nb);
            }
        }
        // ---- the state after the chunk
        const float decay = expf(m0 - Me);
#pragma unroll
        for (int i = 0; i < MT; ++i) {
#pragma unroll
            for (int j = 0; j < NT; ++j) { acc[i][j][0] *= decay; acc[i][j][1] *= decay; acc[i][j][2] *= decay; acc[i][j][3] *= decay; }
            if (MEM) { accn[i][0] *= decay; accn[i][2] *= decay; }
        }
#pragma unroll
        for (int k = 0; k < 4; ++k) {                   // 16 positions
            uint32_t b[NT][2];
#pragma unroll
            for (int j = 0; j < NT; j += 2) {
                uint32_t r[4];
                ch_ldsm_t(r, vb + (uint32_t)(((k * 16 + (lane & 15)) * VS + (n0 + j) * 8 + (lane >> 4) * 8) * 2));
                b[j][0] = r[0]; b[j][1] = r[1]; b[j + 1][0] = r[2]; b[j + 1][1] = r[3];
            }
            const float *ak = sa[p] + k * 16 + t4 * 2;
            const float w0 = expf(ak[0] - Me), w1 = expf(ak[1] - Me), w2 = expf(ak[8] - Me), w3 = expf(ak[9] - Me);
#pragma unroll
            for (int i = 0; i < MT; ++i) {
                uint32_t x[4], hi[4], lo[4];
                ch_ldsm_t(x, kb + (uint32_t)(((k * 16 + ((lane >> 4) << 3) + (lane & 7)) * KS + (tile0 + i) * 16 + ((lane >> 3) & 1) * 8) * 2));
                ch_split(bf_lo(x[0]) * w0, bf_hi(x[0]) * w1, hi[0], lo[0]); ch_split(bf_lo(x[1]) * w0, bf_hi(x[1]) * w1, hi[1], lo[1]);
                ch_split(bf_lo(x[2]) * w2, bf_hi(x[2]) * w3, hi[2], lo[2]); ch_split(bf_lo(x[3]) * w2, bf_hi(x[3]) * w3, hi[3], lo[3]);
#pragma unroll
                for (int j = 0; j < NT; ++j) { ch_mma(acc[i][j], hi, b[j][0], b[j][1]); ch_mma(acc[i][j], lo, b[j][0], b[j][1]); }
                if (MEM) { ch_mma(accn[i], hi, ones, ones); ch_mma(accn[i], lo, ones, ones); }
            }
        }
        if (MEM) m0 = Fe + Me;
        Ftotal += Fe;
    }
    if (a.segments == 1) put_state(S, m0);
    else if (!OUT) { put_state(seg(run + 1), m0); if (tid == 0) fsum[(size_t)run * cells + cell] = Ftotal; }
    else if (run == a.segments - 1) put_state(S, m0);
}
