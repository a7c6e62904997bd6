// Kernels of the layered decoders: a residual stream in fp32, norms before and after every sublayer or one layer norm in front
// of a parallel block, (differential, rotary, windowed) attention with normed queries and keys and an output gate, mixture-of-experts
// feed-forward with a shared expert, clamped gated feed-forward.
//
// Two families.  The *row* kernels work on M consecutive positions (prompt portions); activations between the matrix
// products are T = bf16 or float, everything a norm, a router, a softmax or the residual touches is fp32.  The *decode*
// kernels work on one position with fp32 activations throughout: they are bound by the weights they stream, so the wider
// activations cost nothing.  Weights are bf16 rows [n, k] with k padded by zeros to a multiple of 64, so no product has a
// ragged K; activation buffers carry the same zero padding.
#pragma once
#include "fk_layer_ops.cuh"

// ---------------------------------------------------------------- embedding rows, fp32
struct EmbedRowsArgs { const uint16_t *table; float *x; const uint32_t *tokens; int d, vocab, ld; };
__global__ void k_embed_rows(FkState *st, EmbedRowsArgs a) {
    pdl_wait(); pdl_launch_dependents();
    const int m = blockIdx.x;
    uint32_t tok = a.tokens ? __ldcg(a.tokens + m) : st->token[m];
    if (tok >= (uint32_t)a.vocab) { if (threadIdx.x == 0) atomicOr(&st->error, FKL_ERR_TOKEN); tok = 0; }
    const uint16_t *src = a.table + (size_t)tok * a.ld; float *dst = a.x + (size_t)m * a.d;
    for (int i = threadIdx.x; i < a.d; i += blockDim.x) dst[i] = bf2f(src[i]);
}

// ---------------------------------------------------------------- residual add with post-norm, then the next pre-norm
// x <- x + norm(y) * post_w (+ add), h <- norm(x) * norm_w, per row.  y is a product's rows, or the rows of a mixture of
// experts: y (shared expert, may be absent) + sum_j weight[j] * moe_y[slot[j]].  `index` picks the rows that are wanted
// (final norm): output row r comes from row index[r] and x is not written.
struct ResNormArgs {
    const float *x; const void *y; const uint16_t *post_w; const float *add; float *x_out; const uint16_t *norm_w; void *h; const uint32_t *index;
    const void *moe_y; const int *slot; const float *weight; int d, ldh, top, ldy; float eps;
};
// rows of a multiple of 4 and at most NV * 4 * blockDim.x values: everything in registers, one round of loads
template <typename T, int NV>
__global__ void __launch_bounds__(256) k_residual_norm_rows4(const FkState *st, ResNormArgs a) {
    __shared__ float red[40];
    const int tid = threadIdx.x, nt = blockDim.x;
    pdl_wait(); pdl_launch_dependents();
    const size_t row = a.index ? a.index[blockIdx.x] : blockIdx.x;
    const bool pend = a.y || a.moe_y;
    float4 x[NV], y[NV];
#pragma unroll
    for (int v = 0; v < NV; ++v) {
        const int i = (v * nt + tid) * 4;
        x[v] = y[v] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (i < a.d) {
            x[v] = ld4(a.x + row * a.d + i);
            if (a.y) y[v] = ld4((const T *)a.y + row * a.ldy + i);
            if (a.add) { const float4 e = ld4(a.add + row * a.d + i); x[v].x += e.x; x[v].y += e.y; x[v].z += e.z; x[v].w += e.w; }
        }
    }
    if (a.moe_y) for (int j = 0; j < a.top; ++j) {
        const float w = a.weight[row * a.top + j]; const T *src = (const T *)a.moe_y + (size_t)a.slot[row * a.top + j] * a.ldy;
#pragma unroll
        for (int v = 0; v < NV; ++v) {
            const int i = (v * nt + tid) * 4;
            if (i < a.d) { const float4 e = ld4(src + i); y[v].x = fmaf(w, e.x, y[v].x); y[v].y = fmaf(w, e.y, y[v].y); y[v].z = fmaf(w, e.z, y[v].z); y[v].w = fmaf(w, e.w, y[v].w); }
        }
    }
    if (pend) {
        float ss = 0.0f;
#pragma unroll
        for (int v = 0; v < NV; ++v) ss = fmaf(y[v].x, y[v].x, fmaf(y[v].y, y[v].y, fmaf(y[v].z, y[v].z, fmaf(y[v].w, y[v].w, ss))));
        const float ry = inv_rms(block_sum(ss, red), a.d, a.eps);
#pragma unroll
        for (int v = 0; v < NV; ++v) {
            const int i = (v * nt + tid) * 4;
            if (i < a.d) {
                const float4 p = ld4(a.post_w + i);
                x[v].x = fmaf(y[v].x * ry, p.x, x[v].x); x[v].y = fmaf(y[v].y * ry, p.y, x[v].y); x[v].z = fmaf(y[v].z * ry, p.z, x[v].z); x[v].w = fmaf(y[v].w * ry, p.w, x[v].w);
            }
        }
    }
    float ss = 0.0f;
#pragma unroll
    for (int v = 0; v < NV; ++v) ss = fmaf(x[v].x, x[v].x, fmaf(x[v].y, x[v].y, fmaf(x[v].z, x[v].z, fmaf(x[v].w, x[v].w, ss))));
    const float r = inv_rms(block_sum(ss, red), a.d, a.eps);
#pragma unroll
    for (int v = 0; v < NV; ++v) {
        const int i = (v * nt + tid) * 4;
        if (i >= a.d) continue;
        if (a.x_out) st4(a.x_out + row * a.d + i, x[v]);
        const float4 w = ld4(a.norm_w + i);
        st4((T *)a.h + (size_t)blockIdx.x * a.ldh + i, make_float4(x[v].x * r * w.x, x[v].y * r * w.y, x[v].z * r * w.z, x[v].w * r * w.w));
    }
}
template <typename T>
__global__ void __launch_bounds__(512) k_residual_norm_rows(const FkState *st, ResNormArgs a) {
    extern __shared__ float xs[];                       // [d]
    __shared__ float red[40];
    pdl_wait(); pdl_launch_dependents();
    const size_t row = a.index ? a.index[blockIdx.x] : blockIdx.x;
    const float *x = a.x + row * a.d;
    float ry = 0.0f;
    const bool pend = a.y || a.moe_y;
    if (pend) {
        float ss = 0.0f;
        for (int i = threadIdx.x; i < a.d; i += blockDim.x) {
            float v = a.y ? ldT((const T *)a.y + row * a.ldy + i) : 0.0f;
            if (a.moe_y) for (int j = 0; j < a.top; ++j) v = fmaf(a.weight[row * a.top + j], ldT((const T *)a.moe_y + (size_t)a.slot[row * a.top + j] * a.ldy + i), v);
            xs[i] = v; ss = fmaf(v, v, ss);
        }
        ry = inv_rms(block_sum(ss, red), a.d, a.eps);
    }
    float ss = 0.0f;
    for (int i = threadIdx.x; i < a.d; i += blockDim.x) {
        float v = x[i];
        if (pend) v = fmaf(xs[i] * ry, bf2f(a.post_w[i]), v);
        if (a.add) v += a.add[row * a.d + i];
        xs[i] = v; ss = fmaf(v, v, ss);
        if (a.x_out) a.x_out[row * a.d + i] = v;
    }
    const float r = inv_rms(block_sum(ss, red), a.d, a.eps);
    T *h = (T *)a.h + (size_t)blockIdx.x * a.ldh;
    for (int i = threadIdx.x; i < a.d; i += blockDim.x) stT(h + i, xs[i] * r * bf2f(a.norm_w[i]));
}

// ---------------------------------------------------------------- matrix product on rows, CUDA cores
// Y[m, n] = act(sum_k X[m, k] W[row0 + n, k]); with `offsets` the rows of X are grouped by expert (expert e owns rows
// offsets[e] .. offsets[e + 1] - 1 and the weight rows e * N ..).  fp32 arithmetic: the product of the 32-bit mode.
// The joint projection of a parallel block stores its columns in three ways: [0, plain) as activations (a silu on the first `silu`),
// [plain, exact) as fp32, from `exact` on (gate, up) neighbours folded by the clamped gated unit.  All borders are multiples of 32.
struct BlockCols { float *y2; void *y3; int silu, plain, exact, ld3; float limit; };
struct LinRowsArgs { const float *x; const uint16_t *w; float *y; const int *offsets; int m, n, k, ldx, ldw, ldy, act; float scale; BlockCols b; };
template <bool BLOCK>
__global__ void __launch_bounds__(256) k_linear_rows(const FkState *st, LinRowsArgs a) {
    __shared__ float As[16][68], Bs[16][68];
    pdl_wait(); pdl_launch_dependents();
    int m0 = blockIdx.y * 64, mend = a.m; const uint16_t *w = a.w;
    if (a.offsets) {
        const int e = blockIdx.z, o = a.offsets[e];
        m0 += o; mend = a.offsets[e + 1]; w += (size_t)e * a.n * a.ldw;
    }
    if (m0 >= mend) return;
    const int n0 = blockIdx.x * 64, tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    float acc[4][4] = {};
    const int lr = tid >> 2, lk = (tid & 3) * 4;        // 64 rows x 16 k, four k per thread
    for (int k0 = 0; k0 < a.k; k0 += 16) {
        const int mr = m0 + lr, nr = n0 + lr;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            As[lk + j][lr] = mr < mend ? a.x[(size_t)mr * a.ldx + k0 + lk + j] : 0.0f;
            Bs[lk + j][lr] = nr < a.n ? bf2f(w[(size_t)nr * a.ldw + k0 + lk + j]) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 16; ++k) {
            const float4 av = *reinterpret_cast<const float4 *>(&As[k][ty * 4]), bv = *reinterpret_cast<const float4 *>(&Bs[k][tx * 4]);
            const float am[4] = {av.x, av.y, av.z, av.w}, bn[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(am[i], bn[j], acc[i][j]);
        }
        __syncthreads();
    }
    for (int i = 0; i < 4; ++i) for (int j = 0; j < 4; ++j) {
        const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
        if (m >= mend || n >= a.n) continue;
        if (!BLOCK) { a.y[(size_t)m * a.ldy + n] = act_apply(acc[i][j], a.act) * a.scale; continue; }
        if (n < a.b.plain) a.y[(size_t)m * a.ldy + n] = n < a.b.silu ? act_apply(acc[i][j], FKL_ACT_SILU) : acc[i][j];
        else if (n < a.b.exact) a.b.y2[(size_t)m * (a.b.exact - a.b.plain) + n - a.b.plain] = acc[i][j];
        else if (!(j & 1)) ((float *)a.b.y3)[(size_t)m * a.b.ld3 + (n - a.b.exact) / 2] = clamped_glu(acc[i][j], acc[i][j | 1], a.b.limit);
    }
}

// ---------------------------------------------------------------- q/k norm and the cache store of M positions
// Input rows q | k | v (| gate), heads laid out head by head with `maps` sub-heads of `dim` each.  q is normalised into a
// buffer of its own, k into the cache [G * maps, capacity, dpad], v is copied into [G, capacity, vpad] (padding stays zero).
struct QkStoreArgs { const void *qkv; const uint16_t *qn, *kn; void *q, *ck, *cv; int H, G, maps, dim, vdim, dpad, vpad, cap, rows, ld; float eps; };
template <typename T>
__global__ void __launch_bounds__(128) k_qk_norm_store_rows(FkState *st, QkStoreArgs a) {
    pdl_wait(); pdl_launch_dependents();
    const int lane = threadIdx.x & 31, item = blockIdx.y * 4 + (threadIdx.x >> 5), row = blockIdx.x;
    const int nq = a.H * a.maps, nk = a.G * a.maps;
    if (item >= nq + nk + a.G) return;
    const uint32_t pos = st->offset + (uint32_t)row;
    if (pos >= (uint32_t)a.cap) { if (lane == 0) atomicOr(&st->error, FKL_ERR_CAPACITY); return; }
    const T *src = (const T *)a.qkv + (size_t)row * a.ld;
    if (item >= nq + nk) {
        const int g = item - nq - nk;
        src += (nq + nk) * a.dim + g * a.vdim;
        T *dst = (T *)a.cv + ((size_t)g * a.cap + pos) * a.vpad;
        for (int i = lane; i < a.vdim; i += 32) dst[i] = src[i];
        return;
    }
    src += item * a.dim;
    const bool is_q = item < nq;
    T *dst = is_q ? (T *)a.q + ((size_t)row * nq + item) * a.dpad : (T *)a.ck + ((size_t)(item - nq) * a.cap + pos) * a.dpad;
    const uint16_t *w = is_q ? a.qn : a.kn;
    float ss = 0.0f;
    for (int i = lane; i < a.dim; i += 32) { const float v = ldT(src + i); ss = fmaf(v, v, ss); }
    const float r = inv_rms(warp_sum(ss), a.dim, a.eps);
    for (int i = lane; i < a.dim; i += 32) stT(dst + i, ldT(src + i) * r * bf2f(w[i]));
}

// ---------------------------------------------------------------- attention on CUDA cores (decode, and rows in 32-bit)
// One block per (key split, kv head x tile of 8 query rows, position).  The query rows of a kv head are its H / G heads
// times `maps`; all maps of a head sit in one tile.  A warp takes 32 keys at a time: scores with the lanes spread over
// (key, 8-wide slice of dim), online softmax with one key per lane, then the values with the lanes spread over vdim.
// Differential maps are combined at the end: a1 - lambda a2, unit rms over vdim, times 1 - diff; then the output gate.
// DECODE: one position; q and k come raw from the projection (fp32) and are normalised here, the new key and value go into
// the cache, and the keys are split over blocks (partials in global memory, the last block of a tile merges them).
#define FKL_ATT_ROWS 8
#define FKL_ATT_WARPS 8
struct AttnArgs {
    const float *qkv; const uint16_t *qn, *kn; const void *q; void *ck, *cv, *out; const void *gate; float *part; uint32_t *counter;
    int H, G, maps, dim, vdim, dpad, vpad, cap, ldo, ldg, splits, tiles; float scale, lambda, diff, eps;
    const float *rot;           // cos / sin of every position's pairs, [capacity][rot_dims], or null
    int rot_dims, joint, window, keep;          // joint: q (and k) rows are normed all together, a weight for each
};
__host__ __device__ inline size_t attn_smem_floats(int dpad, int vpad) {
    return (size_t)FKL_ATT_ROWS * dpad + FKL_ATT_WARPS * 32 * FKL_ATT_ROWS + FKL_ATT_WARPS * FKL_ATT_ROWS * ((size_t)vpad + 2) + FKL_ATT_ROWS * ((size_t)vpad + 2);
}
template <typename T, typename A, int VPL, bool DECODE>      // T: cache and q type; A: gate and output type
__global__ void __launch_bounds__(FKL_ATT_WARPS * 32) k_attention(FkState *st, AttnArgs a) {
    extern __shared__ float sm[];
    constexpr int RT = FKL_ATT_ROWS, NW = FKL_ATT_WARPS;
    float *qs = sm, *sc0 = qs + RT * a.dpad, *ow = sc0 + NW * 32 * RT, *mw = ow + (size_t)NW * RT * a.vpad, *of = mw + NW * RT * 2, *mf = of + RT * a.vpad;
    __shared__ int s_last;
    pdl_wait(); pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, wid = tid >> 5, row = blockIdx.z;
    const int g = blockIdx.y / a.tiles, tile = blockIdx.y - g * a.tiles, group = a.H / a.G, nrow_kv = group * a.maps;
    const int r0 = tile * RT, nr = min(RT, nrow_kv - r0);
    const uint32_t pos = st->offset + (uint32_t)row;
    if (pos >= (uint32_t)a.cap) { if (tid == 0) atomicOr(&st->error, FKL_ERR_CAPACITY); return; }
    const Visible vis = visible_keys((int)pos, a.window, a.keep);
    const int n = vis.n, per = ((n + a.splits - 1) / a.splits + 31) / 32 * 32;
    const int k0 = blockIdx.x * per, k1 = min(n, k0 + per);
    T *ck = (T *)a.ck + (size_t)g * a.maps * a.cap * a.dpad, *cv = (T *)a.cv + (size_t)g * a.cap * a.vpad;
    // ---- the query rows (normalised), and in decode the new key and value
    for (int i = tid; i < RT * a.dpad; i += NW * 32) qs[i] = 0.0f;
    __syncthreads();
    if (DECODE) {
        const bool mine = n - 1 >= k0 && n - 1 < k1;
        __shared__ float red[66];
        float2 joint = make_float2(0.0f, 0.0f);
        if (a.joint) {
            float sq = 0.0f, sk = 0.0f;
            for (int i = tid; i < a.H * a.dim; i += NW * 32) { const float v = a.qkv[i]; sq = fmaf(v, v, sq); }
            for (int i = tid; i < a.G * a.dim; i += NW * 32) { const float v = a.qkv[a.H * a.dim + i]; sk = fmaf(v, v, sk); }
            joint = block_sum2(sq, sk, red);
            joint = make_float2(inv_rms(joint.x, a.H * a.dim, a.eps), inv_rms(joint.y, a.G * a.dim, a.eps));
        }
        const float *rot = a.rot ? a.rot + (size_t)pos * a.rot_dims : nullptr;
        const int items = nr + (mine ? a.maps + 1 : 0);
        for (int it = wid; it < items; it += NW) {
            if (it == nr + a.maps) {
                const float *src = a.qkv + (a.H + a.G) * a.maps * a.dim + g * a.vdim;
                for (int i = lane; i < a.vdim; i += 32) stT(cv + (size_t)pos * a.vpad + i, src[i]);
                continue;
            }
            const bool is_q = it < nr;
            const float *src = a.qkv + (is_q ? (g * nrow_kv + r0 + it) : (a.H * a.maps + g * a.maps + (it - nr))) * a.dim;
            const uint16_t *w = (is_q ? a.qn : a.kn) + (a.joint ? (is_q ? g * nrow_kv + r0 + it : g) * a.dim : 0);
            float r = is_q ? joint.x : joint.y;
            if (!a.joint) {
                float ss = 0.0f;
                for (int i = lane; i < a.dim; i += 32) ss = fmaf(src[i], src[i], ss);
                r = inv_rms(warp_sum(ss), a.dim, a.eps);
            }
            for (int i = lane; i < a.dim; i += 32) {
                float v = src[i] * r * bf2f(w[i]);
                if (rot && i < a.rot_dims) v = rotate_dim(v, src[i ^ 1] * r * bf2f(w[i ^ 1]), i, a.rot_dims, rot);
                if (is_q) qs[it * a.dpad + i] = v; else stT(ck + ((size_t)(it - nr) * a.cap + pos) * a.dpad + i, v);
            }
        }
    } else {
        const T *q = (const T *)a.q + ((size_t)row * a.H * a.maps + g * nrow_kv + r0) * a.dpad;
        for (int i = tid; i < nr * a.dpad; i += NW * 32) qs[i] = ldT(q + i);
    }
    __syncthreads();
    // ---- keys
    int lpk = 1; while (lpk < 32 && lpk * 8 < a.dpad) lpk <<= 1;
    const int kpp = 32 / lpk, sub = lane & (lpk - 1), kin = lane / lpk;
    float *sc = sc0 + wid * 32 * RT;                   // [32 keys][RT]
    float mrow[RT], lrow[RT], o[RT][VPL];
#pragma unroll
    for (int r = 0; r < RT; ++r) { mrow[r] = -INFINITY; lrow[r] = 0.0f; for (int i = 0; i < VPL; ++i) o[r][i] = 0.0f; }
    for (int kb = k0 + wid * 32; kb < k1; kb += NW * 32) {
        const int nk = min(32, k1 - kb);
        for (int p0 = 0; p0 < nk; p0 += kpp) {
            const int kk = p0 + kin; const bool kv = kk < nk;
            for (int m = 0; m < a.maps; ++m) {
                const T *krow = ck + ((size_t)m * a.cap + vis.key(kb + (kv ? kk : 0))) * a.dpad;
                float dot[RT] = {};
                for (int d = sub * 8; d < a.dpad; d += lpk * 8) {
                    float kf[8]; load8(krow + d, kf);
#pragma unroll
                    for (int r = 0; r < RT; ++r) if (r < nr && (r0 + r) % a.maps == m) {
                        const float4 q0 = *reinterpret_cast<const float4 *>(qs + r * a.dpad + d), q1 = *reinterpret_cast<const float4 *>(qs + r * a.dpad + d + 4);
                        dot[r] = fmaf(q0.x, kf[0], fmaf(q0.y, kf[1], fmaf(q0.z, kf[2], fmaf(q0.w, kf[3], dot[r]))));
                        dot[r] = fmaf(q1.x, kf[4], fmaf(q1.y, kf[5], fmaf(q1.z, kf[6], fmaf(q1.w, kf[7], dot[r]))));
                    }
                }
#pragma unroll
                for (int r = 0; r < RT; ++r) if (r < nr && (r0 + r) % a.maps == m) {
                    float v = dot[r];
                    for (int s = lpk >> 1; s > 0; s >>= 1) v += __shfl_xor_sync(0xffffffffu, v, s);
                    if (sub == 0 && kv) sc[kk * RT + r] = v;
                }
            }
        }
        __syncwarp();
#pragma unroll
        for (int r = 0; r < RT; ++r) if (r < nr) {
            const float s = lane < nk ? sc[lane * RT + r] * a.scale : -INFINITY;
            const float mn = fmaxf(mrow[r], warp_max(s)), corr = expf(mrow[r] - mn), p = expf(s - mn);
            lrow[r] = lrow[r] * corr + warp_sum(p); mrow[r] = mn;
            sc[lane * RT + r] = p;
#pragma unroll
            for (int i = 0; i < VPL; ++i) o[r][i] *= corr;
        }
        __syncwarp();
        for (int k = 0; k < nk; ++k) {
            float v[VPL];
            const T *vrow = cv + (size_t)vis.key(kb + k) * a.vpad;
#pragma unroll
            for (int i = 0; i < VPL; ++i) { const int d = lane * VPL + i; v[i] = d < a.vpad ? ldT(vrow + d) : 0.0f; }
#pragma unroll
            for (int r = 0; r < RT; ++r) {
                const float p = r < nr ? sc[k * RT + r] : 0.0f;
#pragma unroll
                for (int i = 0; i < VPL; ++i) o[r][i] = fmaf(p, v[i], o[r][i]);
            }
        }
        __syncwarp();
    }
    // ---- fold the warps
#pragma unroll
    for (int r = 0; r < RT; ++r) {
#pragma unroll
        for (int i = 0; i < VPL; ++i) { const int d = lane * VPL + i; if (d < a.vpad) ow[((size_t)wid * RT + r) * a.vpad + d] = o[r][i]; }
        if (lane == 0) { mw[(wid * RT + r) * 2] = mrow[r]; mw[(wid * RT + r) * 2 + 1] = lrow[r]; }
    }
    __syncthreads();
    for (int i = tid; i < nr * a.vpad; i += NW * 32) {
        const int r = i / a.vpad, d = i - r * a.vpad;
        float mx = -INFINITY;
        for (int w = 0; w < NW; ++w) mx = fmaxf(mx, mw[(w * RT + r) * 2]);
        float s = 0.0f, l = 0.0f;
        for (int w = 0; w < NW; ++w) {
            const float f = mx == -INFINITY ? 0.0f : expf(mw[(w * RT + r) * 2] - mx);
            s = fmaf(f, ow[((size_t)w * RT + r) * a.vpad + d], s); l = fmaf(f, mw[(w * RT + r) * 2 + 1], l);
        }
        of[r * a.vpad + d] = a.splits > 1 ? s : s / l;
        if (d == 0) { mf[r * 2] = mx; mf[r * 2 + 1] = l; }
    }
    __syncthreads();
    if (a.splits > 1) {
        const size_t stride = (size_t)RT * (a.vpad + 2);
        float *mine = a.part + ((size_t)blockIdx.y * a.splits + blockIdx.x) * stride;
        for (int i = tid; i < nr * a.vpad; i += NW * 32) __stcg(mine + i, of[i]);
        for (int i = tid; i < nr * 2; i += NW * 32) __stcg(mine + RT * a.vpad + i, mf[i]);
        __threadfence();
        __syncthreads();
        if (tid == 0) { s_last = atomicAdd(a.counter + blockIdx.y, 1u) == (uint32_t)a.splits - 1u; if (s_last) a.counter[blockIdx.y] = 0u; }
        __syncthreads();
        if (!s_last) return;
        __threadfence();
        const float *base = a.part + (size_t)blockIdx.y * a.splits * stride;
        // factor of every (split, row): exp(m - max), into shared memory reused from the warp partials
        float *fac = ow;                                // [splits][RT]
        for (int i = tid; i < a.splits * nr; i += NW * 32) fac[(i / nr) * RT + i % nr] = __ldcg(base + (size_t)(i / nr) * stride + RT * a.vpad + (i % nr) * 2);
        __syncthreads();
        if (tid < nr) {
            float mx = -INFINITY, l = 0.0f;
            for (int s = 0; s < a.splits; ++s) mx = fmaxf(mx, fac[s * RT + tid]);
            for (int s = 0; s < a.splits; ++s) {
                const float f = expf(fac[s * RT + tid] - mx);
                fac[s * RT + tid] = f; l = fmaf(f, __ldcg(base + (size_t)s * stride + RT * a.vpad + tid * 2 + 1), l);
            }
            mf[tid * 2 + 1] = l;
        }
        __syncthreads();
        for (int i = tid; i < nr * a.vpad; i += NW * 32) {
            const int r = i / a.vpad;
            float s = 0.0f;
            for (int p = 0; p < a.splits; ++p) s = fmaf(fac[p * RT + r], __ldcg(base + (size_t)p * stride + i), s);
            of[i] = s / mf[r * 2 + 1];
        }
        __syncthreads();
    }
    // ---- combine the maps, gate, store
    for (int hh = wid; hh < nr / a.maps; hh += NW) {
        const int head = g * group + r0 / a.maps + hh;
        const float *o1 = of + hh * a.maps * a.vpad, *o2 = o1 + a.vpad;
        float f = 1.0f;
        if (a.maps == 2) {
            float ss = 0.0f;
            for (int d = lane; d < a.vdim; d += 32) { const float v = o1[d] - a.lambda * o2[d]; ss = fmaf(v, v, ss); }
            f = inv_rms(warp_sum(ss), a.vdim, a.eps) * (1.0f - a.diff);
        }
        if (a.gate) f *= sigmoid_f(ldT((const A *)a.gate + (size_t)row * a.ldg + head));
        A *out = (A *)a.out + (size_t)row * a.ldo + head * a.vdim;
        for (int d = lane; d < a.vdim; d += 32) stT(out + d, (a.maps == 2 ? o1[d] - a.lambda * o2[d] : o1[d]) * f);
    }
}

// ---------------------------------------------------------------- attention of one position, bf16 caches
// The same task as the DECODE form above, laid out for latency.  A block takes 64 keys at a time: the maps' keys and the values of
// a chunk arrive in shared memory by cp.async (two chunks in flight, the first two requested before the dependency wait: the
// cached rows are older than the kernel before this one), then a thread scores one key against two query rows, a warp runs the
// softmax of one row, and the threads spread over (value columns, key parts) for the weighted sum.  The new key and value, known
// only after the wait, go to the cache and straight into the last chunk.  Partials of the blocks meet in global memory; the last
// block of a (kv head, row tile) folds them, combines the maps and applies the gate.
#define FKL_AD_KEYS 64
#define FKL_AD_THREADS 256
#define FKL_AD_ROT 256               // rotated dimensions whose table row fits in shared memory
struct AdLayout { int ks, vs, stage, q, sc, pr, nk, nv, of, total; };      // byte offsets; ks / vs: row strides in elements
__host__ __device__ inline AdLayout ad_layout(int maps, int dpad, int vpad) {
    AdLayout l; l.ks = ((dpad / 8) | 1) * 8; l.vs = ((vpad / 8) | 1) * 8;           // odd multiples of 16 bytes
    l.stage = FKL_AD_KEYS * 2 * (maps * l.ks + l.vs);
    const int red = FKL_AD_THREADS * FKL_ATT_ROWS * 2 * 4;                           // the key parts' sums, over the chunk buffers
    l.q = 2 * l.stage > red ? 2 * l.stage : red;
    l.sc = l.q + FKL_ATT_ROWS * dpad * 4; l.pr = l.sc + FKL_ATT_ROWS * (FKL_AD_KEYS + 1) * 4; l.pr = (l.pr + 15) & ~15;
    l.nk = l.pr + FKL_AD_KEYS * FKL_ATT_ROWS * 4; l.nv = l.nk + ((maps * dpad * 2 + 15) & ~15); l.of = l.nv + ((vpad * 2 + 15) & ~15);
    l.total = l.of + FKL_ATT_ROWS * vpad * 4;
    return l;
}
__global__ void __launch_bounds__(FKL_AD_THREADS) k_attention_decode(FkState *st, AttnArgs a) {
    extern __shared__ __align__(128) unsigned char ad_smem[];
    constexpr int RT = FKL_ATT_ROWS, KC = FKL_AD_KEYS, NT = FKL_AD_THREADS;
    const AdLayout L = ad_layout(a.maps, a.dpad, a.vpad);
    float *qs = reinterpret_cast<float *>(ad_smem + L.q), *sc = reinterpret_cast<float *>(ad_smem + L.sc), *pr = reinterpret_cast<float *>(ad_smem + L.pr);
    uint16_t *nk = reinterpret_cast<uint16_t *>(ad_smem + L.nk), *nv = reinterpret_cast<uint16_t *>(ad_smem + L.nv);
    float *of = reinterpret_cast<float *>(ad_smem + L.of);
    __shared__ float s_corr[RT], s_m[RT], s_l[RT], s_fac[256 * RT], s_red[66], s_rot[FKL_AD_ROT]; __shared__ int s_last;
    const int tid = threadIdx.x, lane = tid & 31, wid = tid >> 5;
    const int g = blockIdx.y / a.tiles, tile = blockIdx.y - g * a.tiles, group = a.H / a.G, nrow_kv = group * a.maps, r0 = tile * RT, nr = min(RT, nrow_kv - r0);
    const uint32_t upos = st->offset;                   // advanced by the head of the token before, long since finished
    const int pos = (int)upos;
    const Visible vis = visible_keys(pos, a.window, a.keep);
    const int n = vis.n, newest = n - 1, per = ((n + a.splits - 1) / a.splits + KC - 1) / KC * KC, active = (n + per - 1) / per;
    const int k0 = blockIdx.x * per, k1 = min(n, k0 + per), nchunk = k1 > k0 ? (k1 - k0 + KC - 1) / KC : 0;
    const bool fits = upos < (uint32_t)a.cap;
    uint16_t *ck = (uint16_t *)a.ck + (size_t)g * a.maps * a.cap * a.dpad, *cv = (uint16_t *)a.cv + (size_t)g * a.cap * a.vpad;
    const uint32_t sbase = (uint32_t)__cvta_generic_to_shared(ad_smem);
    auto request = [&](int c) {                         // chunk c into stage c & 1; the new position's row comes from registers later
        const uint32_t kb = sbase + (uint32_t)((c & 1) * L.stage), vb = kb + (uint32_t)(a.maps * KC * L.ks * 2);
        const int kn = a.dpad / 8, vn = a.vpad / 8, key0 = k0 + c * KC;
        for (int i = tid; i < a.maps * KC * kn; i += NT) {
            const int r = i / kn, cc = (i - r * kn) * 8, key = key0 + (r & (KC - 1)); const bool v = key < newest;
            if (key != newest) cp16_zfill(kb + (uint32_t)((r * L.ks + cc) * 2), v ? ck + ((size_t)(r / KC) * a.cap + vis.key(key)) * a.dpad + cc : ck, v);
        }
        for (int i = tid; i < KC * vn; i += NT) {
            const int r = i / vn, cc = (i - r * vn) * 8, key = key0 + r; const bool v = key < newest;
            if (key != newest) cp16_zfill(vb + (uint32_t)((r * L.vs + cc) * 2), v ? cv + (size_t)vis.key(key) * a.vpad + cc : cv, v);
        }
    };
    if (fits) for (int c = 0; c < 2; ++c) { if (c < nchunk) request(c); asm volatile("cp.async.commit_group;" ::: "memory"); }
    // what else does not depend on the kernel before: rows without a query, the position's rotation, the norm weights of the warp's first item
    const bool mine = newest >= k0 && newest < k1;
    const int items = nr + (mine ? a.maps + 1 : 0);     // query rows, new keys, new value
    auto weight_of = [&](int it) { const bool is_q = it < nr; return (is_q ? a.qn : a.kn) + (a.joint ? (is_q ? g * nrow_kv + r0 + it : g) * a.dim : 0); };
    auto source_of = [&](int it) { return a.qkv + (it < nr ? (g * nrow_kv + r0 + it) : (a.H * a.maps + g * a.maps + (it - nr))) * a.dim; };
    float xv[4], wv[4];                                 // the first 128 values of the warp's item
#pragma unroll
    for (int j = 0; j < 4; ++j) { const int i = lane + j * 32; wv[j] = wid < items && wid != nr + a.maps && i < a.dim ? bf2f(weight_of(wid)[i]) : 0.0f; }
    for (int i = tid; i < (RT - nr) * a.dpad; i += NT) qs[nr * a.dpad + i] = 0.0f;
    const float *rot = a.rot && fits ? a.rot + (size_t)pos * a.rot_dims : nullptr;
    if (rot && a.rot_dims <= FKL_AD_ROT) { for (int i = tid; i < a.rot_dims; i += NT) s_rot[i] = rot[i]; rot = s_rot; __syncthreads(); }
    pdl_wait(); pdl_launch_dependents();
    if (!fits) { if (tid == 0) atomicOr(&st->error, FKL_ERR_CAPACITY); return; }
    if (nchunk == 0) return;                            // more splits than this many keys need
    // ---- query rows, and where the position falls here the new key and value
#pragma unroll
    for (int j = 0; j < 4; ++j) { const int i = lane + j * 32; xv[j] = wid < items && wid != nr + a.maps && i < a.dim ? __ldcg(source_of(wid) + i) : 0.0f; }
    float2 joint = make_float2(0.0f, 0.0f);
    if (a.joint) {
        const int nq = a.H * a.dim, nk = a.G * a.dim;
        float sq = 0.0f, sk = 0.0f;
        if ((((uintptr_t)a.qkv | (uintptr_t)(a.qkv + nq)) & 15) == 0 && (nq & 3) == 0 && (nk & 3) == 0) {
            const float4 *p = reinterpret_cast<const float4 *>(a.qkv);
            for (int b = tid; b < (nq + nk) / 4; b += 4 * NT) {
                float4 v[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) v[j] = b + j * NT < (nq + nk) / 4 ? __ldcg(p + b + j * NT) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float e = fmaf(v[j].x, v[j].x, fmaf(v[j].y, v[j].y, fmaf(v[j].z, v[j].z, v[j].w * v[j].w)));
                    if (b + j * NT < nq / 4) sq += e; else sk += e;
                }
            }
        } else {
            for (int i = tid; i < nq; i += NT) { const float v = __ldcg(a.qkv + i); sq = fmaf(v, v, sq); }
            for (int i = tid; i < nk; i += NT) { const float v = __ldcg(a.qkv + nq + i); sk = fmaf(v, v, sk); }
        }
        joint = block_sum2(sq, sk, s_red);
        joint = make_float2(inv_rms(joint.x, nq, a.eps), inv_rms(joint.y, nk, a.eps));
    }
    for (int it = wid; it < items; it += NT / 32) {
        if (it == nr + a.maps) {
            const float *src = a.qkv + (a.H + a.G) * a.maps * a.dim + g * a.vdim;
            for (int i = lane; i < a.vpad; i += 32) { const uint16_t v = i < a.vdim ? f2bf(__ldcg(src + i)) : (uint16_t)0; nv[i] = v; if (i < a.vdim) cv[(size_t)pos * a.vpad + i] = v; }
            continue;
        }
        const bool is_q = it < nr;
        const float *src = source_of(it);
        const uint16_t *w = weight_of(it);
        if (it != wid) {
#pragma unroll
            for (int j = 0; j < 4; ++j) { const int i = lane + j * 32; xv[j] = i < a.dim ? __ldcg(src + i) : 0.0f; wv[j] = i < a.dim ? bf2f(w[i]) : 0.0f; }
        }
        float r = is_q ? joint.x : joint.y;
        if (!a.joint) {
            float ss = 0.0f;
#pragma unroll
            for (int j = 0; j < 4; ++j) ss = fmaf(xv[j], xv[j], ss);
            for (int i = lane + 128; i < a.dim; i += 32) { const float v = __ldcg(src + i); ss = fmaf(v, v, ss); }
            r = inv_rms(warp_sum(ss), a.dim, a.eps);
        }
        auto put = [&](int i, float v) {
            if (rot) v = rotate_dim(v, __shfl_xor_sync(0xffffffffu, v, 1), i, a.rot_dims, rot);
            if (i >= a.dpad) return;
            if (is_q) qs[it * a.dpad + i] = v * a.scale;
            else { nk[(it - nr) * a.dpad + i] = f2bf(v); if (i < a.dim) ck[((size_t)(it - nr) * a.cap + pos) * a.dpad + i] = f2bf(v); }
        };
#pragma unroll
        for (int j = 0; j < 4; ++j) if (j * 32 < a.dpad) put(lane + j * 32, xv[j] * r * wv[j]);
        for (int i = lane + 128; i - lane < a.dpad; i += 32) put(i, i < a.dim ? __ldcg(src + i) * r * bf2f(w[i]) : 0.0f);
    }
    // ---- chunks
    int tpc = 1; while (tpc < NT && tpc < a.vpad / 2) tpc <<= 1;        // threads over pairs of value columns
    const int parts = NT / tpc, col = (tid & (tpc - 1)) * 2, part = tid / tpc;
    float o[RT][2];
#pragma unroll
    for (int r = 0; r < RT; ++r) o[r][0] = o[r][1] = 0.0f;
    float m = -INFINITY, l = 0.0f;                      // row `wid` of the softmax
    for (int c = 0; c < nchunk; ++c) {
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        const unsigned char *kb = ad_smem + (c & 1) * L.stage; unsigned char *kbw = ad_smem + (c & 1) * L.stage;
        const uint16_t *ks = reinterpret_cast<const uint16_t *>(kb), *vs = ks + a.maps * KC * L.ks;
        const int key0 = k0 + c * KC;
        if (mine && newest >= key0 && newest < key0 + KC) {
            uint16_t *kw = reinterpret_cast<uint16_t *>(kbw), *vw = kw + a.maps * KC * L.ks;
            for (int i = tid; i < a.maps * a.dpad; i += NT) { const int mm = i / a.dpad; kw[(mm * KC + newest - key0) * L.ks + i - mm * a.dpad] = nk[i]; }
            for (int i = tid; i < a.vpad; i += NT) vw[(newest - key0) * L.vs + i] = nv[i];
            __syncthreads();
        }
        {   // scores: key tid % 64, rows tid / 64 and 4 more (of the same map)
            const int key = tid & (KC - 1), ra = tid / KC, rb = ra + 4, mm = a.maps == 2 ? (ra & 1) : 0;
            const uint16_t *kr = ks + (mm * KC + key) * L.ks; const float *qa = qs + ra * a.dpad, *qb = qs + rb * a.dpad;
            float da = 0.0f, db = 0.0f;
            for (int d = 0; d < a.dpad; d += 8) {
                float f[8]; unpack8f(*reinterpret_cast<const uint4 *>(kr + d), f);
                const float4 a0 = *reinterpret_cast<const float4 *>(qa + d), a1 = *reinterpret_cast<const float4 *>(qa + d + 4);
                const float4 b0 = *reinterpret_cast<const float4 *>(qb + d), b1 = *reinterpret_cast<const float4 *>(qb + d + 4);
                da = fmaf(a0.x, f[0], fmaf(a0.y, f[1], fmaf(a0.z, f[2], fmaf(a0.w, f[3], fmaf(a1.x, f[4], fmaf(a1.y, f[5], fmaf(a1.z, f[6], fmaf(a1.w, f[7], da))))))));
                db = fmaf(b0.x, f[0], fmaf(b0.y, f[1], fmaf(b0.z, f[2], fmaf(b0.w, f[3], fmaf(b1.x, f[4], fmaf(b1.y, f[5], fmaf(b1.z, f[6], fmaf(b1.w, f[7], db))))))));
            }
            const bool v = key0 + key < k1;
            sc[ra * (KC + 1) + key] = v ? da : -INFINITY; sc[rb * (KC + 1) + key] = v ? db : -INFINITY;
        }
        __syncthreads();
        {   // softmax of row wid
            const float s0 = sc[wid * (KC + 1) + lane], s1 = sc[wid * (KC + 1) + lane + 32];
            const float mn = fmaxf(m, warp_max(fmaxf(s0, s1))), corr = expf(m - mn), p0 = expf(s0 - mn), p1 = expf(s1 - mn);
            l = l * corr + warp_sum(p0 + p1); m = mn;
            pr[lane * RT + wid] = p0; pr[(lane + 32) * RT + wid] = p1;
            if (lane == 0) s_corr[wid] = corr;
        }
        __syncthreads();
        if (col < a.vpad) {
#pragma unroll
            for (int r = 0; r < RT; ++r) { const float f = s_corr[r]; o[r][0] *= f; o[r][1] *= f; }
            const int nkey = min(KC, k1 - key0);
#pragma unroll 4
            for (int k = part; k < nkey; k += parts) {
                const uint32_t vv = *reinterpret_cast<const uint32_t *>(vs + k * L.vs + col);
                const float v0 = bf_lo(vv), v1 = bf_hi(vv);
                const float4 pa = *reinterpret_cast<const float4 *>(pr + k * RT), pb = *reinterpret_cast<const float4 *>(pr + k * RT + 4);
                const float p[RT] = {pa.x, pa.y, pa.z, pa.w, pb.x, pb.y, pb.z, pb.w};
#pragma unroll
                for (int r = 0; r < RT; ++r) { o[r][0] = fmaf(p[r], v0, o[r][0]); o[r][1] = fmaf(p[r], v1, o[r][1]); }
            }
        }
        __syncthreads();                                // the stage is free
        if (c + 2 < nchunk) request(c + 2);
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
    // ---- fold the key parts (chunk buffers reused; nothing is in flight: the groups above are empty)
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    if (lane == 0) { s_m[wid] = m; s_l[wid] = l; }
    float *red = reinterpret_cast<float *>(ad_smem);
    __syncthreads();
    for (int r = 0; r < RT; ++r) *reinterpret_cast<float2 *>(red + (r * NT + tid) * 2) = make_float2(o[r][0], o[r][1]);
    __syncthreads();
    for (int i = tid; i < nr * (a.vpad / 2); i += NT) {
        const int r = i / (a.vpad / 2), cp = i - r * (a.vpad / 2);
        float2 s = make_float2(0.0f, 0.0f);
        for (int p = 0; p < parts; ++p) { const float2 v = *reinterpret_cast<const float2 *>(red + (r * NT + p * tpc + cp) * 2); s.x += v.x; s.y += v.y; }
        const float f = active > 1 ? 1.0f : 1.0f / s_l[r];
        *reinterpret_cast<float2 *>(of + r * a.vpad + cp * 2) = make_float2(s.x * f, s.y * f);
    }
    __syncthreads();
    if (active > 1) {
        const size_t stride = (size_t)RT * (a.vpad + 2);
        const float *base = a.part + (size_t)blockIdx.y * a.splits * stride;
        float *mine_p = a.part + ((size_t)blockIdx.y * a.splits + blockIdx.x) * stride;
        for (int i = tid; i < RT * a.vpad / 4; i += NT) __stcg(reinterpret_cast<float4 *>(mine_p) + i, reinterpret_cast<const float4 *>(of)[i]);
        if (tid < RT) { __stcg(mine_p + RT * a.vpad + tid * 2, s_m[tid]); __stcg(mine_p + RT * a.vpad + tid * 2 + 1, s_l[tid]); }
        __threadfence();
        __syncthreads();
        if (tid == 0) { s_last = atomicAdd(a.counter + blockIdx.y, 1u) == (uint32_t)active - 1u; if (s_last) a.counter[blockIdx.y] = 0u; }
        __syncthreads();
        if (!s_last) return;
        __threadfence();
        // a thread folds four values; what the first splits left of them is requested before the factors are known
        constexpr int PRE = 8;
        float4 pre[PRE];
        const bool own = tid < nr * a.vpad / 4;
#pragma unroll
        for (int p = 0; p < PRE; ++p) pre[p] = own && p < active ? __ldcg(reinterpret_cast<const float4 *>(base + (size_t)p * stride) + tid) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        // factors exp(m - max) / sum of every (split, row): warp r takes row r (there are as many warps as rows of a tile)
        if (wid < nr) {
            const int r = wid;
            float2 ml[2];
#pragma unroll
            for (int j = 0; j < 2; ++j) ml[j] = lane + j * 32 < active ? __ldcg(reinterpret_cast<const float2 *>(base + (size_t)(lane + j * 32) * stride + RT * a.vpad) + r) : make_float2(-INFINITY, 0.0f);
            float mx = fmaxf(ml[0].x, ml[1].x);
            for (int p = lane + 64; p < active; p += 32) mx = fmaxf(mx, __ldcg(base + (size_t)p * stride + RT * a.vpad + r * 2));
            mx = warp_max(mx);
            float f0 = expf(ml[0].x - mx), f1 = expf(ml[1].x - mx), ls = fmaf(f0, ml[0].y, f1 * ml[1].y);
            for (int p = lane + 64; p < active; p += 32) ls = fmaf(expf(__ldcg(base + (size_t)p * stride + RT * a.vpad + r * 2) - mx), __ldcg(base + (size_t)p * stride + RT * a.vpad + r * 2 + 1), ls);
            const float inv = 1.0f / warp_sum(ls);
            if (lane < active) s_fac[lane * RT + r] = f0 * inv;
            if (lane + 32 < active) s_fac[(lane + 32) * RT + r] = f1 * inv;
            for (int p = lane + 64; p < active; p += 32) s_fac[p * RT + r] = expf(__ldcg(base + (size_t)p * stride + RT * a.vpad + r * 2) - mx) * inv;
        }
        __syncthreads();
        for (int i = tid; i < nr * a.vpad / 4; i += NT) {
            const int r = i * 4 / a.vpad;
            float4 s = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            int p = 0;
            if (i == tid) {
#pragma unroll
                for (int q = 0; q < PRE; ++q) if (q < active) {
                    const float f = s_fac[q * RT + r];
                    s.x = fmaf(f, pre[q].x, s.x); s.y = fmaf(f, pre[q].y, s.y); s.z = fmaf(f, pre[q].z, s.z); s.w = fmaf(f, pre[q].w, s.w);
                }
                p = PRE;
            }
#pragma unroll 8
            for (; p < active; ++p) {
                const float4 v = __ldcg(reinterpret_cast<const float4 *>(base + (size_t)p * stride) + i); const float f = s_fac[p * RT + r];
                s.x = fmaf(f, v.x, s.x); s.y = fmaf(f, v.y, s.y); s.z = fmaf(f, v.z, s.z); s.w = fmaf(f, v.w, s.w);
            }
            reinterpret_cast<float4 *>(of)[i] = s;
        }
        __syncthreads();
    }
    for (int hh = wid; hh < nr / a.maps; hh += NT / 32) {
        const int head = g * group + r0 / a.maps + hh;
        const float *o1 = of + hh * a.maps * a.vpad, *o2 = o1 + a.vpad;
        float f = 1.0f;
        if (a.maps == 2) {
            float ss = 0.0f;
            for (int d = lane; d < a.vdim; d += 32) { const float v = o1[d] - a.lambda * o2[d]; ss = fmaf(v, v, ss); }
            f = inv_rms(warp_sum(ss), a.vdim, a.eps) * (1.0f - a.diff);
        }
        if (a.gate) f *= sigmoid_f(__ldcg((const float *)a.gate + head));
        float *out = (float *)a.out + head * a.vdim;
        for (int d = lane; d < a.vdim; d += 32) out[d] = (a.maps == 2 ? o1[d] - a.lambda * o2[d] : o1[d]) * f;
    }
}

// ---------------------------------------------------------------- mixture of experts: choice and grouping of M rows
// The `top` largest logits of z[0 .. E) by one warp (lowest index first among equals), into idx / val (lane 0 of the warp
// and everyone else sees them after a __syncwarp).
__device__ __forceinline__ void warp_top(const float *z, int E, int top, int *idx, float *val, int lane) {
    // a candidate is taken strictly after the previous one in (value descending, index ascending) order
    float pv = INFINITY; int pi = -1;
    for (int j = 0; j < top; ++j) {
        float bv = -INFINITY; int bi = 0x7fffffff;
        for (int e = lane; e < E; e += 32) {
            const float v = z[e];
            const bool after = v < pv || (v == pv && e > pi);
            if (after && (v > bv || (v == bv && e < bi))) { bv = v; bi = e; }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, bv, o); const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
        }
        if (bi >= E) { bi = min(pi + 1, E - 1); bv = z[bi]; }      // only with NaN logits: keep the index in range
        if (lane == 0) { idx[j] = bi; val[j] = bv; }
        pv = bv; pi = bi;
    }
    __syncwarp();
}
// softmax over the chosen logits, in place (one warp; val[0] is the largest)
__device__ __forceinline__ void warp_top_softmax(float *val, int top, int lane) {
    const float mx = val[0];
    float s = 0.0f;
    for (int j = lane; j < top; j += 32) s += expf(val[j] - mx);
    s = warp_sum(s);
    __syncwarp();
    for (int j = lane; j < top; j += 32) val[j] = expf(val[j] - mx) / s;
    __syncwarp();
}
struct RouteArgs {
    const float *logits; const void *h; float *weight; int *expert, *rank, *count, *slot, *offsets; void *hp; int rows, E, top, ldl, ld;
};
// each row's experts, weights, and its rank among the rows of that expert (the order inside an expert does not matter: every
// row of a grouped product is computed by itself)
__global__ void __launch_bounds__(128) k_moe_route(const FkState *st, RouteArgs a) {
    __shared__ int idx[4][FKL_MAX_TOP]; __shared__ float val[4][FKL_MAX_TOP];
    pdl_wait(); pdl_launch_dependents();
    const int wid = threadIdx.x >> 5, lane = threadIdx.x & 31, row = blockIdx.x * 4 + wid;
    if (row >= a.rows) return;
    warp_top(a.logits + (size_t)row * a.ldl, a.E, a.top, idx[wid], val[wid], lane);
    warp_top_softmax(val[wid], a.top, lane);
    for (int j = lane; j < a.top; j += 32) {
        const int s = row * a.top + j, e = idx[wid][j];
        a.weight[s] = val[wid][j]; a.expert[s] = e; a.rank[s] = atomicAdd(a.count + e, 1);
    }
}
// rows grouped by expert: slot of every (row, choice), expert offsets, and the copied activations
template <typename T>
__global__ void __launch_bounds__(256) k_moe_gather(const FkState *st, RouteArgs a) {
    __shared__ int off[FKL_MAX_EXPERTS + 1]; __shared__ int wsum[8];
    pdl_wait(); pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, wid = tid >> 5;
    int carry = 0;
    for (int base = 0; base < a.E; base += 256) {       // exclusive scan of the counts
        const int e = base + tid, c = e < a.E ? a.count[e] : 0;
        int v = c;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) { const int t = __shfl_up_sync(0xffffffffu, v, o); if (lane >= o) v += t; }
        if (lane == 31) wsum[wid] = v;
        __syncthreads();
        int before = carry, total = 0;
        for (int w = 0; w < 8; ++w) { if (w < wid) before += wsum[w]; total += wsum[w]; }
        if (e < a.E) off[e] = before + v - c;
        carry += total;
        __syncthreads();
    }
    if (tid == 0) off[a.E] = carry;
    __syncthreads();
    if (blockIdx.x == 0) for (int e = tid; e <= a.E; e += 256) a.offsets[e] = off[e];
    const int s = blockIdx.x, row = s / a.top, dst = off[a.expert[s]] + a.rank[s];
    if (tid == 0) a.slot[s] = dst;
    const uint4 *src = reinterpret_cast<const uint4 *>((const T *)a.h + (size_t)row * a.ld);
    uint4 *d = reinterpret_cast<uint4 *>((T *)a.hp + (size_t)dst * a.ld);
    for (int i = tid; i < a.ld * (int)sizeof(T) / 16; i += 256) d[i] = __ldcg(src + i);
}

// ---------------------------------------------------------------- one row: matrix-vector products over bf16 rows
// A warp owns R = 2 weight rows at a time and streams them in chunks of 256 weights (16 bytes per lane and row), two batches
// of U = 4 chunks in two register buffers: one being multiplied, one in flight.  The activations sit in shared memory as fp32, in the
// order the lanes read them without bank conflicts.  With few rows, 2 .. 16 warps of a block share a row group and split K.
// A chunk is described by (base of row 0, row stride, weights in it), which also expresses the concatenated K ranges of a
// mixture's down projection.  The first batch is fetched before the dependency wait where the rows do not depend on it.
// SEGMENTS: up to three products W_s x_s of n rows each in one launch (outputs one after the other), each with a K range of its own;
// one of the inputs may be a mixer's raw output that is RMS-normed in groups, scaled and gated while it is staged.
#define FKL_GV_R 2
#define FKL_GV_U 4
#define FKL_GV_WARPS 16
enum { FKL_GV_LINEAR = 0, FKL_GV_MOE_UP = 1, FKL_GV_MOE_DOWN = 2, FKL_GV_SEGMENTS = 3 };
struct GvChunk { const uint16_t *base; int stride, len; };
struct GemvArgs {
    // input vector: x, or with norm_w set: x' = x + pscale * sum_p norm(pend_p) * post_w_p + the rest of the pending vectors as they are
    // (+ add) -> x_out, then norm(x') * norm_w (-> h_out); with norm_b a layer norm.  npend vectors of k values, the first nnorm normed.
    const float *x, *pend; const uint16_t *post_w; const float *add; float *x_out; const uint16_t *norm_w; float *h_out;
    const uint16_t *w; float *y; int k, ldk, n, act, act_row0; float eps;
    unsigned long long *amax; uint32_t *counter, *history;             // greedy choice over y (the last block advances the state)
    // mixture of experts
    const float *logits; int *sel; float *wts; const float *sact; const uint16_t *w2; int E, top, ff, ldff, ffs, ldffs;
    int kslices, nchunks;
    const uint16_t *norm_b; int npend, nnorm, act_end, pair0; float pscale, limit, oscale;      // rows from pair0 on: (gate, up) neighbours -> one value
    const float *sx[3]; const uint16_t *sw[3]; int sk[3], sld[3], sc[4], nseg, gseg, group;     // SEGMENTS; sc: first chunk; gseg: the normed input or -1
    const uint16_t *gw; const float *gate;
};
__host__ __device__ inline int gv_chunks(int ldk) { return (ldk + 255) / 256; }
__host__ __device__ inline size_t gv_smem_bytes(int nchunks) { return (size_t)nchunks * (256 * 4 + sizeof(GvChunk)); }
__device__ __forceinline__ int gv_place(int i) { const int j = i & 7; return (i & ~255) + (j >> 2) * 128 + ((i & 255) >> 3) * 4 + (j & 3); }
__device__ __forceinline__ uint4 ldg_stream(const uint16_t *p) {
    uint4 v; asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p)); return v;
}
// NV > 0: the norm prologue keeps NV x 4 values per thread in registers (inputs of up to NV * 2048 values, a multiple of 4): one
// round of loads, the weights' before the dependency wait.  NV = 0: any length, several passes.
template <int MODE, int NV>
__global__ void __launch_bounds__(FKL_GV_WARPS * 32, 1) k_gemv(FkState *st, GemvArgs a) {
    extern __shared__ __align__(16) unsigned char gv_smem[];
    constexpr int R = FKL_GV_R, U = FKL_GV_U, NT = FKL_GV_WARPS * 32;
    float *xs = reinterpret_cast<float *>(gv_smem); GvChunk *tab = reinterpret_cast<GvChunk *>(gv_smem + (size_t)a.nchunks * 1024);
    __shared__ float red[66], part[2][FKL_GV_WARPS][R], tval[FKL_MAX_TOP]; __shared__ int tsel[FKL_MAX_TOP];
    __shared__ unsigned long long wbest[FKL_GV_WARPS]; __shared__ int is_last;
    __shared__ float slog[MODE == FKL_GV_MOE_UP ? FKL_MAX_EXPERTS : MODE == FKL_GV_SEGMENTS ? FKL_GV_MAX_GROUPS : 1];
    const int tid = threadIdx.x, lane = tid & 31, wid = tid >> 5, KS = a.kslices, spb = FKL_GV_WARPS / KS, ksl = wid % KS, slot = wid / KS;
    int c0 = a.nchunks * ksl / KS, c1 = a.nchunks * (ksl + 1) / KS, nb = (c1 - c0 + U - 1) / U;       // of the group being fetched
    const int sgroups = (a.n + R - 1) / R, groups = MODE == FKL_GV_SEGMENTS ? sgroups * a.nseg : sgroups, gstride = gridDim.x * spb;
    int g = blockIdx.x * spb + slot;
    size_t roff[R];                                    // rows of the current fetch group: index into the chunk's rows
    auto set_rows = [&](int gg) {
        if (MODE == FKL_GV_SEGMENTS) {
            const int s = gg / sgroups, nc = a.sc[s + 1] - a.sc[s];
            gg -= s * sgroups;
            c0 = a.sc[s] + nc * ksl / KS; c1 = a.sc[s] + nc * (ksl + 1) / KS; nb = (c1 - c0 + U - 1) / U;
        }
#pragma unroll
        for (int r = 0; r < R; ++r) {
            int row = gg * R + r; row = row < a.n ? row : a.n - 1;
            if (MODE == FKL_GV_MOE_UP) { const int j = row / a.ff; row = tsel[j] * a.ff + (row - j * a.ff); }
            roff[r] = (size_t)row;
        }
    };
    uint4 buf0[U][R], buf1[U][R];
    auto fetch = [&](uint4 (&dst)[U][R], int c) {
#pragma unroll
        for (int u = 0; u < U; ++u) {
            if (c + u < c1) {
                const GvChunk ch = tab[c + u];
#pragma unroll
                for (int r = 0; r < R; ++r) dst[u][r] = lane * 8 < ch.len ? ldg_stream(ch.base + roff[r] * ch.stride + lane * 8) : make_uint4(0, 0, 0, 0);
            } else {
#pragma unroll
                for (int r = 0; r < R; ++r) dst[u][r] = make_uint4(0, 0, 0, 0);
            }
        }
    };
    for (int i = tid; i < a.nchunks * 256; i += NT) xs[i] = 0.0f;
    if (MODE != FKL_GV_MOE_DOWN) {
        if (MODE == FKL_GV_SEGMENTS) {
            for (int s = 0; s < a.nseg; ++s) for (int c = a.sc[s] + tid; c < a.sc[s + 1]; c += NT) {
                const int o = (c - a.sc[s]) * 256;
                tab[c] = GvChunk{a.sw[s] + o, a.sld[s], min(256, a.sld[s] - o)};
            }
        } else for (int c = tid; c < a.nchunks; c += NT) tab[c] = GvChunk{a.w + c * 256, a.ldk, min(256, a.ldk - c * 256)};
        __syncthreads();
        if ((MODE == FKL_GV_LINEAR || MODE == FKL_GV_SEGMENTS) && g < groups && nb > 0) { set_rows(g); fetch(buf0, c0); }
    }
    uint2 pw[NV > 0 ? NV : 1], nw[NV > 0 ? NV : 1];
    const bool block = a.norm_b || a.npend > 1 || a.nnorm < a.npend;       // several pending vectors, or a layer norm
    if (NV > 0 && a.norm_w && !block) {
#pragma unroll
        for (int v = 0; v < NV; ++v) {
            const int i = (v * NT + tid) * 4;
            nw[v] = i < a.k ? __ldg(reinterpret_cast<const uint2 *>(a.norm_w + i)) : make_uint2(0, 0);
            pw[v] = a.pend && i < a.k ? __ldg(reinterpret_cast<const uint2 *>(a.post_w + i)) : make_uint2(0, 0);
        }
    }
    pdl_wait(); pdl_launch_dependents();
    // ---- the input vector
    if (MODE == FKL_GV_MOE_DOWN) {
        const int nce = gv_chunks(a.ldff), nshared = a.nchunks - a.top * nce;
        for (int j = tid; j < a.top; j += NT) { tsel[j] = a.sel[j]; tval[j] = a.wts[j]; }
        __syncthreads();
        for (int c = tid; c < a.nchunks; c += NT) {
            const int j = c / nce, cc = c - j * nce;
            if (j < a.top) tab[c] = GvChunk{a.w + (size_t)tsel[j] * a.n * a.ldff + cc * 256, a.ldff, min(256, a.ldff - cc * 256)};
            else { const int cs = c - a.top * nce; tab[c] = GvChunk{a.w2 + cs * 256, a.ldffs, min(256, a.ldffs - cs * 256)}; }
        }
        (void)nshared;
        __syncthreads();
        if (g < groups && nb > 0) { set_rows(g); fetch(buf0, c0); }
        for (int j = 0; j < a.top; ++j) for (int i = tid; i < a.ff; i += NT) xs[gv_place(j * nce * 256 + i)] = tval[j] * __ldcg(a.x + j * a.ff + i);
        for (int i = tid; i < a.ffs; i += NT) xs[gv_place(a.top * nce * 256 + i)] = __ldcg(a.sact + i);
        __syncthreads();
    } else if (MODE == FKL_GV_MOE_UP) {
        for (int i = tid; i < a.k; i += NT) xs[gv_place(i)] = __ldcg(a.x + i);
        for (int i = tid; i < a.E; i += NT) slog[i] = __ldcg(a.logits + i);
        __syncthreads();
        if (wid == 0) {
            warp_top(slog, a.E, a.top, tsel, tval, lane);
            if (blockIdx.x == 0) {
                warp_top_softmax(tval, a.top, lane);
                for (int j = lane; j < a.top; j += 32) { a.sel[j] = tsel[j]; a.wts[j] = tval[j]; }
            }
        }
        __syncthreads();
        if (g < groups && nb > 0) { set_rows(g); fetch(buf0, c0); }
    } else if (MODE == FKL_GV_SEGMENTS) {
        for (int s = 0; s < a.nseg; ++s) {
            const float *x = a.sx[s]; const int k = a.sk[s], o = a.sc[s] * 256;
            if (s != a.gseg) {
                if ((k & 3) == 0 && ((uintptr_t)x & 15) == 0) {
                    for (int i = tid * 4; i < k; i += NT * 4) *reinterpret_cast<float4 *>(xs + gv_place(o + i)) = __ldcg(reinterpret_cast<const float4 *>(x + i));
                } else for (int i = tid; i < k; i += NT) xs[gv_place(o + i)] = __ldcg(x + i);
                continue;
            }
            const int ng = k / a.group;
            if (ng == 1) {
                float ss = 0.0f;
                for (int i = tid; i < k; i += NT) { const float v = __ldcg(x + i); ss = fmaf(v, v, ss); }
                ss = block_sum(ss, red);
                if (tid == 0) slog[0] = inv_rms(ss, k, a.eps);
            } else for (int q = wid; q < ng; q += FKL_GV_WARPS) {
                float ss = 0.0f;
                for (int i = lane; i < a.group; i += 32) { const float v = __ldcg(x + q * a.group + i); ss = fmaf(v, v, ss); }
                ss = warp_sum(ss);
                if (lane == 0) slog[q] = inv_rms(ss, a.group, a.eps);
            }
            __syncthreads();
            for (int i = tid; i < k; i += NT) xs[gv_place(o + i)] = __ldcg(x + i) * slog[i / a.group] * bf2f(a.gw[i]) * sigmoid_f(__ldcg(a.gate + i));
        }
        __syncthreads();
    } else if (NV > 0 && a.norm_w && block) {
        // everything this needs is requested at once; two normed pending vectors share a reduction
        float4 x[NV > 0 ? NV : 1], y[3][NV > 0 ? NV : 1];
#pragma unroll
        for (int v = 0; v < NV; ++v) {
            const int i = (v * NT + tid) * 4;
            x[v] = i < a.k ? __ldcg(reinterpret_cast<const float4 *>(a.x + i)) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
            for (int p = 0; p < 3; ++p) y[p][v] = p < a.npend && i < a.k ? __ldcg(reinterpret_cast<const float4 *>(a.pend + (size_t)p * a.k + i)) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
        float f[3] = {1.0f, 1.0f, 1.0f};
        if (a.nnorm > 0) {
            float ss[3] = {};
#pragma unroll
            for (int p = 0; p < 3; ++p)
#pragma unroll
                for (int v = 0; v < NV; ++v) ss[p] = fmaf(y[p][v].x, y[p][v].x, fmaf(y[p][v].y, y[p][v].y, fmaf(y[p][v].z, y[p][v].z, fmaf(y[p][v].w, y[p][v].w, ss[p]))));
            const float2 s01 = block_sum2(ss[0], ss[1], red);
            f[0] = a.pscale * inv_rms(s01.x, a.k, a.eps);
            if (a.nnorm > 1) f[1] = a.pscale * inv_rms(s01.y, a.k, a.eps);
            if (a.nnorm > 2) f[2] = a.pscale * inv_rms(block_sum(ss[2], red), a.k, a.eps);
        }
        float sum = 0.0f;
#pragma unroll
        for (int v = 0; v < NV; ++v) {
            const int i = (v * NT + tid) * 4;
#pragma unroll
            for (int p = 0; p < 3; ++p) if (p < a.npend && i < a.k) {
                float4 w = make_float4(1.0f, 1.0f, 1.0f, 1.0f);
                if (p < a.nnorm) { const uint2 q = __ldg(reinterpret_cast<const uint2 *>(a.post_w + (size_t)p * a.k + i)); w = make_float4(bf_lo(q.x), bf_hi(q.x), bf_lo(q.y), bf_hi(q.y)); }
                x[v].x = fmaf(y[p][v].x * f[p], w.x, x[v].x); x[v].y = fmaf(y[p][v].y * f[p], w.y, x[v].y);
                x[v].z = fmaf(y[p][v].z * f[p], w.z, x[v].z); x[v].w = fmaf(y[p][v].w * f[p], w.w, x[v].w);
            }
            sum += (x[v].x + x[v].y) + (x[v].z + x[v].w);
        }
        const float mean = a.norm_b ? block_sum(sum, red) / (float)a.k : 0.0f;
        float ss = 0.0f;
#pragma unroll
        for (int v = 0; v < NV; ++v) if ((v * NT + tid) * 4 < a.k) {
            const float d0 = x[v].x - mean, d1 = x[v].y - mean, d2 = x[v].z - mean, d3 = x[v].w - mean;
            ss = fmaf(d0, d0, fmaf(d1, d1, fmaf(d2, d2, fmaf(d3, d3, ss))));
        }
        const float r = inv_rms(block_sum(ss, red), a.k, a.eps);
#pragma unroll
        for (int v = 0; v < NV; ++v) {
            const int i = (v * NT + tid) * 4;
            if (i >= a.k) continue;
            if (a.x_out && blockIdx.x == 0) *reinterpret_cast<float4 *>(a.x_out + i) = x[v];
            const uint2 w = __ldg(reinterpret_cast<const uint2 *>(a.norm_w + i)), b = a.norm_b ? __ldg(reinterpret_cast<const uint2 *>(a.norm_b + i)) : make_uint2(0, 0);
            const float4 h = make_float4(fmaf((x[v].x - mean) * r, bf_lo(w.x), bf_lo(b.x)), fmaf((x[v].y - mean) * r, bf_hi(w.x), bf_hi(b.x)),
                                         fmaf((x[v].z - mean) * r, bf_lo(w.y), bf_lo(b.y)), fmaf((x[v].w - mean) * r, bf_hi(w.y), bf_hi(b.y)));
            *reinterpret_cast<float4 *>(xs + gv_place(i)) = h;
            if (a.h_out && blockIdx.x == 0) *reinterpret_cast<float4 *>(a.h_out + i) = h;
        }
        __syncthreads();
    } else if (NV > 0 && a.norm_w) {
        float4 x[NV > 0 ? NV : 1], y[NV > 0 ? NV : 1];
#pragma unroll
        for (int v = 0; v < NV; ++v) {
            const int i = (v * NT + tid) * 4;
            x[v] = y[v] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (i < a.k) {
                x[v] = __ldcg(reinterpret_cast<const float4 *>(a.x + i));
                if (a.pend) y[v] = __ldcg(reinterpret_cast<const float4 *>(a.pend + i));
                if (a.add) { const float4 e = __ldcg(reinterpret_cast<const float4 *>(a.add + i)); x[v].x += e.x; x[v].y += e.y; x[v].z += e.z; x[v].w += e.w; }
            }
        }
        if (a.pend) {
            float ss = 0.0f;
#pragma unroll
            for (int v = 0; v < NV; ++v) ss = fmaf(y[v].x, y[v].x, fmaf(y[v].y, y[v].y, fmaf(y[v].z, y[v].z, fmaf(y[v].w, y[v].w, ss))));
            const float ry = inv_rms(block_sum(ss, red), a.k, a.eps);
#pragma unroll
            for (int v = 0; v < NV; ++v) {
                x[v].x = fmaf(y[v].x * ry, bf_lo(pw[v].x), x[v].x); x[v].y = fmaf(y[v].y * ry, bf_hi(pw[v].x), x[v].y);
                x[v].z = fmaf(y[v].z * ry, bf_lo(pw[v].y), x[v].z); x[v].w = fmaf(y[v].w * ry, bf_hi(pw[v].y), x[v].w);
            }
        }
        float ss = 0.0f;
#pragma unroll
        for (int v = 0; v < NV; ++v) ss = fmaf(x[v].x, x[v].x, fmaf(x[v].y, x[v].y, fmaf(x[v].z, x[v].z, fmaf(x[v].w, x[v].w, ss))));
        const float r = inv_rms(block_sum(ss, red), a.k, a.eps);
#pragma unroll
        for (int v = 0; v < NV; ++v) {
            const int i = (v * NT + tid) * 4;
            if (i >= a.k) continue;
            if (a.x_out && blockIdx.x == 0) *reinterpret_cast<float4 *>(a.x_out + i) = x[v];
            const float4 h = make_float4(x[v].x * r * bf_lo(nw[v].x), x[v].y * r * bf_hi(nw[v].x), x[v].z * r * bf_lo(nw[v].y), x[v].w * r * bf_hi(nw[v].y));
            *reinterpret_cast<float4 *>(xs + gv_place(i)) = h;          // four neighbours stay neighbours
            if (a.h_out && blockIdx.x == 0) *reinterpret_cast<float4 *>(a.h_out + i) = h;
        }
        __syncthreads();
    } else if (a.norm_w) {
        __syncthreads();
        float ry[3] = {1.0f, 1.0f, 1.0f};
        for (int p = 0; p < a.nnorm; ++p) {
            float ss = 0.0f;
            for (int i = tid; i < a.k; i += NT) { const float v = __ldcg(a.pend + (size_t)p * a.k + i); ss = fmaf(v, v, ss); }
            ry[p] = a.pscale * inv_rms(block_sum(ss, red), a.k, a.eps);
        }
        float ss = 0.0f, sum = 0.0f, mean = 0.0f;
        for (int i = tid; i < a.k; i += NT) {
            float v = __ldcg(a.x + i);
            for (int p = 0; p < a.npend; ++p) v = fmaf(__ldcg(a.pend + (size_t)p * a.k + i) * ry[p], p < a.nnorm ? bf2f(a.post_w[(size_t)p * a.k + i]) : 1.0f, v);
            if (a.add) v += __ldcg(a.add + i);
            xs[gv_place(i)] = v; ss = fmaf(v, v, ss); sum += v;
            if (a.x_out && blockIdx.x == 0) a.x_out[i] = v;
        }
        if (a.norm_b) {
            mean = block_sum(sum, red) / (float)a.k; ss = 0.0f;
            for (int i = tid; i < a.k; i += NT) { const float v = xs[gv_place(i)] - mean; ss = fmaf(v, v, ss); }
        }
        const float r = inv_rms(block_sum(ss, red), a.k, a.eps);
        for (int i = tid; i < a.k; i += NT) {
            const float v = fmaf((xs[gv_place(i)] - mean) * r, bf2f(a.norm_w[i]), a.norm_b ? bf2f(a.norm_b[i]) : 0.0f);
            xs[gv_place(i)] = v;
            if (a.h_out && blockIdx.x == 0) a.h_out[i] = v;
        }
        __syncthreads();
    } else {
        __syncthreads();
        for (int i = tid; i < a.k; i += NT) xs[gv_place(i)] = __ldcg(a.x + i);
        __syncthreads();
    }
    // ---- rows
    unsigned long long best = 0ull;
    float acc[R] = {};
    int bi = 0, parity = 0, mc0 = c0, mc1 = c1, mnb = nb;          // the group being multiplied
    // one batch: request the next one (of this row group or the following) into the other buffer, multiply this one; after a
    // group's last batch, fold the lanes (and the warps that share the group, behind a barrier of their own) and store
    auto step = [&](uint4 (&cur)[U][R], uint4 (&next)[U][R]) {
        const bool last = bi + 1 == mnb;
        if (!last) fetch(next, mc0 + (bi + 1) * U);
        else if (g + gstride < groups) { set_rows(g + gstride); fetch(next, c0); }
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int c = mc0 + bi * U + u;
            if (c < mc1) {
                const float4 x0 = *reinterpret_cast<const float4 *>(xs + c * 256 + lane * 4), x1 = *reinterpret_cast<const float4 *>(xs + c * 256 + 128 + lane * 4);
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    float f[8]; unpack8f(cur[u][r], f);
                    acc[r] = fmaf(f[0], x0.x, fmaf(f[1], x0.y, fmaf(f[2], x0.z, fmaf(f[3], x0.w, acc[r]))));
                    acc[r] = fmaf(f[4], x1.x, fmaf(f[5], x1.y, fmaf(f[6], x1.z, fmaf(f[7], x1.w, acc[r]))));
                }
            }
        }
        if (!last) { ++bi; return; }
#pragma unroll
        for (int r = 0; r < R; ++r) acc[r] = warp_sum(acc[r]);
        if (KS > 1) {
            if (lane == 0) for (int r = 0; r < R; ++r) part[parity][wid][r] = acc[r];
            asm volatile("bar.sync %0, %1;" ::"r"(1 + slot), "r"(KS * 32) : "memory");
            if (ksl == 0) for (int r = 0; r < R; ++r) for (int q = 1; q < KS; ++q) acc[r] += part[parity][wid + q][r];
            parity ^= 1;                               // the next group writes the other half while this one is still being read
        }
        if (ksl == 0 && MODE == FKL_GV_LINEAR && g * R >= a.pair0) {
            if (lane == 0) a.y[a.pair0 + (g * R - a.pair0) / 2] = clamped_glu(acc[0], acc[1], a.limit);
        } else if (ksl == 0 && MODE == FKL_GV_SEGMENTS) {
            const int s = g / sgroups;
#pragma unroll
            for (int r = 0; r < R; ++r) {
                const int row = (g - s * sgroups) * R + r;
                if (row < a.n && lane == 0) a.y[(size_t)s * a.n + row] = acc[r];
            }
        } else if (ksl == 0) {
#pragma unroll
            for (int r = 0; r < R; ++r) {
                const int row = g * R + r;
                if (row < a.n) {
                    const float v = (row >= a.act_row0 && row < a.act_end ? act_apply(acc[r], a.act) : acc[r]) * (MODE == FKL_GV_LINEAR ? a.oscale : 1.0f);
                    if (lane == 0) a.y[row] = v;
                    if (a.amax) {
                        const uint32_t u = __float_as_uint(v), key = (u & 0x80000000u) ? ~u : u | 0x80000000u;
                        const unsigned long long kk = ((unsigned long long)key << 32) | (unsigned long long)(0xffffffffu - (uint32_t)row);
                        best = kk > best ? kk : best;
                    }
                }
            }
        }
#pragma unroll
        for (int r = 0; r < R; ++r) acc[r] = 0.0f;
        bi = 0; g += gstride; mc0 = c0; mc1 = c1; mnb = nb;
    };
    while (g < groups) {
        step(buf0, buf1);
        if (g >= groups) break;
        step(buf1, buf0);
    }
    if (MODE != FKL_GV_LINEAR || !a.amax) return;
    if (lane == 0) wbest[wid] = best;
    __syncthreads();
    if (tid == 0) {
        for (int i = 1; i < FKL_GV_WARPS; ++i) best = wbest[i] > best ? wbest[i] : best;
        a.amax[blockIdx.x] = best;
        __threadfence();
        is_last = atomicAdd(a.counter, 1u) == gridDim.x - 1;
        if (is_last) *a.counter = 0u;
    }
    __syncthreads();
    if (!is_last || wid != 0) return;
    __threadfence();
    unsigned long long b = 0ull;
    for (int i = lane; i < (int)gridDim.x; i += 32) { const unsigned long long v = __ldcg(a.amax + i); b = v > b ? v : b; }
    b = warp_max_u64(b);
    if (lane == 0) {
        const uint32_t next = 0xffffffffu - (uint32_t)(b & 0xffffffffull);
        st->token[0] = next;
        if (a.history && st->hist_counter < st->hist_cap) a.history[st->hist_counter] = next;
        st->hist_counter += 1; st->offset += 1; st->epoch += 1;
    }
}

// greedy token of one row of fp32 logits, ties to the lowest index; advances the position by `advance` (end of a portion)
__global__ void __launch_bounds__(1024) k_argmax_row_f32(FkState *st, const float *logits, uint32_t *history, int v, int advance) {
    __shared__ unsigned long long wbest[32];
    pdl_wait(); pdl_launch_dependents();
    unsigned long long best = 0ull;
    for (int i = threadIdx.x; i < v; i += blockDim.x) {
        const uint32_t u = __float_as_uint(__ldcg(logits + i)), key = (u & 0x80000000u) ? ~u : u | 0x80000000u;
        const unsigned long long kk = ((unsigned long long)key << 32) | (unsigned long long)(0xffffffffu - (uint32_t)i);
        best = kk > best ? kk : best;
    }
    best = warp_max_u64(best);
    if ((threadIdx.x & 31) == 0) wbest[threadIdx.x >> 5] = best;
    __syncthreads();
    if (threadIdx.x == 0) {
        for (int i = 1; i < (int)(blockDim.x >> 5); ++i) best = wbest[i] > best ? wbest[i] : best;
        const uint32_t next = 0xffffffffu - (uint32_t)(best & 0xffffffffull);
        st->token[0] = next;
        if (history && st->hist_counter < st->hist_cap) history[st->hist_counter] = next;
        st->hist_counter += 1; st->offset += (uint32_t)advance; st->epoch += 1;
    }
}
