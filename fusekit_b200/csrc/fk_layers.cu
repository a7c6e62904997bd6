// Host side of the layered decoders' kernels: argument checks and launches, one case per task kind.
#include "fk_launch.h"
#include "fk_layers.cuh"
#include "fk_gemm_tc.cuh"
#include "fk_flash.cuh"

bool fkl_owns(int kind) { return kind >= FK_TASK_EMBED_ROWS && kind <= FK_TASK_SEGMENT_LINEAR; }
#define FKL_FLASH_MIN_ROWS 8          // up to this many positions one block per (position, kv head) on CUDA cores does better

// CALL with VPL = values per lane of the attention kernel (a power of two covering vpad)
#define VPL_SWITCH(vpad, CALL)                                   \
    do {                                                         \
        if ((vpad) <= 32) { constexpr int VPL = 1; CALL; }       \
        else if ((vpad) <= 64) { constexpr int VPL = 2; CALL; }  \
        else if ((vpad) <= 128) { constexpr int VPL = 4; CALL; } \
        else if ((vpad) <= 256) { constexpr int VPL = 8; CALL; } \
        else { constexpr int VPL = 16; CALL; }                   \
    } while (0)

cudaError_t fkl_init() {
    cudaError_t e = cudaSuccess, r;
#define TRY(x) do { r = (x); if (e == cudaSuccess) e = r; } while (0)
#define ATT(VPL) TRY(big_smem(k_attention<uint16_t, float, VPL, true>)); TRY(big_smem(k_attention<float, float, VPL, true>)); \
                 TRY(big_smem(k_attention<uint16_t, uint16_t, VPL, false>)); TRY(big_smem(k_attention<float, float, VPL, false>))
    ATT(1); ATT(2); ATT(4); ATT(8); ATT(16);
    TRY(big_smem(k_residual_norm_rows<uint16_t>)); TRY(big_smem(k_residual_norm_rows<float>));
    TRY(big_smem(k_gemv<FKL_GV_LINEAR, 0>)); TRY(big_smem(k_gemv<FKL_GV_LINEAR, 1>)); TRY(big_smem(k_gemv<FKL_GV_LINEAR, 2>)); TRY(big_smem(k_gemv<FKL_GV_LINEAR, 4>));
    TRY(big_smem(k_gemv<FKL_GV_SEGMENTS, 0>)); TRY(fkb_init());
    TRY(big_smem(k_gemv<FKL_GV_MOE_UP, 0>)); TRY(big_smem(k_gemv<FKL_GV_MOE_DOWN, 0>)); TRY(big_smem(k_attention_decode));
    TRY(cudaFuncSetAttribute(k_gemm_tc<64, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)TcTile<64>::SMEM)); TRY(cudaFuncSetAttribute(k_gemm_tc<64, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)TcTile<64>::SMEM));
    TRY(cudaFuncSetAttribute(k_gemm_tc<128, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)TcTile<128>::SMEM)); TRY(cudaFuncSetAttribute(k_gemm_tc<128, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)TcTile<128>::SMEM));
    TRY(cudaFuncSetAttribute(k_gemm_tc<256, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)TcTile<256>::SMEM)); TRY(cudaFuncSetAttribute(k_gemm_tc<256, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)TcTile<256>::SMEM));
#define FL(KD, W) TRY(big_smem(k_flash_rows<KD, 64, W>)); TRY(big_smem(k_flash_rows<KD, 128, W>)); TRY(big_smem(k_flash_rows<KD, 256, W>))
    FL(32, false); FL(64, false); FL(128, false); FL(32, true); FL(64, true); FL(128, true);
#undef FL
#undef ATT
#undef TRY
    return e;
}


// Blocks and K split of a matrix-vector product: one block per SM; of the possible splits the one with the shortest critical
// path, row groups of the busiest block x batches of a warp per group (plus a quarter of a batch to finish a group).
static cudaError_t launch_gemv(FklEnv &c, int mode, GemvArgs &a) {
    const int groups = (a.n + FKL_GV_R - 1) / FKL_GV_R, slots = c.sm_count;
    int ks = 1; double best = 1e30;
    // SEGMENTS: the groups of all products, a K range of average length (a split never exceeds the shortest)
    int total = groups, shortest = a.nchunks, average = a.nchunks;
    if (mode == FKL_GV_SEGMENTS) {
        total = groups * a.nseg; average = (a.nchunks + a.nseg - 1) / a.nseg;
        for (int s = 0; s < a.nseg; ++s) if (a.sc[s + 1] - a.sc[s] < shortest) shortest = a.sc[s + 1] - a.sc[s];
    }
    if (!a.act_end) a.act_end = a.n;
    if (!a.pair0) a.pair0 = 0x7fffffff;
    if (a.oscale == 0.0f) a.oscale = 1.0f;
    for (int k = 1; k <= FKL_GV_WARPS && k <= shortest; k *= 2) {
        const int per = FKL_GV_WARPS / k, nblk = (total + per - 1) / per, rounds = (nblk + slots - 1) / slots, chunks = (average + k - 1) / k;
        const double cost = rounds * ((chunks + FKL_GV_U - 1) / FKL_GV_U + 0.25);
        if (cost < best - 1e-9) { best = cost; ks = k; }
    }
    a.kslices = ks;
    const int spb = FKL_GV_WARPS / ks, blocks = (total + spb - 1) / spb, grid = blocks < slots ? blocks : slots;
    const size_t smem = gv_smem_bytes(a.nchunks);
    const dim3 g(grid), b(FKL_GV_WARPS * 32);
    if (mode == FKL_GV_SEGMENTS) return launch(c, k_gemv<FKL_GV_SEGMENTS, 0>, g, b, smem, c.state, a);
    if (mode == FKL_GV_MOE_UP) return launch(c, k_gemv<FKL_GV_MOE_UP, 0>, g, b, smem, c.state, a);
    if (mode == FKL_GV_MOE_DOWN) return launch(c, k_gemv<FKL_GV_MOE_DOWN, 0>, g, b, smem, c.state, a);
    const bool vec = a.norm_w && a.k % 4 == 0 && (((uintptr_t)a.x | (uintptr_t)a.pend | (uintptr_t)a.add | (uintptr_t)a.x_out | (uintptr_t)a.h_out) & 15) == 0;
    const int per = FKL_GV_WARPS * 32 * 4;              // values in one register round of a block
    if (vec && a.k <= per) return launch(c, k_gemv<FKL_GV_LINEAR, 1>, g, b, smem, c.state, a);
    if (vec && a.k <= 2 * per) return launch(c, k_gemv<FKL_GV_LINEAR, 2>, g, b, smem, c.state, a);
    if (vec && a.k <= 4 * per) return launch(c, k_gemv<FKL_GV_LINEAR, 4>, g, b, smem, c.state, a);
    return launch(c, k_gemv<FKL_GV_LINEAR, 0>, g, b, smem, c.state, a);
}
// bf16 rows [rows, k] (row stride ld elements) in boxes of 64 columns x box_rows, 128-byte swizzle
typedef CUresult (*EncodeTiled)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *, const cuuint64_t *, const cuuint32_t *, const cuuint32_t *,
                                CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
static bool tensor_map(CUtensorMap *m, const void *p, long long rows, long long k, long long ld, int box_rows) {
    static EncodeTiled fn = nullptr;
    if (!fn) {
        void *f = nullptr; cudaDriverEntryPointQueryResult qr;
        if (cudaGetDriverEntryPointByVersion("cuTensorMapEncodeTiled", &f, 12000, cudaEnableDefault, &qr) != cudaSuccess || qr != cudaDriverEntryPointSuccess) return false;
        fn = (EncodeTiled)f;
    }
    const cuuint64_t dims[2] = {(cuuint64_t)k, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2] = {FKL_TC_BK, (cuuint32_t)box_rows}, es[2] = {1, 1};
    return fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, (void *)p, dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
              CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}
// the widest tile that still gives (almost) every SM one
static int tc_tile(int sm, long long mtiles, int n) {
    if (mtiles * ((n + 255) / 256) * 10 >= sm * 9) return 256;
    if (mtiles * ((n + 127) / 128) * 10 >= sm * 7) return 128;
    return 64;
}
template <int BN, bool BLOCK> static cudaError_t launch_tc(FklEnv &c, int grid, const CUtensorMap &mx, const CUtensorMap &mw, const TcGemmArgs &a) {
    return launch(c, k_gemm_tc<BN, BLOCK>, dim3(grid), dim3(FKL_TC_THREADS), TcTile<BN>::SMEM, c.state, mx, mw, a);
}
template <int KD, bool WIN> static cudaError_t launch_flash(FklEnv &c, const FlashArgs &a) {
    const dim3 g(a.H, (a.rows + 63) / 64), b(128 * a.maps);
    if (a.vdim <= 64) return launch(c, k_flash_rows<KD, 64, WIN>, g, b, flash_smem_bytes<KD, 64>(a.maps), c.state, a);
    if (a.vdim <= 128) return launch(c, k_flash_rows<KD, 128, WIN>, g, b, flash_smem_bytes<KD, 128>(a.maps), c.state, a);
    return launch(c, k_flash_rows<KD, 256, WIN>, g, b, flash_smem_bytes<KD, 256>(a.maps), c.state, a);
}
template <int KD> static cudaError_t launch_flash(FklEnv &c, const FlashArgs &a) { return a.window > 0 ? launch_flash<KD, true>(c, a) : launch_flash<KD, false>(c, a); }
static bool gv_fits(int nchunks) { return nchunks > 0 && gv_smem_bytes(nchunks) <= 200 * 1024; }

fk_status fkl_run(FklEnv &c, const fk_task &t, char *err, size_t ecap) {
    const uint64_t *b = t.buf; const int32_t *i = t.iarg; const float *f = t.farg;
    cudaError_t e = cudaSuccess;
    FklWeight w, w2;
    switch (t.kind) {
    case FK_TASK_EMBED_ROWS: {
        if ((!b[0] && !b[3]) || !b[1] || i[0] <= 0 || i[1] <= 0 || i[2] <= 0 || (!b[2] && i[1] > FK_MAX_ROWS)) return bad(err, ecap, "embed_rows: bad arguments");
        EmbedRowsArgs a{(const uint16_t *)b[0], (float *)b[1], (const uint32_t *)b[2], i[0], i[2], i[0]};
        if (b[3]) {                                       // the table is a product's weight
            if (!c.weight(c.owner, b[3], &w) || w.n < i[2] || w.k < i[0]) return bad(err, ecap, "embed_rows: table weight missing or too small");
            a.table = w.rows; a.ld = (int)w.k;
        }
        e = launch(c, k_embed_rows, dim3(i[1]), dim3(256), 0, c.state, a);
        break;
    }
    case FK_TASK_RESIDUAL_NORM_ROWS: {
        if (!b[0] || !b[5] || !b[6] || i[0] <= 0 || i[1] <= 0 || i[3] < i[0] || ((b[1] || b[8]) && (!b[2] || i[5] < i[0])) || (b[8] && (!b[9] || !b[10] || i[4] <= 0)))
            return bad(err, ecap, "residual_norm_rows: bad arguments");
        if ((size_t)i[0] * 4 > 200 * 1024) return bad(err, ecap, "residual_norm_rows: width above 51200");
        ResNormArgs a{(const float *)b[0], (const void *)b[1], (const uint16_t *)b[2], (const float *)b[3], (float *)b[4], (const uint16_t *)b[5], (void *)b[6],
                      (const uint32_t *)b[7], (const void *)b[8], (const int *)b[9], (const float *)b[10], i[0], i[3], i[4], i[5], f[0]};
        if (i[0] % 4 == 0 && i[0] <= 8192 && i[3] % 4 == 0 && i[5] % 4 == 0) {
            const dim3 g4(i[1]), b4(i[0] <= 512 ? 128 : 256);
#define RN(T, NV) launch(c, k_residual_norm_rows4<T, NV>, g4, b4, 0, (const FkState *)c.state, a)
            if (i[2]) e = i[0] <= 1024 ? RN(float, 1) : i[0] <= 2048 ? RN(float, 2) : i[0] <= 4096 ? RN(float, 4) : RN(float, 8);
            else e = i[0] <= 1024 ? RN(uint16_t, 1) : i[0] <= 2048 ? RN(uint16_t, 2) : i[0] <= 4096 ? RN(uint16_t, 4) : RN(uint16_t, 8);
#undef RN
            break;
        }
        const dim3 g(i[1]), blk(i[0] >= 2048 ? 512 : 256);
        e = i[2] ? launch(c, k_residual_norm_rows<float>, g, blk, (size_t)i[0] * 4, (const FkState *)c.state, a)
                 : launch(c, k_residual_norm_rows<uint16_t>, g, blk, (size_t)i[0] * 4, (const FkState *)c.state, a);
        break;
    }
    case FK_TASK_LINEAR_ROWS: case FK_TASK_BLOCK_LINEAR_ROWS: {
        const bool block = t.kind == FK_TASK_BLOCK_LINEAR_ROWS;
        if (!c.weight(c.owner, b[1], &w)) return bad(err, ecap, "linear_rows: weight missing or not kept as rows");
        const int M = i[0], row0 = block ? 0 : i[1], N = block ? i[3] : i[2], ldx = block ? (int)w.k : i[3], ldy = i[4], f32 = block ? i[6] : i[5];
        const int act = block ? 0 : i[6] & 255, outf = block ? 0 : (i[6] >> 8) & 1, E = block ? 0 : i[7];
        const int *groups = block ? nullptr : (const int *)b[3];
        BlockCols cols; memset(&cols, 0, sizeof cols);
        if (block) {
            cols = BlockCols{(float *)b[3], (void *)b[4], i[7], i[1], i[2], i[5], f[0]};
            if (cols.silu < 0 || cols.silu > cols.plain || cols.plain < 0 || cols.exact < cols.plain || N < cols.exact || cols.plain % 32 || cols.exact % 32 || (N & 1) || ldy < cols.plain ||
                (cols.exact > cols.plain && !b[3]) || (N > cols.exact && (!b[4] || cols.ld3 < (N - cols.exact) / 2 || cols.ld3 % 8 || (b[4] & 15))) || (b[3] & 15)) return bad(err, ecap, "block_linear_rows: bad columns");
        }
        if (!b[0] || !b[2] || M <= 0 || N <= 0 || row0 < 0 || ldx < w.k || ldx % 8 || (!block && ldy < N) || (groups && E <= 0)) return bad(err, ecap, "linear_rows: bad arguments");
        if (groups ? w.n != (long long)E * N : row0 + N > w.n) return bad(err, ecap, "linear_rows: shape mismatch");
        const float scale = block || f[0] == 0.0f ? 1.0f : f[0];
        if (!f32) {           // tensor cores
            if (ldx % 64 || (b[0] & 15) || (block && ((b[2] & 15) || ldy % 8))) return bad(err, ecap, "linear_rows: bf16 rows need a stride in multiples of 64 and 16-byte alignment");
            TcGemmArgs a{(void *)b[2], groups, M, N, (int)(w.k / FKL_TC_BK), row0, ldy, act, outf, E, scale, cols};
            const long long mt = groups ? (M < E ? M : E) + M / 128 : (M + 127) / 128;
            const int bn = tc_tile(c.sm_count, mt, N);
            const long long tiles = mt * ((N + bn - 1) / bn);
            const int grid = tiles < c.sm_count ? (int)tiles : c.sm_count;
            CUtensorMap mx, mw;
            if (!tensor_map(&mx, (const void *)b[0], M, w.k, ldx, 128) || !tensor_map(&mw, w.rows, w.n, w.k, w.k, bn)) return bad(err, ecap, "linear_rows: tensor map refused");
            if (block) e = bn == 256 ? launch_tc<256, true>(c, grid, mx, mw, a) : bn == 128 ? launch_tc<128, true>(c, grid, mx, mw, a) : launch_tc<64, true>(c, grid, mx, mw, a);
            else e = bn == 256 ? launch_tc<256, false>(c, grid, mx, mw, a) : bn == 128 ? launch_tc<128, false>(c, grid, mx, mw, a) : launch_tc<64, false>(c, grid, mx, mw, a);
            break;
        }
        LinRowsArgs a{(const float *)b[0], w.rows + (size_t)row0 * w.k, (float *)b[2], groups, M, N, (int)w.k, ldx, (int)w.k, ldy, act, scale, cols};
        const dim3 g((N + 63) / 64, (M + 63) / 64, groups ? E : 1);
        if (g.y > 65535 || g.z > 65535) return bad(err, ecap, "linear_rows: too many rows");
        e = block ? launch(c, k_linear_rows<true>, g, dim3(256), 0, (const FkState *)c.state, a) : launch(c, k_linear_rows<false>, g, dim3(256), 0, (const FkState *)c.state, a);
        break;
    }
    case FK_TASK_QK_NORM_STORE_ROWS: {
        QkStoreArgs a{(const void *)b[0], (const uint16_t *)b[1], (const uint16_t *)b[2], (void *)b[3], (void *)b[4], (void *)b[5],
                      i[0], i[1], i[6] >> 8, i[2], i[3], round_up(i[2], 8), round_up(i[3], 8), i[4], i[5], i[7], f[0]};
        for (int q = 0; q < 6; ++q) if (!b[q]) return bad(err, ecap, "qk_norm_store_rows: missing buffer %d", q);
        if (a.H <= 0 || a.G <= 0 || a.H % a.G || a.dim <= 0 || a.vdim <= 0 || a.cap <= 0 || a.rows <= 0 || (a.maps != 1 && a.maps != 2) ||
            a.ld < (a.H + a.G) * a.maps * a.dim + a.G * a.vdim) return bad(err, ecap, "qk_norm_store_rows: bad arguments");
        const dim3 g(a.rows, ((a.H + a.G) * a.maps + a.G + 3) / 4);
        e = (i[6] & 1) ? launch(c, k_qk_norm_store_rows<float>, g, dim3(128), 0, c.state, a) : launch(c, k_qk_norm_store_rows<uint16_t>, g, dim3(128), 0, c.state, a);
        break;
    }
    case FK_TASK_ATTENTION_ROWS: case FK_TASK_ATTENTION_DECODE: case FK_TASK_WINDOW_ATTENTION_ROWS: case FK_TASK_WINDOW_ATTENTION_DECODE: {
        const bool win = t.kind == FK_TASK_WINDOW_ATTENTION_ROWS || t.kind == FK_TASK_WINDOW_ATTENTION_DECODE;
        const bool dec = t.kind == FK_TASK_ATTENTION_DECODE || t.kind == FK_TASK_WINDOW_ATTENTION_DECODE;
        AttnArgs a; memset(&a, 0, sizeof a);
        int f32, rows = 1;
        a.scale = f[0];
        if (win) {            // heads and sizes two to a word; all queries normed together, rotation, window
            a.H = i[0] & 0xffff; a.G = i[0] >> 16; a.dim = i[1] & 0xffff; a.vdim = i[1] >> 16; a.cap = i[2]; a.maps = 1;
            f32 = dec ? i[3] : i[4]; a.eps = f[1];
            a.window = i[5]; a.keep = i[6];
            if (dec) { a.splits = i[4]; a.rot = (const float *)b[8]; a.rot_dims = i[7]; a.joint = 1; } else rows = i[3];
            if (a.window < 0 || a.keep < 0 || a.rot_dims < 0 || a.rot_dims > a.dim || (a.rot_dims & 1) || (a.rot_dims && !a.rot)) return bad(err, ecap, "attention: bad window or rotation");
            if (!a.rot_dims) a.rot = nullptr;
        } else {
            a.H = i[0]; a.G = i[1]; a.dim = i[2]; a.vdim = i[3]; a.cap = i[4]; a.maps = i[6] >> 8; f32 = i[6] & 1;
            a.lambda = f[1]; a.diff = f[2]; a.eps = f[3];
            if (dec) a.splits = i[7]; else rows = i[5];
        }
        if (a.H <= 0 || a.G <= 0 || a.H % a.G || a.dim <= 0 || a.vdim <= 0 || a.vdim > 512 || a.cap <= 0 || rows <= 0 || rows > 65535 || (a.maps != 1 && a.maps != 2))
            return bad(err, ecap, "attention: bad arguments (value size up to 512)");
        a.dpad = round_up(a.dim, 8); a.vpad = round_up(a.vdim, 8);
        a.tiles = (a.H / a.G * a.maps + FKL_ATT_ROWS - 1) / FKL_ATT_ROWS;
        const size_t smem = attn_smem_floats(a.dpad, a.vpad) * 4;
        if (smem > 220 * 1024) return bad(err, ecap, "attention: head size too large");
        if (dec) {
            for (int q = 0; q < 8; ++q) if (!b[q]) return bad(err, ecap, "attention_decode: missing buffer %d", q);
            a.qkv = (const float *)b[0]; a.qn = (const uint16_t *)b[1]; a.kn = (const uint16_t *)b[2]; a.ck = (void *)b[3]; a.cv = (void *)b[4]; a.out = (void *)b[5];
            a.part = (float *)b[6]; a.counter = (uint32_t *)b[7];
            a.gate = !win && i[5] ? (const void *)(a.qkv + (a.H + a.G) * a.maps * a.dim + a.G * a.vdim) : nullptr;
            if (a.splits <= 0 || a.splits > 8 * a.vpad || a.splits > 256) return bad(err, ecap, "attention_decode: bad number of key splits");
            const dim3 g(a.splits, a.G * a.tiles, 1), blk(FKL_ATT_WARPS * 32);
            const int ad = ad_layout(a.maps, a.dpad, a.vpad).total;
            if (!f32 && ad <= 200 * 1024) { e = launch(c, k_attention_decode, g, dim3(FKL_AD_THREADS), (size_t)ad, c.state, a); break; }
            if (f32) VPL_SWITCH(a.vpad, e = launch(c, (k_attention<float, float, VPL, true>), g, blk, smem, c.state, a));
            else VPL_SWITCH(a.vpad, e = launch(c, (k_attention<uint16_t, float, VPL, true>), g, blk, smem, c.state, a));
        } else {
            for (int q = 0; q < 4; ++q) if (!b[q]) return bad(err, ecap, "attention_rows: missing buffer %d", q);
            a.splits = 1;
            a.q = (const void *)b[0]; a.ck = (void *)b[1]; a.cv = (void *)b[2]; a.out = (void *)b[3]; a.gate = win ? nullptr : (const void *)b[4];
            a.ldo = round_up(a.H * a.vdim, 64); a.ldg = win ? 0 : i[7];
            if (!f32 && rows > FKL_FLASH_MIN_ROWS && a.dim <= 128 && a.vdim <= 256) {
                FlashArgs fa{(const uint16_t *)a.q, (const uint16_t *)a.ck, (const uint16_t *)a.cv, (const uint16_t *)a.gate, (uint16_t *)a.out, a.H, a.G, a.maps, a.vdim,
                             a.dpad, a.vpad, a.cap, a.ldo, a.ldg, rows, a.scale, a.lambda, a.diff, a.eps, a.window, a.keep};
                e = a.dim <= 32 ? launch_flash<32>(c, fa) : a.dim <= 64 ? launch_flash<64>(c, fa) : launch_flash<128>(c, fa);
                break;
            }
            const dim3 g(1, a.G * a.tiles, rows), blk(FKL_ATT_WARPS * 32);
            if (f32) VPL_SWITCH(a.vpad, e = launch(c, (k_attention<float, float, VPL, false>), g, blk, smem, c.state, a));
            else VPL_SWITCH(a.vpad, e = launch(c, (k_attention<uint16_t, uint16_t, VPL, false>), g, blk, smem, c.state, a));
        }
        break;
    }
    case FK_TASK_MOE_ROUTE_ROWS: {
        RouteArgs a; memset(&a, 0, sizeof a);
        for (int q = 0; q < 9; ++q) if (!b[q]) return bad(err, ecap, "moe_route_rows: missing buffer %d", q);
        a.logits = (const float *)b[0]; a.h = (const void *)b[1]; a.weight = (float *)b[2]; a.expert = (int *)b[3]; a.rank = (int *)b[4]; a.count = (int *)b[5];
        a.slot = (int *)b[6]; a.offsets = (int *)b[7]; a.hp = (void *)b[8];
        a.rows = i[0]; a.E = i[1]; a.top = i[2]; a.ldl = i[3]; a.ld = i[4];
        if (a.rows <= 0 || a.E <= 0 || a.E > FKL_MAX_EXPERTS || a.top <= 0 || a.top > FKL_MAX_TOP || a.top > a.E || a.ldl < a.E || a.ld <= 0 || a.ld % 8)
            return bad(err, ecap, "moe_route_rows: bad arguments (at most %d experts, %d chosen)", FKL_MAX_EXPERTS, FKL_MAX_TOP);
        e = cudaMemsetAsync(a.count, 0, (size_t)a.E * 4, c.stream);
        if (e == cudaSuccess) e = launch(c, k_moe_route, dim3((a.rows + 3) / 4), dim3(128), 0, (const FkState *)c.state, a);
        if (e == cudaSuccess) e = i[5] ? launch(c, k_moe_gather<float>, dim3(a.rows * a.top), dim3(256), 0, (const FkState *)c.state, a)
                                       : launch(c, k_moe_gather<uint16_t>, dim3(a.rows * a.top), dim3(256), 0, (const FkState *)c.state, a);
        break;
    }
    case FK_TASK_NORM_LINEAR: {
        if (!c.weight(c.owner, b[6], &w)) return bad(err, ecap, "norm_linear: weight missing or not kept as rows");
        GemvArgs a; memset(&a, 0, sizeof a);
        a.x = (const float *)b[0]; a.pend = (const float *)b[1]; a.post_w = (const uint16_t *)b[2]; a.add = (const float *)b[3]; a.x_out = (float *)b[4];
        a.norm_w = (const uint16_t *)b[5]; a.y = (float *)b[7]; a.h_out = (float *)b[8]; a.amax = (unsigned long long *)b[9]; a.counter = (uint32_t *)b[10];
        a.w = w.rows; a.k = i[0]; a.n = i[1]; a.act = i[2]; a.act_row0 = i[3]; a.ldk = (int)w.k; a.eps = f[0]; a.history = c.history;
        a.npend = a.nnorm = a.pend ? 1 : 0; a.pscale = 1.0f;
        if (i[4] > 0) { a.npend = i[4]; a.nnorm = i[5]; a.pscale = f[1]; }
        a.norm_b = (const uint16_t *)b[11]; a.pair0 = i[6]; a.act_end = i[7]; a.limit = f[2]; a.oscale = f[3];
        if (a.npend > 3 || a.nnorm < 0 || a.nnorm > a.npend || (a.npend && !a.pend) || a.pair0 < 0 || a.pair0 % 2 || a.act_end < 0 || (a.norm_b && !a.norm_w) ||
            (a.pair0 && a.amax)) return bad(err, ecap, "norm_linear: bad pending vectors or row ranges");
        if (!a.x || !a.y || a.k <= 0 || a.k > w.k || a.n <= 0 || a.n > w.n || (a.pend && ((a.nnorm && !a.post_w) || !a.norm_w)) || (a.amax && !a.counter) ||
            (a.x_out && a.x_out == a.x)) return bad(err, ecap, "norm_linear: bad arguments");
        a.nchunks = gv_chunks(a.ldk);
        if (!gv_fits(a.nchunks)) return bad(err, ecap, "norm_linear: input of %d values is too long", a.k);
        e = launch_gemv(c, FKL_GV_LINEAR, a);
        break;
    }
    case FK_TASK_SEGMENT_LINEAR: {
        GemvArgs a; memset(&a, 0, sizeof a);
        a.n = i[0]; a.nseg = i[1]; a.gseg = i[5]; a.group = i[6]; a.y = (float *)b[6]; a.gw = (const uint16_t *)b[7]; a.gate = (const float *)b[8]; a.eps = f[0];
        if (a.n <= 0 || a.nseg < 1 || a.nseg > 3 || !a.y || a.gseg >= a.nseg) return bad(err, ecap, "segment_linear: bad arguments");
        for (int s = 0; s < a.nseg; ++s) {
            if (!c.weight(c.owner, b[2 * s + 1], &w) || !b[2 * s] || i[2 + s] <= 0 || i[2 + s] > w.k || w.n != a.n) return bad(err, ecap, "segment_linear: product %d: weight missing or of another shape", s);
            a.sx[s] = (const float *)b[2 * s]; a.sw[s] = w.rows; a.sk[s] = i[2 + s]; a.sld[s] = (int)w.k; a.sc[s + 1] = a.sc[s] + gv_chunks((int)w.k);
        }
        if (a.gseg >= 0 && (!a.gw || !a.gate || a.group <= 0 || a.sk[a.gseg] % a.group || a.sk[a.gseg] / a.group > FKL_GV_MAX_GROUPS)) return bad(err, ecap, "segment_linear: bad norm groups");
        a.nchunks = a.sc[a.nseg];
        if (!gv_fits(a.nchunks)) return bad(err, ecap, "segment_linear: the inputs do not fit in shared memory");
        e = launch_gemv(c, FKL_GV_SEGMENTS, a);
        break;
    }
    case FK_TASK_MOE_UP: {
        if (!c.weight(c.owner, b[2], &w)) return bad(err, ecap, "moe_up: weight missing or not kept as rows");
        GemvArgs a; memset(&a, 0, sizeof a);
        a.logits = (const float *)b[0]; a.x = (const float *)b[1]; a.w = w.rows; a.y = (float *)b[3]; a.sel = (int *)b[4]; a.wts = (float *)b[5];
        a.k = i[0]; a.E = i[1]; a.top = i[2]; a.ff = i[3]; a.act = i[4]; a.ldk = (int)w.k; a.n = a.top * a.ff;
        if (!a.logits || !a.x || !a.y || !a.sel || !a.wts || a.k <= 0 || a.k > w.k || a.E <= 0 || a.E > FKL_MAX_EXPERTS || a.top <= 0 || a.top > FKL_MAX_TOP || a.top > a.E ||
            a.ff <= 0 || w.n != (long long)a.E * a.ff) return bad(err, ecap, "moe_up: bad arguments");
        a.nchunks = gv_chunks(a.ldk);
        if (!gv_fits(a.nchunks)) return bad(err, ecap, "moe_up: input of %d values is too long", a.k);
        e = launch_gemv(c, FKL_GV_MOE_UP, a);
        break;
    }
    case FK_TASK_MOE_DOWN: {
        if (!c.weight(c.owner, b[3], &w)) return bad(err, ecap, "moe_down: weight missing or not kept as rows");
        GemvArgs a; memset(&a, 0, sizeof a);
        a.x = (const float *)b[0]; a.sel = (int *)b[1]; a.wts = (float *)b[2]; a.w = w.rows; a.sact = (const float *)b[4]; a.y = (float *)b[6];
        a.n = i[0]; a.E = i[1]; a.top = i[2]; a.ff = i[3]; a.ffs = i[4]; a.ldff = (int)w.k;
        if (!a.x || !a.sel || !a.wts || !a.y || a.n <= 0 || a.E <= 0 || a.top <= 0 || a.top > FKL_MAX_TOP || a.ff <= 0 || a.ff > a.ldff || w.n != (long long)a.E * a.n)
            return bad(err, ecap, "moe_down: bad arguments");
        a.nchunks = a.top * gv_chunks(a.ldff);
        if (a.ffs > 0) {
            if (!c.weight(c.owner, b[5], &w2) || w2.n != a.n || w2.k < a.ffs || !a.sact) return bad(err, ecap, "moe_down: shared weight missing or of another shape");
            a.w2 = w2.rows; a.ldffs = (int)w2.k; a.nchunks += gv_chunks(a.ldffs);
        }
        if (!gv_fits(a.nchunks)) return bad(err, ecap, "moe_down: the chosen experts' activations do not fit in shared memory");
        e = launch_gemv(c, FKL_GV_MOE_DOWN, a);
        break;
    }
    case FK_TASK_ARGMAX_ROW: {
        if (!b[0] || i[0] <= 0 || i[1] < 0) return bad(err, ecap, "argmax_row: bad arguments");
        e = launch(c, k_argmax_row_f32, dim3(1), dim3(1024), 0, c.state, (const float *)b[0], c.history, i[0], i[1]);
        break;
    }
    default: return fkb_run(c, t, err, ecap);
    }
    if (e != cudaSuccess) { snprintf(err, ecap, "launch of task kind %d failed: %s", t.kind, cudaGetErrorString(e)); return FK_ERR_CUDA; }
    return FK_OK;
}
