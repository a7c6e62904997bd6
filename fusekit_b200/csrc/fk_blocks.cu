// Host side of the parallel blocks' kernels: argument checks and launches.
#include "fk_launch.h"
#include "fk_blocks.cuh"

#define FKB_CHUNK_MIN_ROWS 16         // below, position by position does better
#define FKB_MAX_SEGMENTS 16

template <int KD> static cudaError_t chunk_init() {
    cudaError_t e = cudaSuccess, r;
#define TRY(x) do { r = (x); if (e == cudaSuccess) e = r; } while (0)
    TRY(big_smem(k_recurrence_chunks<KD, false, false>)); TRY(big_smem(k_recurrence_chunks<KD, false, true>));
    TRY(big_smem(k_recurrence_chunks<KD, true, false>)); TRY(big_smem(k_recurrence_chunks<KD, true, true>));
    return e;
}
cudaError_t fkb_init() {
    cudaError_t e = cudaSuccess, r;
    TRY(chunk_init<32>()); TRY(chunk_init<64>()); TRY(chunk_init<128>()); TRY(chunk_init<256>());
    TRY(big_smem(k_block_norm_rows<uint16_t>)); TRY(big_smem(k_block_norm_rows<float>));
#undef TRY
    return e;
}
template <typename T, bool MEM> static cudaError_t launch_recurrence(FklEnv &c, const RecArgs &a) {
    const dim3 g((a.vdim + FKL_RC_COLS - 1) / FKL_RC_COLS, a.heads), b(FKL_RC_THREADS);
#define RC(RPT) launch(c, (k_recurrence<T, MEM, RPT>), g, b, 0, c.state, a)
    return a.dim <= 32 ? RC(4) : a.dim <= 64 ? RC(8) : a.dim <= 128 ? RC(16) : a.dim <= 256 ? RC(32) : RC(64);
#undef RC
}
template <int KD, bool MEM> static cudaError_t launch_chunks(FklEnv &c, const RecArgs &a) {
    dim3 g((a.vdim + FKL_RC_COLS - 1) / FKL_RC_COLS, a.heads, a.segments);
    const size_t smem = ChunkSmem<KD>::TOTAL;
    if (a.segments > 1) {
        dim3 first = g; first.z = a.segments - 1;        // what the last run leaves comes out of the second pass
        cudaError_t e = launch(c, (k_recurrence_chunks<KD, MEM, false>), first, dim3(FKL_CH_THREADS), smem, c.state, a);
        if (e != cudaSuccess) return e;
    }
    return launch(c, (k_recurrence_chunks<KD, MEM, true>), g, dim3(FKL_CH_THREADS), smem, c.state, a);
}
template <bool MEM> static cudaError_t chunks_by_size(FklEnv &c, const RecArgs &a) {
    return a.dim <= 32 ? launch_chunks<32, MEM>(c, a) : a.dim <= 64 ? launch_chunks<64, MEM>(c, a) : a.dim <= 128 ? launch_chunks<128, MEM>(c, a) : launch_chunks<256, MEM>(c, a);
}

fk_status fkb_run(FklEnv &c, const fk_task &t, char *err, size_t ecap) {
    const uint64_t *b = t.buf; const int32_t *i = t.iarg; const float *f = t.farg;
    cudaError_t e = cudaSuccess;
    const FkState *st = c.state;
    switch (t.kind) {
    case FK_TASK_BLOCK_NORM_ROWS: {
        BlockNormArgs a{(const float *)b[0], {(const void *)b[1], (const void *)b[2], (const void *)b[3]}, (const uint16_t *)b[9], (float *)b[4], (const uint16_t *)b[5], (const uint16_t *)b[8],
                        (void *)b[6], (const uint32_t *)b[7], i[0], i[3], i[4], i[5], i[6], f[0], f[1]};
        if (!a.x || !a.w || !a.h || a.d <= 0 || i[1] <= 0 || a.ldh < a.d || a.np < 0 || a.np > 3 || a.nnorm < 0 || a.nnorm > a.np || (a.nnorm && !a.post) || (a.np && a.ldy < a.d))
            return bad(err, ecap, "block_norm_rows: bad arguments");
        for (int p = 0; p < a.np; ++p) if (!a.y[p]) return bad(err, ecap, "block_norm_rows: missing pending rows %d", p);
        if ((size_t)a.d * 4 > 200 * 1024) return bad(err, ecap, "block_norm_rows: width above 51200");
        const dim3 g(i[1]);
        if (a.d % 4 == 0 && a.d <= 8192 && a.ldh % 4 == 0 && a.ldy % 4 == 0) {
            // one round of four values per thread up to 2048, two above; as many threads as that takes
            const int nv = a.d <= 2048 ? 1 : 2;
            const dim3 blk(round_up((a.d / 4 + nv - 1) / nv, 32));
#define BN(T, NV, NT, BLOCKS) launch(c, (k_block_norm_rows4<T, NV, NT, BLOCKS>), g, blk, 0, st, a)
            if (i[2]) e = a.d <= 2048 ? BN(float, 1, 512, 2) : a.d <= 4096 ? BN(float, 2, 512, 1) : BN(float, 2, 1024, 1);
            else e = a.d <= 2048 ? BN(uint16_t, 1, 512, 3) : a.d <= 4096 ? BN(uint16_t, 2, 512, 2) : a.d <= 5120 ? BN(uint16_t, 2, 640, 2) : BN(uint16_t, 2, 1024, 1);
#undef BN
            break;
        }
        e = i[2] ? launch(c, k_block_norm_rows<float>, g, dim3(256), (size_t)a.d * 4, st, a) : launch(c, k_block_norm_rows<uint16_t>, g, dim3(256), (size_t)a.d * 4, st, a);
        break;
    }
    case FK_TASK_ROTARY_STORE_ROWS: {
        RotaryStoreArgs a{(const void *)b[0], (const uint16_t *)b[1], (const uint16_t *)b[2], (void *)b[3], (void *)b[4], (void *)b[5], (const float *)b[6], i[0] & 0xffff, i[0] >> 16,
                          i[1] & 0xffff, i[1] >> 16, round_up(i[1] & 0xffff, 8), round_up(i[1] >> 16, 8), i[2], i[4], i[5], f[0]};
        for (int q = 0; q < 6; ++q) if (!b[q]) return bad(err, ecap, "rotary_store_rows: missing buffer %d", q);
        if (a.H <= 0 || a.G <= 0 || a.H % a.G || a.dim <= 0 || a.vdim <= 0 || a.cap <= 0 || i[3] <= 0 || a.ld < (a.H + a.G) * a.dim + a.G * a.vdim || a.rot_dims < 0 || a.rot_dims > a.dim ||
            (a.rot_dims & 1) || (a.rot_dims && !a.rot)) return bad(err, ecap, "rotary_store_rows: bad arguments");
        if (!a.rot_dims) a.rot = nullptr;
        e = i[6] ? launch(c, k_rotary_store_rows<float>, dim3(i[3]), dim3(256), 0, c.state, a) : launch(c, k_rotary_store_rows<uint16_t>, dim3(i[3]), dim3(256), 0, c.state, a);
        break;
    }
    case FK_TASK_NORM_GATE_ROWS: {
        NormGateArgs a{(const void *)b[0], (const uint16_t *)b[1], (const void *)b[2], (void *)b[3], i[0], i[1], i[3], i[4], i[5], f[0]};
        if (!a.o || !a.w || !a.gate || !a.out || a.n <= 0 || a.group <= 0 || a.n % a.group || a.n / a.group > FKL_GV_MAX_GROUPS || i[2] <= 0 || a.ldo < a.n || a.ldg < a.n || a.ld < a.n)
            return bad(err, ecap, "norm_gate_rows: bad arguments");
        e = i[6] ? launch(c, k_norm_gate_rows<float>, dim3(i[2]), dim3(256), 0, st, a) : launch(c, k_norm_gate_rows<uint16_t>, dim3(i[2]), dim3(256), 0, st, a);
        break;
    }
    case FK_TASK_RECURRENCE_ROWS: case FK_TASK_RECURRENCE_DECODE: {
        const bool dec = t.kind == FK_TASK_RECURRENCE_DECODE, mem = !b[5], f32 = dec || (i[0] >> 16);
        RecArgs a; memset(&a, 0, sizeof a);
        a.q = (const void *)b[0]; a.k = (const void *)b[1]; a.v = (const void *)b[2]; a.logits = (const float *)b[3]; a.bias = (const uint16_t *)b[4]; a.log_decay = (const float *)b[5];
        a.state = (float *)b[6]; a.out = (void *)b[7];
        a.heads = i[0] & 0xffff; a.dim = i[1]; a.vdim = i[2]; a.rows = dec ? 1 : i[3]; a.ld = i[4]; a.ldl = i[5]; a.ldo = i[6]; a.qscale = f[0]; a.cap = f[1];
        if (!a.q || !a.k || !a.v || !a.state || !a.out || a.heads <= 0 || a.dim <= 0 || a.dim > 512 || a.vdim <= 0 || a.rows <= 0 || (mem && (!a.logits || !a.bias || !(a.cap > 0.0f))) ||
            (!dec && (a.ld < a.heads * (a.dim > a.vdim ? a.dim : a.vdim) || a.ldo < a.heads * a.vdim || (mem && a.ldl < 2 * a.heads)))) return bad(err, ecap, "recurrence: bad arguments (key size up to 512)");
        a.sstride = rec_state_stride(a.dim, mem);
        const bool aligned = ((b[0] | b[1] | b[2]) & 15) == 0 && a.ld % 8 == 0 && a.dim % 8 == 0 && a.vdim % 8 == 0 && (b[7] & 3) == 0 && a.ldo % 2 == 0;
        if (!f32 && a.rows >= FKB_CHUNK_MIN_ROWS && a.dim <= 256 && aligned) {
            // runs of chunks side by side: as many as it takes to fill every SM, at least four chunks each
            const int chunks = (a.rows + FKL_CH - 1) / FKL_CH, cells = a.heads * ((a.vdim + FKL_RC_COLS - 1) / FKL_RC_COLS);
            int runs = b[8] ? (a.dim <= 128 ? 2 : 1) * c.sm_count / cells : 1;
            if (runs > chunks / 4) runs = chunks / 4;
            if (runs > FKB_MAX_SEGMENTS) runs = FKB_MAX_SEGMENTS;
            while (runs > 1 && (long long)(runs + 1) * cells * a.sstride + (long long)runs * cells > i[7]) --runs;
            if (runs < 1) runs = 1;
            a.per = (chunks + runs - 1) / runs; a.segments = (chunks + a.per - 1) / a.per; a.seg = (float *)b[8];
            e = mem ? chunks_by_size<true>(c, a) : chunks_by_size<false>(c, a);
            break;
        }
        if (f32) e = mem ? launch_recurrence<float, true>(c, a) : launch_recurrence<float, false>(c, a);
        else e = mem ? launch_recurrence<uint16_t, true>(c, a) : launch_recurrence<uint16_t, false>(c, a);
        break;
    }
    default: return bad(err, ecap, "unknown task kind %d", t.kind);
    }
    if (e != cudaSuccess) { snprintf(err, ecap, "launch of task kind %d failed: %s", t.kind, cudaGetErrorString(e)); return FK_ERR_CUDA; }
    return FK_OK;
}
