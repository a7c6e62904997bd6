// Boundary between the host runtime (fk_runtime.cu) and the kernels of the layered decoders (fk_layers.cu; fk_blocks.cu for those of the
// parallel blocks), which are translation units of their own so that all compile side by side.
#pragma once
#include "../../include/fusekit_cuda.h"
#include "fk_common.cuh"

struct FklWeight { const uint16_t *rows; long long n, k; };       // bf16 rows [n, k] as uploaded (fk_weight_keep_rows)
struct FklEnv {
    cudaStream_t stream; bool pdl; int sm_count;
    FkState *state; uint32_t *history; long long *launches;
    void *owner; bool (*weight)(void *owner, uint64_t id, FklWeight *out);      // false: no such weight, or not frozen as rows
};
bool fkl_owns(int kind);                                           // whether a task kind is handled here
fk_status fkl_run(FklEnv &env, const fk_task &t, char *err, size_t cap);
cudaError_t fkl_init();                                            // shared-memory limits of the kernels, once per context
fk_status fkb_run(FklEnv &env, const fk_task &t, char *err, size_t cap);      // the kinds of fk_blocks.cu
cudaError_t fkb_init();
