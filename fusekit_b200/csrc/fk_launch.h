// Launch and error helpers of the layered decoders' host files.
#pragma once
#include "fk_layers.h"
#include <stdarg.h>
#include <stdio.h>
#include <string.h>

template <typename K> inline cudaError_t big_smem(K kern) {
    cudaFuncAttributes fa; cudaError_t e = cudaFuncGetAttributes(&fa, kern);
    if (e != cudaSuccess) return e;
    return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024 - (int)fa.sharedSizeBytes);
}
template <typename... KA, typename... A>
inline cudaError_t launch(FklEnv &c, void (*kern)(KA...), dim3 grid, dim3 block, size_t smem, A... args) {
    cudaLaunchConfig_t cfg; memset(&cfg, 0, sizeof cfg);
    cfg.gridDim = grid; cfg.blockDim = block; cfg.dynamicSmemBytes = smem; cfg.stream = c.stream;
    cudaLaunchAttribute at[1];
    at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = at; cfg.numAttrs = c.pdl ? 1 : 0;
    ++*c.launches;
    return cudaLaunchKernelEx(&cfg, kern, KA(args)...);
}
inline fk_status bad(char *err, size_t cap, const char *fmt, ...) {
    va_list ap; va_start(ap, fmt); vsnprintf(err, cap, fmt, ap); va_end(ap);
    return FK_ERR_VALUE;
}
inline int round_up(int v, int m) { return (v + m - 1) / m * m; }
