// Kernel launch helper: every kernel of a decoder step is launched with the
// programmatic-stream-serialization attribute so that its prologue (weight
// prefetch) overlaps the tail of the previous kernel.
#pragma once
#include "dc_internal.h"

// The same for a kernel whose CTAs form clusters of `cluster` neighbours.
template <typename... KArgs, typename... Args>
static inline int dc_launch_cluster(dc_ctx* ctx, const char* name, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, int cluster,
                                    Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = ctx->stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = cluster;
    attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = ctx->use_pdl ? 2 : 1;
    return dc_check_cuda(ctx, cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...), name);
}

template <typename... KArgs, typename... Args>
static inline int dc_launch(dc_ctx* ctx, const char* name, void (*kernel)(KArgs...), dim3 grid, dim3 block,
                            size_t smem, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = ctx->stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = ctx->use_pdl ? 1 : 0;
    return dc_check_cuda(ctx, cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...), name);
}

// The same without the attribute: the kernel starts once the one before has left the SMs.  For the successor of a kernel with
// much shared memory: SMs that never drain keep its split between shared memory and L1, and streaming kernels need the L1.
template <typename... KArgs, typename... Args>
static inline int dc_launch_drained(dc_ctx* ctx, const char* name, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = ctx->stream;
    return dc_check_cuda(ctx, cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...), name);
}
