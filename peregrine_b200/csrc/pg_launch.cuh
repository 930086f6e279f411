// Launches with programmatic stream serialisation (the next kernel's prologue overlaps this one's tail), optionally as
// clusters; shared by the row kernels.
#pragma once

#include "pg_internal.cuh"

template <typename K, typename... Args>
inline int32_t launch_pdl_cluster(pg_ctx *ctx, K kern, dim3 grid, dim3 block, size_t smem, int cs, Args... args)
{
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = (unsigned)cs;
    attr[1].val.clusterDim.y = 1;
    attr[1].val.clusterDim.z = 1;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = ctx->stream;
    cfg.attrs = attr;
    cfg.numAttrs = cs > 1 ? 2 : 1;
    PG_CUDA(cudaLaunchKernelEx(&cfg, kern, args...));
    PG_LAUNCHED();
    return PG_OK;
}

// The same, but started when everything before it has ended.  The first kernel of a step is launched this way, so that the
// kernels behind it may read the batch's arrays, and what earlier steps left in caches and states, before they wait.
template <typename K, typename... Args>
inline int32_t launch_whole_cluster(pg_ctx *ctx, K kern, dim3 grid, dim3 block, size_t smem, int cs, Args... args)
{
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = (unsigned)cs;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = 1;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = ctx->stream;
    cfg.attrs = attr;
    cfg.numAttrs = cs > 1 ? 1 : 0;
    PG_CUDA(cudaLaunchKernelEx(&cfg, kern, args...));
    PG_LAUNCHED();
    return PG_OK;
}

// CTAs per row for the row kernels: as many (up to 8) as keep the grid within about two CTAs per SM, divide the row's
// `units` evenly and leave each CTA at least `min_units`.
inline int row_cluster(const pg_ctx *ctx, int64_t rows, int64_t units, int64_t min_units)
{
    int cs = 8;
    while (cs > 1 && (rows * cs > 2 * (int64_t)ctx->sm_count || units % cs != 0 || units / cs < min_units)) cs >>= 1;
    return cs;
}

template <typename K, typename... Args>
inline int32_t launch_pdl(pg_ctx *ctx, K kern, dim3 grid, dim3 block, size_t smem, Args... args)
{
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = ctx->stream;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    PG_CUDA(cudaLaunchKernelEx(&cfg, kern, args...));
    PG_LAUNCHED();
    return PG_OK;
}

// A launch that starts when everything before it has ended.  For long kernels with about one CTA per SM: started early,
// their CTAs are placed around those of the predecessor, several on one SM and none on others, and stay there.
template <typename K, typename... Args>
inline int32_t launch_whole(pg_ctx *ctx, K kern, dim3 grid, dim3 block, size_t smem, Args... args)
{
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = ctx->stream;
    PG_CUDA(cudaLaunchKernelEx(&cfg, kern, args...));
    PG_LAUNCHED();
    return PG_OK;
}
