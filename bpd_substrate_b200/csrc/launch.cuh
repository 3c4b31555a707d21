// Launch helpers of the forward passes.
#pragma once
#include "bpdq_common.cuh"

namespace bpdq {

// A launch that may be scheduled while the launch ahead of it on the stream still runs (every kernel launched this way
// waits for that launch before it touches memory that is not constant).
template <typename... KArgs, typename... Args>
static int launch_cluster(void (*kern)(KArgs...), dim3 grid, dim3 cluster, int block, size_t smem, cudaStream_t s, Args... args)
{
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = dim3((unsigned)block);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute at[2];
    int n = 0;
    if (cluster.x * cluster.y * cluster.z > 1) {
        at[n].id = cudaLaunchAttributeClusterDimension;
        at[n].val.clusterDim.x = cluster.x;
        at[n].val.clusterDim.y = cluster.y;
        at[n++].val.clusterDim.z = cluster.z;
    }
    if (tuning().pdl) {
        at[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        at[n++].val.programmaticStreamSerializationAllowed = 1;
    }
    cfg.attrs = at;
    cfg.numAttrs = n;
    return check_cuda(cudaLaunchKernelEx(&cfg, kern, static_cast<KArgs>(args)...));
}
template <typename... KArgs, typename... Args>
static int launch_ordered(void (*kern)(KArgs...), dim3 grid, int block, size_t smem, cudaStream_t s, Args... args)
{
    return launch_cluster(kern, grid, dim3(1, 1, 1), block, smem, s, args...);
}

static inline int grid_1d(long n)
{
    long want = (n + 255) / 256, cap = (long)sm_count() * 8;
    return (int)(want < 1 ? 1 : (want < cap ? want : cap));
}

// Raises the dynamic shared memory limit of a kernel once per device.
template <auto Kern>
static int allow_smem(int bytes)
{
    static bool done[64] = {false};
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev >= 0 && dev < 64 && done[dev]) return 0;
    int rc = check_cuda(cudaFuncSetAttribute(Kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes));
    if (!rc && dev >= 0 && dev < 64) done[dev] = true;
    return rc;
}

}  // namespace bpdq
