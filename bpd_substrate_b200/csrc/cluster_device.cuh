// Thread-block clusters and distributed shared memory; clusters here extend along y only.
#pragma once
#include "bpdq_common.cuh"

namespace bpdq {

__device__ __forceinline__ uint32_t cluster_size()
{
    uint32_t n;
    asm volatile("mov.u32 %0, %%cluster_nctaid.y;" : "=r"(n));
    return n;
}
__device__ __forceinline__ uint32_t cluster_rank()
{
    uint32_t r;
    asm volatile("mov.u32 %0, %%cluster_ctaid.y;" : "=r"(r));
    return r;
}
// All threads of all CTAs; memory written before the arrival is seen after the wait.
__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }

__device__ __forceinline__ uint32_t peer_addr(const void* p, uint32_t rank)
{
    uint32_t a;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(a) : "r"(smem_addr(p)), "r"(rank));
    return a;
}
__device__ __forceinline__ void store_peer(const float* p, uint32_t rank, float v)
{
    asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(peer_addr(p, rank)), "f"(v) : "memory");
}
__device__ __forceinline__ float load_peer(const float* p, uint32_t rank)
{
    float v;
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(peer_addr(p, rank)) : "memory");
    return v;
}
__device__ __forceinline__ float4 load_peer4(const float* p, uint32_t rank)
{
    float4 v;
    asm volatile("ld.shared::cluster.v4.f32 {%0,%1,%2,%3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(peer_addr(p, rank)) : "memory");
    return v;
}

}  // namespace bpdq
