// Device and host helpers shared by the operator kernels: programmatic dependent launch, warp
// reductions, f32 <-> bf16 element access.
#pragma once
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_runtime.h>

#include <cstdint>

#include "mgq_internal.h"

namespace mgq {

__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;\n" ::: "memory"); }
__device__ __forceinline__ void pdl_launch_dependents() { asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory"); }

// cluster_y: CTAs along y that form a cluster.
template <typename... Params, typename... Args>
int launch_clustered(void (*kernel)(Params...), dim3 grid, dim3 block, uint32_t cluster_y, size_t smem, cudaStream_t stream, Args... args)
{
    cudaLaunchConfig_t lc{};
    lc.gridDim = grid;
    lc.blockDim = block;
    lc.dynamicSmemBytes = smem;
    lc.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = 1;
    attr[1].val.clusterDim.y = cluster_y;
    attr[1].val.clusterDim.z = 1;
    lc.attrs = attr;
    lc.numAttrs = cluster_y > 1 ? 2 : 1;
    MGQ_CUDA(cudaLaunchKernelEx(&lc, kernel, static_cast<Params>(args)...));
    return MGQ_OK;
}
template <typename... Params, typename... Args>
int launch(void (*kernel)(Params...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream, Args... args)
{
    return launch_clustered(kernel, grid, block, 1, smem, stream, static_cast<Params>(args)...);
}

// All CTAs of the cluster: arrive and wait, shared-memory writes before are visible behind.
__device__ __forceinline__ void cluster_sync()
{
    asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;\n" ::: "memory");
}
// A float of the same shared variable in CTA `rank` of the cluster.
__device__ __forceinline__ float cluster_load(const float *p, uint32_t rank)
{
    uint32_t addr;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(addr) : "r"((uint32_t)__cvta_generic_to_shared(p)), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
    return v;
}

// Opts a kernel into more than 48 KB of shared memory, static part included (a no-op for the driver when repeated).
template <typename K>
int allow_smem(K *kernel, size_t bytes)
{
    if (bytes <= 32 * 1024) return MGQ_OK;
    MGQ_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes));
    return MGQ_OK;
}

__device__ __forceinline__ float warp_sum(float v)
{
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v)
{
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f32(__half v) { return __half2float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }
template <> __device__ __forceinline__ __half from_f32<__half>(float v) { return __float2half_rn(fminf(fmaxf(v, -65504.f), 65504.f)); }       // clamped to the range

// 8 consecutive elements, 16-byte aligned source.  Plain loads: activations are written by the kernel this one
// overlaps with, and a read-only-path load might be moved across the wait for it.
__device__ __forceinline__ void unpack8(const uint4 &q, float (&f)[8])
{
    const uint32_t w[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
    for (int i = 0; i < 4; i++) {
        f[2 * i] = __uint_as_float(w[i] << 16);
        f[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u);
    }
}
__device__ __forceinline__ void load8(const __nv_bfloat16 *p, float (&f)[8]) { unpack8(*reinterpret_cast<const uint4 *>(p), f); }
__device__ __forceinline__ void load8(const float *p, float (&f)[8])
{
    const float4 a = *reinterpret_cast<const float4 *>(p), b = *(reinterpret_cast<const float4 *>(p) + 1);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }

// g = min(gate, limit), u = clamp(up, +-limit):  g sigmoid(alpha g) (u + offset).
// limit = infinity, alpha = 1, offset = 0 is the plain silu(gate) * up.
struct Glu {
    float limit, alpha, offset;
};
__device__ __forceinline__ float glu_f(float gate, float up, const Glu &p)
{
    const float g = fminf(gate, p.limit), u = fminf(fmaxf(up, -p.limit), p.limit);
    return g * sigmoid_f(p.alpha * g) * (u + p.offset);
}

}  // namespace mgq
