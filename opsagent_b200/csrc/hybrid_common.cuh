// hybrid_common.cuh — small device helpers shared by the hybrid family's kernel files: typed loads / stores of the activation type
// (bf16 or fp32, arithmetic always fp32), activations, block reductions, cp.async, and the launch wrapper that joins every kernel to the
// stream's programmatic-dependent-launch chain.
#pragma once
#include <cuda_bf16.h>
#include <math.h>

#include <utility>

#include "common.cuh"
#include "kernels.hpp"

namespace oa {
namespace hyk {

__device__ __forceinline__ float ldf(const float* p) { return *p; }
__device__ __forceinline__ float ldf(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stf(float* p, float v) { *p = v; }
__device__ __forceinline__ void stf(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float sigmoidf_(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float siluf_(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float gelu_tanhf_(float z) { return gelu_tanh_f32(z); }
__device__ __forceinline__ float softplusf_(float z) { return z > 20.0f ? z : log1pf(expf(z)); }
// sum over the block (blockDim.x <= 1024, a multiple of 32); every thread gets the result
__device__ __forceinline__ float block_sum(float v, float* red) {
    v = warp_sum(v);
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = blockDim.x >> 5;
    __syncthreads();
    if (l == 0) red[w] = v;
    __syncthreads();
    float t = 0.f;
    for (int i = 0; i < nw; ++i) t += red[i];
    return t;
}

__device__ __forceinline__ void cp_async16(void* smem, const void* gmem) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem)), "l"(gmem) : "memory");
}

// 8 channels of an aligned bf16 / fp32 row
__device__ __forceinline__ void unpack8(const uint4& r, float* f) {
    f[0] = bf16lo(r.x); f[1] = bf16hi(r.x); f[2] = bf16lo(r.y); f[3] = bf16hi(r.y); f[4] = bf16lo(r.z); f[5] = bf16hi(r.z); f[6] = bf16lo(r.w); f[7] = bf16hi(r.w);
}
__device__ __forceinline__ void ld8f(const float* p, float* f) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void st8f(float* p, const float* f) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); *reinterpret_cast<float4*>(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
}
// an fp32 value as a bf16 value plus a bf16 remainder: together accurate to about 2^-16 of its size
__device__ __forceinline__ void split_bf16(float x, __nv_bfloat16& hi, __nv_bfloat16& lo) { hi = __float2bfloat16_rn(x); lo = __float2bfloat16_rn(x - __bfloat162float(hi)); }
__device__ __forceinline__ void split_pack(float a, float b, uint32_t& hi, uint32_t& lo) { hi = pack_bf16x2(a, b); lo = pack_bf16x2(a - bf16lo(hi), b - bf16hi(hi)); }

// Every kernel of the family opens with HY_PDL(): it lets the next kernel of the stream become resident early (programmatic dependent
// launch) and then waits until every predecessor grid has completed and its memory is visible — nothing is read or written before that, so
// the kernels stay strictly ordered; what overlaps is only the launch latency and the ramp of the next grid.
#define HY_PDL() do { griddep_launch(); griddep_wait(); } while (0)
template <typename... KArgs, typename... Args>
cudaError_t launch_plain(void (*kern)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t st, Args&&... args) {
    return launch_k(kern, grid, block, smem, st, std::forward<Args>(args)...);
}


}  // namespace hyk
}  // namespace oa
