// Element access and scalar functions shared by the kernels of the hybrid decoders (recurrent and attention mixers). Every
// kernel is instantiated for bf16 and for fp32 activations; arithmetic is fp32 in both. The files that include this are
// compiled without --use_fast_math, so expf, log1pf, division and square root are the accurate ones.
#pragma once
#include "plz_launch.h"

namespace plz {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// eight consecutive elements, 16-byte aligned
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&f)[8]) {
    const uint4 r = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) { f[2 * i] = __uint_as_float(w[i] << 16); f[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u); }
}
__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

__device__ __forceinline__ float gelu_tanh_f(float z) { return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * fmaf(0.044715f * z * z, z, z))); }

// ACT_GLU_GELU: rows 2 i and 2 i + 1 of the weight are a gate / up pair, output column i is gelu_tanh(gate) * up
enum SeqAct { ACT_NONE = 0, ACT_RELU2 = 1, ACT_GLU_GELU = 2 };
__device__ __forceinline__ float activate(float v, int act) {
    if (act == ACT_RELU2) { const float r = fmaxf(v, 0.f); return r * r; }
    return v;
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, o);
    return v;
}
// sum over a block of NW warps; every thread gets the result. `part` is NW floats of shared memory.
template <int NW>
__device__ __forceinline__ float block_sum(float v, float* part) {
    v = warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
    __syncthreads();
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NW; ++i) s += part[i];
    return s;
}

inline int seq_sm_count() {
    static int sms[64] = {};
    int dev = 0;
    cudaGetDevice(&dev);
    if (!sms[dev & 63]) cudaDeviceGetAttribute(&sms[dev & 63], cudaDevAttrMultiProcessorCount, dev);
    return sms[dev & 63];
}

}  // namespace plz
