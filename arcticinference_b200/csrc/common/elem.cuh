// Element access shared by the kernels that serve 16-bit and 32-bit models: loads widen to fp32,
// stores round once. Gated activations in fp32.
#pragma once

#include <math.h>

#include "ptx.cuh"

namespace ab200 {

template <typename T>
__device__ __forceinline__ float to_f32(T v);
template <>
__device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// four consecutive elements (the address is a multiple of four elements)
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 q = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float4& v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}

// Packed fp32 pairs
__device__ __forceinline__ void fma2(float2& d, const float2& a, const float2& b) {
  asm("fma.rn.f32x2 %0, %1, %2, %0;"
      : "+l"(reinterpret_cast<unsigned long long&>(d))
      : "l"(reinterpret_cast<const unsigned long long&>(a)),
        "l"(reinterpret_cast<const unsigned long long&>(b)));
}
__device__ __forceinline__ void mul2(float2& d, const float2& a) {
  asm("mul.rn.f32x2 %0, %0, %1;"
      : "+l"(reinterpret_cast<unsigned long long&>(d))
      : "l"(reinterpret_cast<const unsigned long long&>(a)));
}
__device__ __forceinline__ void add2(float2& d, const float2& a) {
  asm("add.rn.f32x2 %0, %0, %1;"
      : "+l"(reinterpret_cast<unsigned long long&>(d))
      : "l"(reinterpret_cast<const unsigned long long&>(a)));
}

// Block-wide sum; `red` is 32 floats of shared memory. Every thread gets the sum.
__device__ __forceinline__ float block_sum_all(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int nwarps = (blockDim.x + 31) >> 5;
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  return warp_sum(lane < nwarps ? red[lane] : 0.f);
}
__device__ __forceinline__ float block_max_all(float v, float* red) {
  v = warp_max(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int nwarps = (blockDim.x + 31) >> 5;
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  return warp_max(lane < nwarps ? red[lane] : -INFINITY);
}

// Gated activations: silu(g) * u, gelu_tanh(g) * u, and the clamped swish
// min(g, limit) * sigmoid(alpha * min(g, limit)) * (clamp(u, -limit, limit) + 1).
enum GatedAct : int { kActSilu = 1, kActGeluTanh = 2, kActClampedSwish = 3 };

struct GateParams {
  float limit, alpha;   // of the clamped swish
};

__device__ __forceinline__ float gate_silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float gate_gelu_tanh(float z) {
  const float k = 0.79788456080286535588f;   // sqrt(2 / pi)
  return 0.5f * z * (1.f + tanhf(k * (z + 0.044715f * z * z * z)));
}
__device__ __forceinline__ float gated(int act, const GateParams& p, float g, float u) {
  if (act == kActClampedSwish) {
    g = fminf(g, p.limit);
    return g / (1.f + expf(-p.alpha * g)) * (fminf(fmaxf(u, -p.limit), p.limit) + 1.f);
  }
  return (act == kActSilu ? gate_silu(g) : gate_gelu_tanh(g)) * u;
}

// Which keys a token at position `pos` sees: first_visible .. pos.
enum MaskKind : int { kMaskCausal = 0, kMaskWindow = 1, kMaskChunk = 2 };

__host__ __device__ __forceinline__ int first_visible(int kind, int size, int pos) {
  if (kind == kMaskWindow) return pos >= size ? pos - size + 1 : 0;
  if (kind == kMaskChunk) return pos / size * size;
  return 0;
}

// Gate and up projections are stored as one matrix whose rows alternate in blocks of this many:
// 16 gate rows, then the 16 up rows they belong to. A 32-column piece of the product holds both
// factors of 16 outputs, so a tile's epilogue can apply the activation.
constexpr int kGateBlock = 16;

}  // namespace ab200
