// Kernels around a 32-bit residual stream ("norm after the sum" decoders):
//
//   embedding          x (fp32) and its 16-bit copy that the projections read
//   stream_norm        x <- norm(alpha * x + y) * (1 + w), in place, plus the 16-bit copy; y is a
//                      sublayer's output or, for a mixture of experts, the weighted sum of the
//                      chosen experts' rows, gathered here so that it never exists in memory;
//                      with a row list it also serves the final norm of the sampled rows
//   latent_norm_cache  RMS norm of the compressed K/V projection and its write into the paged
//                      latent cache
//   gated_act          act(gate) * up on the interleaved gate / up layout
//
// T is the model's element type (bf16 or fp32); the stream, the norms and the sums are fp32.

#include "api.h"
#include "common/elem.cuh"
#include "common/pdl.cuh"

namespace ab200 {

template <typename T>
__global__ void __launch_bounds__(256)
stream_embedding_kernel(const long long* __restrict__ ids, const T* __restrict__ table,
                        float* __restrict__ x, T* __restrict__ act, int W, long long vocab,
                        int* status) {
  pdl_wait();
  pdl_trigger();
  const long long t = blockIdx.x;
  const long long id = ids[t];
  const bool ok = id >= 0 && id < vocab;
  // (-1 stands for a token that is not known yet, when a decode step is captured)
  if (id >= vocab && threadIdx.x == 0) report_error(status, kErrBounds, 40, (int)t);
  const T* src = table + (ok ? id : 0) * W;
  for (int i = threadIdx.x; i < W; i += blockDim.x) {
    const T v = ok ? src[i] : from_f32<T>(0.f);
    x[t * W + i] = to_f32<T>(v);
    if (act != nullptr) act[t * W + i] = v;
  }
}

struct StreamNormArgs {
  const float* x;
  const long long* rows;   // optional: input row of each output row
  const void* y;           // optional sublayer output (element type T)
  long long ldy;
  const int* y_rows;       // optional [T][top]: rows of y to sum ...
  const float* y_weights;  // ... and their weights
  int top;
  const float* weight;
  float alpha, eps;
  float* x_out;            // optional
  void* act_out;           // optional
  int W;
};

template <typename T, bool VEC>
__global__ void __launch_bounds__(256) stream_norm_kernel(const StreamNormArgs p) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(16) float row[];
  __shared__ float red[32];
  const long long t = blockIdx.x;
  const long long src = p.rows ? p.rows[t] : t;
  const float* xr = p.x + src * p.W;
  const T* yb = reinterpret_cast<const T*>(p.y);
  float ss = 0.f;
  if (VEC) {
    for (int i = threadIdx.x * 4; i < p.W; i += blockDim.x * 4) {
      float4 s = load4(xr + i);
      s.x *= p.alpha; s.y *= p.alpha; s.z *= p.alpha; s.w *= p.alpha;
      if (p.y_rows != nullptr) {
        for (int j = 0; j < p.top; ++j) {
          const float w = p.y_weights[t * p.top + j];
          const float4 v = load4(yb + (long long)p.y_rows[t * p.top + j] * p.ldy + i);
          s.x += w * v.x; s.y += w * v.y; s.z += w * v.z; s.w += w * v.w;
        }
      } else if (yb != nullptr) {
        const float4 v = load4(yb + t * p.ldy + i);
        s.x += v.x; s.y += v.y; s.z += v.z; s.w += v.w;
      }
      store4(row + i, s);
      ss += s.x * s.x + s.y * s.y + s.z * s.z + s.w * s.w;
    }
  } else {
    for (int i = threadIdx.x; i < p.W; i += blockDim.x) {
      float s = xr[i] * p.alpha;
      if (p.y_rows != nullptr) {
        for (int j = 0; j < p.top; ++j)
          s += p.y_weights[t * p.top + j] *
               to_f32<T>(yb[(long long)p.y_rows[t * p.top + j] * p.ldy + i]);
      } else if (yb != nullptr) {
        s += to_f32<T>(yb[t * p.ldy + i]);
      }
      row[i] = s;
      ss += s * s;
    }
  }
  ss = block_sum_all(ss, red);
  const float inv = 1.f / sqrtf(ss / (float)p.W + p.eps);
  T* act = reinterpret_cast<T*>(p.act_out);
  if (VEC) {
    for (int i = threadIdx.x * 4; i < p.W; i += blockDim.x * 4) {
      float4 s = load4(row + i);
      const float4 w = load4(p.weight + i);
      s.x *= inv * (1.f + w.x); s.y *= inv * (1.f + w.y);
      s.z *= inv * (1.f + w.z); s.w *= inv * (1.f + w.w);
      if (p.x_out) store4(p.x_out + t * p.W + i, s);
      if (act) store4(act + t * p.W + i, s);
    }
  } else {
    for (int i = threadIdx.x; i < p.W; i += blockDim.x) {
      const float s = row[i] * inv * (1.f + p.weight[i]);
      if (p.x_out) p.x_out[t * p.W + i] = s;
      if (act) act[t * p.W + i] = from_f32<T>(s);
    }
  }
}

// c = ckv / rms(ckv) * w over R columns -> cache row `slot` of Rp columns (the rest stays zero).
// One warp per token.
template <typename T>
__global__ void __launch_bounds__(256)
latent_norm_cache_kernel(const T* __restrict__ ckv, long long ld, const float* __restrict__ weight,
                         int R, int Rp, float eps, const long long* __restrict__ slots,
                         T* __restrict__ cache, long long num_slots, long long n, int* status) {
  pdl_wait();
  pdl_trigger();
  const long long t = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (t >= n) return;
  const long long slot = slots[t];
  if (slot < 0) return;    // padding token
  if (slot >= num_slots) {
    if (lane == 0) report_error(status, kErrBounds, 41, (int)t);
    return;
  }
  const T* src = ckv + t * ld;
  T* dst = cache + slot * Rp;
  float ss = 0.f;
  if (((R | Rp) & 3) == 0 && (ld & 3) == 0 &&
      ((reinterpret_cast<uintptr_t>(ckv) | reinterpret_cast<uintptr_t>(weight)) & 15) == 0) {
    constexpr int kHeld = 4;   // of the row's four-element pieces, in registers
    float4 v[kHeld];
#pragma unroll
    for (int j = 0; j < kHeld; ++j) {
      const int i = lane * 4 + 128 * j;
      v[j] = i < R ? load4(src + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int j = 0; j < kHeld; ++j)
      ss += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
    for (int i = lane * 4 + 128 * kHeld; i < R; i += 128) {
      const float4 q = load4(src + i);
      ss += q.x * q.x + q.y * q.y + q.z * q.z + q.w * q.w;
    }
    ss = warp_sum(ss);
    const float inv = 1.f / sqrtf(ss / (float)R + eps);
    auto put = [&](int i, const float4& q) {
      const float4 w = load4(weight + i);
      store4(dst + i, make_float4(q.x * inv * w.x, q.y * inv * w.y, q.z * inv * w.z, q.w * inv * w.w));
    };
#pragma unroll
    for (int j = 0; j < kHeld; ++j)
      if (lane * 4 + 128 * j < R) put(lane * 4 + 128 * j, v[j]);
    for (int i = lane * 4 + 128 * kHeld; i < R; i += 128) put(i, load4(src + i));
    return;
  }
  for (int i = lane; i < R; i += 32) {
    const float v = to_f32<T>(src[i]);
    ss += v * v;
  }
  ss = warp_sum(ss);
  const float inv = 1.f / sqrtf(ss / (float)R + eps);
  for (int i = lane; i < R; i += 32) dst[i] = from_f32<T>(to_f32<T>(src[i]) * inv * weight[i]);
}

template <typename T>
__global__ void __launch_bounds__(256)
gated_act_kernel(const T* __restrict__ gu, T* __restrict__ out, long long n, int ff, int act) {
  pdl_wait();
  pdl_trigger();
  // four outputs per thread: they share a block of kGateBlock
  for (long long i = (blockIdx.x * (long long)blockDim.x + threadIdx.x) * 4; i < n;
       i += (long long)gridDim.x * blockDim.x * 4) {
    const long long t = i / ff;
    const int c = (int)(i - t * ff);
    const T* g = gu + t * 2 * ff + (c / kGateBlock) * (2 * kGateBlock) + c % kGateBlock;
    const float4 a = load4(g), b = load4(g + kGateBlock);
    store4(out + i, make_float4(gate_act(act, a.x) * b.x, gate_act(act, a.y) * b.y,
                                gate_act(act, a.z) * b.z, gate_act(act, a.w) * b.w));
  }
}

template <typename T>
static int launch_stream_norm(const StreamNormArgs& a, long long T_rows, cudaStream_t stream) {
  const size_t smem = (size_t)a.W * sizeof(float);
  if (smem > 200 * 1024) return -6;
  const bool vec = a.W % 4 == 0 && a.ldy % 4 == 0 &&
                   ((reinterpret_cast<uintptr_t>(a.y) | reinterpret_cast<uintptr_t>(a.x) |
                     reinterpret_cast<uintptr_t>(a.weight)) & 15) == 0;
  auto k = vec ? stream_norm_kernel<T, true> : stream_norm_kernel<T, false>;
  if (smem > 48 * 1024 &&
      cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return -3;
  return launch_pdl(k, dim3((unsigned)T_rows), dim3(256), smem, stream, a) == cudaSuccess ? 0 : -5;
}

}  // namespace ab200

using namespace ab200;
typedef __nv_bfloat16 bf16;

extern "C" {

// dtype: 0 = bf16, 1 = fp32 (element type of weights, activations and caches)
int ab200_stream_embedding(const void* ids, const void* table, void* x, void* act, long long T,
                           int W, long long vocab, int dtype, int* status, cudaStream_t stream) {
  if (T <= 0) return 0;
  cudaError_t e;
  if (dtype == 0)
    e = launch_pdl(stream_embedding_kernel<bf16>, dim3((unsigned)T), dim3(256), 0, stream,
                   reinterpret_cast<const long long*>(ids), reinterpret_cast<const bf16*>(table),
                   reinterpret_cast<float*>(x), reinterpret_cast<bf16*>(act), W, vocab, status);
  else
    e = launch_pdl(stream_embedding_kernel<float>, dim3((unsigned)T), dim3(256), 0, stream,
                   reinterpret_cast<const long long*>(ids), reinterpret_cast<const float*>(table),
                   reinterpret_cast<float*>(x), reinterpret_cast<float*>(act), W, vocab, status);
  return e == cudaSuccess ? 0 : -5;
}

// out rows t < T: norm(alpha * x[rows ? rows[t] : t] + y[t]) * (1 + weight). x_out may be x itself
// when rows is null (each block owns its row).
int ab200_stream_norm(const void* x, const void* rows, const void* y, long long ldy,
                      const void* y_rows, const void* y_weights, int top, const void* weight,
                      float alpha, float eps, void* x_out, void* act_out, long long T, int W,
                      int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  StreamNormArgs a;
  a.x = reinterpret_cast<const float*>(x);
  a.rows = reinterpret_cast<const long long*>(rows);
  a.y = y;
  a.ldy = ldy;
  a.y_rows = reinterpret_cast<const int*>(y_rows);
  a.y_weights = reinterpret_cast<const float*>(y_weights);
  a.top = top;
  a.weight = reinterpret_cast<const float*>(weight);
  a.alpha = alpha;
  a.eps = eps;
  a.x_out = reinterpret_cast<float*>(x_out);
  a.act_out = act_out;
  a.W = W;
  return dtype == 0 ? launch_stream_norm<bf16>(a, T, stream) : launch_stream_norm<float>(a, T, stream);
}

int ab200_latent_norm_cache(const void* ckv, long long ld, const void* weight, int R, int Rp,
                            float eps, const void* slots, void* cache, long long num_slots,
                            long long T, int dtype, int* status, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (R > Rp) return -2;
  const dim3 grid((unsigned)((T + 7) / 8));
  cudaError_t e;
  if (dtype == 0)
    e = launch_pdl(latent_norm_cache_kernel<bf16>, grid, dim3(256), 0, stream,
                   reinterpret_cast<const bf16*>(ckv), ld, reinterpret_cast<const float*>(weight),
                   R, Rp, eps, reinterpret_cast<const long long*>(slots),
                   reinterpret_cast<bf16*>(cache), num_slots, T, status);
  else
    e = launch_pdl(latent_norm_cache_kernel<float>, grid, dim3(256), 0, stream,
                   reinterpret_cast<const float*>(ckv), ld, reinterpret_cast<const float*>(weight),
                   R, Rp, eps, reinterpret_cast<const long long*>(slots),
                   reinterpret_cast<float*>(cache), num_slots, T, status);
  return e == cudaSuccess ? 0 : -5;
}

// gu [T, 2 * ff] with gate and up columns alternating in blocks of 16 -> out [T, ff]
int ab200_gated_act(const void* gu, void* out, long long T, int ff, int act, int dtype,
                    cudaStream_t stream) {
  if (T <= 0) return 0;
  if (ff % kGateBlock || (act != kActSilu && act != kActGeluTanh)) return -2;
  const long long n = T * ff;
  long long blocks = (n / 4 + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  cudaError_t e;
  if (dtype == 0)
    e = launch_pdl(gated_act_kernel<bf16>, dim3((unsigned)blocks), dim3(256), 0, stream,
                   reinterpret_cast<const bf16*>(gu), reinterpret_cast<bf16*>(out), n, ff, act);
  else
    e = launch_pdl(gated_act_kernel<float>, dim3((unsigned)blocks), dim3(256), 0, stream,
                   reinterpret_cast<const float*>(gu), reinterpret_cast<float*>(out), n, ff, act);
  return e == cudaSuccess ? 0 : -5;
}

}  // extern "C"
