// Kernels around a 32-bit residual stream (decoders that list their layers):
//
//   embedding          x (fp32, scaled) and its 16-bit copy that the projections read; optionally plus
//                      a second table's row, looked up by the token and the one before it
//   stream_norm        x <- norm(alpha * x + y) * (1 + w), in place, plus the 16-bit copy; y is a
//                      sublayer's output or, for a mixture of experts, the weighted sum of the
//                      chosen experts' rows, gathered here so that it never exists in memory;
//                      with a row list it also serves the final norm of the sampled rows
//   stream_sandwich    x <- x + norm(y) * w_out (+ a vector), in place, and the next sublayer's
//                      input act = norm(x) * w_in, in one pass over the row
//   stream_add         x <- x + norm(y) * w, in place, and the 16-bit copy; y is a sublayer's output,
//                      half the sum of two normed ones, or a mixture of experts' weighted sum with
//                      identity experts and a shared expert, formed here in fp32
//   stream_pre         x <- x + m * y (+ the embedding) (+ a vector), in place, and the next sublayer's
//                      input act = norm(x) * w, in one pass over the row; y is a sublayer's output plus
//                      a bias, or a mixture of experts' weighted sum plus a shared expert's rows
//   poly_norm          a N(z) + b N(z^2) + c N(z^3) + e over the rows of an up projection, N dividing
//                      by the row's root mean square; the projection's bias is added here
//   soft_cap           fp32 logits cap * tanh(z / cap)
//   latent_norm_cache  RMS norm of the compressed K/V projection and its write into the paged
//                      latent cache
//   gated_act          act(gate) * up on the interleaved gate / up layout
//
// T is the model's element type (bf16 or fp32); the stream, the norms and the sums are fp32.

#include "api.h"
#include "common/elem.cuh"
#include "common/pdl.cuh"

namespace ab200 {

// The second embedding: row (prev * mul_prev + id * mul_cur) mod buckets of `table`, the last row where
// there is no previous token
struct PairArgs {
  const long long* prev;   // [T], negative: none; null: no second embedding
  const void* table;       // [buckets + 1][W]
  long long buckets, mul_prev, mul_cur;
};

template <typename T>
__global__ void __launch_bounds__(256)
stream_embedding_kernel(const long long* __restrict__ ids, const T* __restrict__ table,
                        float* __restrict__ x, T* __restrict__ act, float* __restrict__ keep, float scale,
                        int W, long long vocab, const PairArgs pairs, int* status) {
  pdl_wait();
  pdl_trigger();
  const long long t = blockIdx.x;
  const long long id = ids[t];
  const bool ok = id >= 0 && id < vocab;
  // (-1 stands for a token that is not known yet, when a decode step is captured)
  if (id >= vocab && threadIdx.x == 0) report_error(status, kErrBounds, 40, (int)t);
  const T* src = table + (ok ? id : 0) * W;
  const T* second = nullptr;
  if (pairs.prev != nullptr) {
    const long long before = pairs.prev[t];
    long long row = pairs.buckets;
    if (before >= 0 && ok) {
      row = (before * pairs.mul_prev + id * pairs.mul_cur) % pairs.buckets;
      if (row < 0) row += pairs.buckets;
    }
    second = reinterpret_cast<const T*>(pairs.table) + row * W;
  }
  if (W % 4 == 0 && ((reinterpret_cast<uintptr_t>(table) | reinterpret_cast<uintptr_t>(x) |
                      reinterpret_cast<uintptr_t>(act) | reinterpret_cast<uintptr_t>(keep) |
                      reinterpret_cast<uintptr_t>(pairs.table)) & 15) == 0) {
    for (int i = threadIdx.x * 4; i < W; i += blockDim.x * 4) {
      float4 v = ok ? load4(src + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      v = make_float4(v.x * scale, v.y * scale, v.z * scale, v.w * scale);
      if (second != nullptr) {
        const float4 u = load4(second + i);
        v = make_float4(v.x + u.x, v.y + u.y, v.z + u.z, v.w + u.w);
      }
      store4(x + t * W + i, v);
      if (keep != nullptr) store4(keep + t * W + i, v);
      if (act != nullptr) store4(act + t * W + i, v);
    }
    return;
  }
  for (int i = threadIdx.x; i < W; i += blockDim.x) {
    float v = ok ? to_f32<T>(src[i]) * scale : 0.f;
    if (second != nullptr) v += to_f32<T>(second[i]);
    x[t * W + i] = v;
    if (keep != nullptr) keep[t * W + i] = v;
    if (act != nullptr) act[t * W + i] = from_f32<T>(v);
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
  float alpha, eps, offset;   // offset: added to the weight
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
      s.x *= inv * (p.offset + w.x); s.y *= inv * (p.offset + w.y);
      s.z *= inv * (p.offset + w.z); s.w *= inv * (p.offset + w.w);
      if (p.x_out) store4(p.x_out + t * p.W + i, s);
      if (act) store4(act + t * p.W + i, s);
    }
  } else {
    for (int i = threadIdx.x; i < p.W; i += blockDim.x) {
      const float s = row[i] * inv * (p.offset + p.weight[i]);
      if (p.x_out) p.x_out[t * p.W + i] = s;
      if (act) act[t * p.W + i] = from_f32<T>(s);
    }
  }
}

struct SandwichArgs {
  float* x;                // updated in place when y or step is given
  const void* y;           // optional sublayer output (element type T)
  long long ldy;
  const float* w_out;      // its norm's weight
  const float* step;       // optional vector added to the stream after it
  const float* w_in;       // optional: norm of the new stream, written to act
  void* act;
  float eps, offset;
  int W;
};

// N4: four-element pieces of the row a thread holds in registers (0: any width, through memory)
template <typename T, int N4>
__global__ void __launch_bounds__(256) stream_sandwich_kernel(const SandwichArgs p) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[32];
  const long long t = blockIdx.x;
  float* xr = p.x + t * p.W;
  const T* yr = p.y ? reinterpret_cast<const T*>(p.y) + t * p.ldy : nullptr;
  T* act = p.act ? reinterpret_cast<T*>(p.act) + t * p.W : nullptr;
  const float rw = 1.f / (float)p.W;
  if constexpr (N4 > 0) {
    float4 x[N4], y[N4];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < N4; ++j) {
      const int i = (threadIdx.x + j * blockDim.x) * 4;
      x[j] = i < p.W ? load4(xr + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      y[j] = (yr != nullptr && i < p.W) ? load4(yr + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += y[j].x * y[j].x + y[j].y * y[j].y + y[j].z * y[j].z + y[j].w * y[j].w;
    }
    if (yr != nullptr) {
      const float inv = 1.f / sqrtf(block_sum_all(ss, red) * rw + p.eps);
#pragma unroll
      for (int j = 0; j < N4; ++j) {
        const int i = (threadIdx.x + j * blockDim.x) * 4;
        if (i >= p.W) continue;
        const float4 w = load4(p.w_out + i);
        x[j].x += y[j].x * inv * (p.offset + w.x);
        x[j].y += y[j].y * inv * (p.offset + w.y);
        x[j].z += y[j].z * inv * (p.offset + w.z);
        x[j].w += y[j].w * inv * (p.offset + w.w);
      }
    }
    ss = 0.f;
#pragma unroll
    for (int j = 0; j < N4; ++j) {
      const int i = (threadIdx.x + j * blockDim.x) * 4;
      if (i >= p.W) continue;
      if (p.step != nullptr) {
        const float4 s = load4(p.step + i);
        x[j].x += s.x; x[j].y += s.y; x[j].z += s.z; x[j].w += s.w;
      }
      if (yr != nullptr || p.step != nullptr) store4(xr + i, x[j]);
      ss += x[j].x * x[j].x + x[j].y * x[j].y + x[j].z * x[j].z + x[j].w * x[j].w;
    }
    if (act == nullptr) return;
    const float inv = 1.f / sqrtf(block_sum_all(ss, red) * rw + p.eps);
#pragma unroll
    for (int j = 0; j < N4; ++j) {
      const int i = (threadIdx.x + j * blockDim.x) * 4;
      if (i >= p.W) continue;
      const float4 w = load4(p.w_in + i);
      store4(act + i, make_float4(x[j].x * inv * (p.offset + w.x), x[j].y * inv * (p.offset + w.y),
                                  x[j].z * inv * (p.offset + w.z), x[j].w * inv * (p.offset + w.w)));
    }
  } else {
    float inv = 0.f, ss = 0.f;
    if (yr != nullptr) {
      for (int i = threadIdx.x; i < p.W; i += blockDim.x) {
        const float v = to_f32<T>(yr[i]);
        ss += v * v;
      }
      inv = 1.f / sqrtf(block_sum_all(ss, red) * rw + p.eps);
    }
    ss = 0.f;
    for (int i = threadIdx.x; i < p.W; i += blockDim.x) {   // a thread re-reads only its own columns
      float v = xr[i];
      if (yr != nullptr) v += to_f32<T>(yr[i]) * inv * (p.offset + p.w_out[i]);
      if (p.step != nullptr) v += p.step[i];
      if (yr != nullptr || p.step != nullptr) xr[i] = v;
      ss += v * v;
    }
    if (act == nullptr) return;
    inv = 1.f / sqrtf(block_sum_all(ss, red) * rw + p.eps);
    for (int i = threadIdx.x; i < p.W; i += blockDim.x)
      act[i] = from_f32<T>(xr[i] * inv * (p.offset + p.w_in[i]));
  }
}

template <typename T>
static int launch_stream_sandwich(const SandwichArgs& a, long long T_rows, cudaStream_t stream) {
  const bool vec = a.W % 4 == 0 && a.ldy % 4 == 0 &&
                   ((reinterpret_cast<uintptr_t>(a.y) | reinterpret_cast<uintptr_t>(a.x) |
                     reinterpret_cast<uintptr_t>(a.w_out) | reinterpret_cast<uintptr_t>(a.step) |
                     reinterpret_cast<uintptr_t>(a.w_in) | reinterpret_cast<uintptr_t>(a.act)) & 15) == 0;
  const int n4 = (a.W + 3) / 4;
  auto k = stream_sandwich_kernel<T, 0>;
  int threads = 256;
  if (vec && n4 <= 256 * 8) {
    // few enough pieces per thread to stay in registers, few enough threads to have work
    while (threads > 64 && n4 <= threads) threads /= 2;
    const int per = (n4 + threads - 1) / threads;
    k = per <= 1   ? stream_sandwich_kernel<T, 1>
        : per <= 2 ? stream_sandwich_kernel<T, 2>
        : per <= 4 ? stream_sandwich_kernel<T, 4>
                   : stream_sandwich_kernel<T, 8>;
  }
  return launch_pdl(k, dim3((unsigned)T_rows), dim3(threads), 0, stream, a) == cudaSuccess ? 0 : -5;
}

struct StreamAddArgs {
  float* x;
  void* act;               // optional copy in element type T
  const float* w;          // norm weight
  const void* y;           // a sublayer's output rows (a mixture: the experts' rows)
  long long ldy;
  const float* wy;         // with y2: weights of the two outputs' own norms
  const void* y2;
  long long ldy2;
  const float* wy2;
  const int* y_rows;       // mixture: [T][top] rows of y, -1: the token's own stream
  const float* y_weights;
  int top;
  const void* shared;      // mixture: further rows to add, or null
  long long ld_shared;
  float eps;
  int W;
};

// N4: four-element pieces a thread holds (0: any width, the sublayer's output through shared memory)
template <typename T, int N4>
__global__ void __launch_bounds__(256) stream_add_kernel(const StreamAddArgs p) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[32];
  extern __shared__ __align__(16) float row[];
  const long long t = blockIdx.x;
  float* xr = p.x + t * p.W;
  const T* yb = reinterpret_cast<const T*>(p.y);
  const T* y2 = p.y2 ? reinterpret_cast<const T*>(p.y2) + t * p.ldy2 : nullptr;
  const T* sh = p.shared ? reinterpret_cast<const T*>(p.shared) + t * p.ld_shared : nullptr;
  T* act = p.act ? reinterpret_cast<T*>(p.act) + t * p.W : nullptr;
  const float rw = 1.f / (float)p.W;
  if constexpr (N4 > 0) {
    float4 x[N4], y[N4];
    auto each = [&](auto f) {
#pragma unroll
      for (int j = 0; j < N4; ++j) {
        const int i = (threadIdx.x + j * blockDim.x) * 4;
        if (i < p.W) f(i, x[j], y[j]);
      }
    };
    auto square = [](const float4& v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; };
    float ss = 0.f;
    if (p.y_rows != nullptr) {
      each([&](int i, float4& xv, float4& yv) {
        xv = load4(xr + i);
        yv = sh != nullptr ? load4(sh + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        for (int k = 0; k < p.top; ++k) {
          const float w = p.y_weights[t * p.top + k];
          const int r = p.y_rows[t * p.top + k];
          const float4 v = r >= 0 ? load4(yb + (long long)r * p.ldy + i) : xv;
          yv.x += w * v.x; yv.y += w * v.y; yv.z += w * v.z; yv.w += w * v.w;
        }
        ss += square(yv);
      });
    } else if (y2 != nullptr) {
      float s2 = 0.f;
      float4 z[N4];
      each([&](int i, float4& xv, float4& yv) {
        xv = load4(xr + i);
        yv = load4(yb + t * p.ldy + i);
        ss += square(yv);
      });
#pragma unroll
      for (int j = 0; j < N4; ++j) {
        const int i = (threadIdx.x + j * blockDim.x) * 4;
        z[j] = i < p.W ? load4(y2 + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        s2 += square(z[j]);
      }
      const float a = 0.5f / sqrtf(block_sum_all(ss, red) * rw + p.eps);
      const float b = 0.5f / sqrtf(block_sum_all(s2, red) * rw + p.eps);
      ss = 0.f;
#pragma unroll
      for (int j = 0; j < N4; ++j) {
        const int i = (threadIdx.x + j * blockDim.x) * 4;
        if (i >= p.W) continue;
        const float4 u = load4(p.wy + i), v = load4(p.wy2 + i);
        y[j] = make_float4(y[j].x * a * u.x + z[j].x * b * v.x, y[j].y * a * u.y + z[j].y * b * v.y,
                           y[j].z * a * u.z + z[j].z * b * v.z, y[j].w * a * u.w + z[j].w * b * v.w);
        ss += square(y[j]);
      }
    } else {
      each([&](int i, float4& xv, float4& yv) {
        xv = load4(xr + i);
        yv = load4(yb + t * p.ldy + i);
        ss += square(yv);
      });
    }
    const float inv = 1.f / sqrtf(block_sum_all(ss, red) * rw + p.eps);
    each([&](int i, float4& xv, float4& yv) {
      const float4 w = load4(p.w + i);
      xv.x += yv.x * inv * w.x; xv.y += yv.y * inv * w.y;
      xv.z += yv.z * inv * w.z; xv.w += yv.w * inv * w.w;
      store4(xr + i, xv);
      if (act != nullptr) store4(act + i, xv);
    });
  } else {
    float ss = 0.f, s2 = 0.f, a = 0.f, b = 0.f;
    if (y2 != nullptr) {
      for (int i = threadIdx.x; i < p.W; i += blockDim.x) {
        const float u = to_f32<T>(yb[t * p.ldy + i]), v = to_f32<T>(y2[i]);
        ss += u * u;
        s2 += v * v;
      }
      a = 0.5f / sqrtf(block_sum_all(ss, red) * rw + p.eps);
      b = 0.5f / sqrtf(block_sum_all(s2, red) * rw + p.eps);
      ss = 0.f;
    }
    for (int i = threadIdx.x; i < p.W; i += blockDim.x) {   // a thread re-reads only its own columns
      float v;
      if (p.y_rows != nullptr) {
        v = sh != nullptr ? to_f32<T>(sh[i]) : 0.f;
        for (int k = 0; k < p.top; ++k) {
          const int r = p.y_rows[t * p.top + k];
          v += p.y_weights[t * p.top + k] * (r >= 0 ? to_f32<T>(yb[(long long)r * p.ldy + i]) : xr[i]);
        }
      } else {
        v = to_f32<T>(yb[t * p.ldy + i]);
        if (y2 != nullptr) v = v * a * p.wy[i] + to_f32<T>(y2[i]) * b * p.wy2[i];
      }
      row[i] = v;
      ss += v * v;
    }
    const float inv = 1.f / sqrtf(block_sum_all(ss, red) * rw + p.eps);
    for (int i = threadIdx.x; i < p.W; i += blockDim.x) {
      const float v = xr[i] + row[i] * inv * p.w[i];
      xr[i] = v;
      if (act != nullptr) act[i] = from_f32<T>(v);
    }
  }
}

template <typename T>
static int launch_stream_add(const StreamAddArgs& a, long long T_rows, cudaStream_t stream) {
  const bool vec = a.W % 4 == 0 && a.ldy % 4 == 0 && a.ldy2 % 4 == 0 && a.ld_shared % 4 == 0 &&
                   ((reinterpret_cast<uintptr_t>(a.y) | reinterpret_cast<uintptr_t>(a.x) |
                     reinterpret_cast<uintptr_t>(a.y2) | reinterpret_cast<uintptr_t>(a.shared) |
                     reinterpret_cast<uintptr_t>(a.w) | reinterpret_cast<uintptr_t>(a.wy) |
                     reinterpret_cast<uintptr_t>(a.wy2) | reinterpret_cast<uintptr_t>(a.act)) & 15) == 0;
  const int n4 = (a.W + 3) / 4;
  auto k = stream_add_kernel<T, 0>;
  int threads = 256;
  size_t smem = 0;
  if (vec && n4 <= 256 * 8) {
    while (threads > 64 && n4 <= threads) threads /= 2;
    const int per = (n4 + threads - 1) / threads;
    k = per <= 1   ? stream_add_kernel<T, 1>
        : per <= 2 ? stream_add_kernel<T, 2>
        : per <= 4 ? stream_add_kernel<T, 4>
                   : stream_add_kernel<T, 8>;
  } else {
    smem = (size_t)a.W * sizeof(float);
    if (smem > 200 * 1024) return -6;
    if (smem > 48 * 1024 &&
        cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return -3;
  }
  return launch_pdl(k, dim3((unsigned)T_rows), dim3(threads), smem, stream, a) == cudaSuccess ? 0 : -5;
}

struct StreamPreArgs {
  float* x;
  const void* y;           // optional sublayer output (a mixture: the experts' rows)
  long long ldy;
  const float* bias;       // optional [W], added to y
  const int* y_rows;       // mixture: [T][top] rows of y
  const float* y_weights;
  int top;
  const void* shared;      // optional further rows to add
  long long ld_shared;
  float mult;              // of all that
  const float* base;       // optional [T][W], added to the stream after it
  const float* step;       // optional [W], likewise
  const float* w_in;       // with act: weight of the new stream's norm, [W] or (w_scalar) one number
  int w_scalar;
  void* act;
  float eps;
  int W;
};

// N4: four-element pieces of the row a thread holds in registers (0: any width, through memory)
template <typename T, int N4>
__global__ void __launch_bounds__(256) stream_pre_kernel(const StreamPreArgs p) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[32];
  const long long t = blockIdx.x;
  float* xr = p.x + t * p.W;
  const T* yb = reinterpret_cast<const T*>(p.y);
  const T* sh = p.shared ? reinterpret_cast<const T*>(p.shared) + t * p.ld_shared : nullptr;
  const float* base = p.base ? p.base + t * p.W : nullptr;
  T* act = p.act ? reinterpret_cast<T*>(p.act) + t * p.W : nullptr;
  const bool moved = yb != nullptr || base != nullptr || p.step != nullptr;
  const float gain = p.w_scalar ? p.w_in[0] : 1.f;
  const float rw = 1.f / (float)p.W;
  if constexpr (N4 > 0) {
    float4 x[N4], f[N4];
    auto add = [](float4& a, const float4& b) { a.x += b.x; a.y += b.y; a.z += b.z; a.w += b.w; };
    auto axpy = [](float4& a, float m, const float4& b) {
      a.x = fmaf(m, b.x, a.x); a.y = fmaf(m, b.y, a.y);
      a.z = fmaf(m, b.z, a.z); a.w = fmaf(m, b.w, a.w);
    };
    auto each = [&](auto g) {
#pragma unroll
      for (int j = 0; j < N4; ++j) {
        const int i = (threadIdx.x + j * blockDim.x) * 4;
        if (i < p.W) g(i, x[j], f[j]);
      }
    };
    each([&](int i, float4& xv, float4& fv) {
      xv = load4(xr + i);
      fv = sh != nullptr ? load4(sh + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    });
    if (p.y_rows != nullptr) {
      for (int k = 0; k < p.top; ++k) {
        const float w = p.y_weights[t * p.top + k];
        const T* yr = yb + (long long)p.y_rows[t * p.top + k] * p.ldy;
        each([&](int i, float4&, float4& fv) { axpy(fv, w, load4(yr + i)); });
      }
    } else if (yb != nullptr) {
      each([&](int i, float4&, float4& fv) { add(fv, load4(yb + t * p.ldy + i)); });
    }
    if (p.bias != nullptr) each([&](int i, float4&, float4& fv) { add(fv, load4(p.bias + i)); });
    float ss = 0.f;
    each([&](int i, float4& xv, float4& fv) {
      axpy(xv, p.mult, fv);
      if (base != nullptr) add(xv, load4(base + i));
      if (p.step != nullptr) add(xv, load4(p.step + i));
      if (moved) store4(xr + i, xv);
      ss += xv.x * xv.x + xv.y * xv.y + xv.z * xv.z + xv.w * xv.w;
    });
    if (act == nullptr) return;
    const float inv = gain / sqrtf(block_sum_all(ss, red) * rw + p.eps);
    each([&](int i, float4& xv, float4&) {
      float4 w = make_float4(inv, inv, inv, inv);
      if (!p.w_scalar) {
        const float4 v = load4(p.w_in + i);
        w = make_float4(inv * v.x, inv * v.y, inv * v.z, inv * v.w);
      }
      store4(act + i, make_float4(xv.x * w.x, xv.y * w.y, xv.z * w.z, xv.w * w.w));
    });
  } else {
    float ss = 0.f;
    for (int i = threadIdx.x; i < p.W; i += blockDim.x) {   // a thread re-reads only its own columns
      float f = sh != nullptr ? to_f32<T>(sh[i]) : 0.f;
      if (p.y_rows != nullptr) {
        for (int k = 0; k < p.top; ++k)
          f = fmaf(p.y_weights[t * p.top + k],
                   to_f32<T>(yb[(long long)p.y_rows[t * p.top + k] * p.ldy + i]), f);
      } else if (yb != nullptr) {
        f += to_f32<T>(yb[t * p.ldy + i]);
      }
      if (p.bias != nullptr) f += p.bias[i];
      float v = fmaf(p.mult, f, xr[i]);
      if (base != nullptr) v += base[i];
      if (p.step != nullptr) v += p.step[i];
      if (moved) xr[i] = v;
      ss += v * v;
    }
    if (act == nullptr) return;
    const float inv = gain / sqrtf(block_sum_all(ss, red) * rw + p.eps);
    for (int i = threadIdx.x; i < p.W; i += blockDim.x)
      act[i] = from_f32<T>(xr[i] * (p.w_scalar ? inv : inv * p.w_in[i]));
  }
}

template <typename T>
static int launch_stream_pre(const StreamPreArgs& a, long long T_rows, cudaStream_t stream) {
  const bool vec = a.W % 4 == 0 && a.ldy % 4 == 0 && a.ld_shared % 4 == 0 &&
                   ((reinterpret_cast<uintptr_t>(a.y) | reinterpret_cast<uintptr_t>(a.x) |
                     reinterpret_cast<uintptr_t>(a.shared) | reinterpret_cast<uintptr_t>(a.bias) |
                     reinterpret_cast<uintptr_t>(a.base) | reinterpret_cast<uintptr_t>(a.step) |
                     (a.w_scalar ? 0 : reinterpret_cast<uintptr_t>(a.w_in)) |
                     reinterpret_cast<uintptr_t>(a.act)) & 15) == 0;
  const int n4 = (a.W + 3) / 4;
  auto k = stream_pre_kernel<T, 0>;
  int threads = 256;
  if (vec && n4 <= 256 * 8) {
    while (threads > 64 && n4 <= threads) threads /= 2;
    const int per = (n4 + threads - 1) / threads;
    k = per <= 1   ? stream_pre_kernel<T, 1>
        : per <= 2 ? stream_pre_kernel<T, 2>
        : per <= 4 ? stream_pre_kernel<T, 4>
                   : stream_pre_kernel<T, 8>;
  }
  return launch_pdl(k, dim3((unsigned)T_rows), dim3(threads), 0, stream, a) == cudaSuccess ? 0 : -5;
}

// Rows of n columns of which the first ff count; a block takes rows gridDim apart, the next one on its way
// while it computes.
struct PolyArgs {
  const void* z;
  const void* bias;    // [n]
  const float* coef;   // a, b, c, e
  void* out;
  long long rows;
  int n, ff;
  float eps;
};

// sums over the block, in every thread
__device__ __forceinline__ float3 block_sum3(float3 v, float* red) {
  v.x = warp_sum(v.x);
  v.y = warp_sum(v.y);
  v.z = warp_sum(v.z);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = (blockDim.x + 31) >> 5;
  if (lane == 0) {
    red[warp] = v.x;
    red[32 + warp] = v.y;
    red[64 + warp] = v.z;
  }
  __syncthreads();
  const bool in = lane < warps;
  return make_float3(warp_sum(in ? red[lane] : 0.f), warp_sum(in ? red[32 + lane] : 0.f),
                     warp_sum(in ? red[64 + lane] : 0.f));
}

// 16 bytes as pairs of floats, and back
__device__ __forceinline__ void widen16(const uint4& q, float2 (&f)[4]) {
  const uint32_t w[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
  for (int i = 0; i < 4; ++i)
    f[i] = make_float2(__uint_as_float(w[i] << 16), __uint_as_float(w[i] & 0xffff0000u));
}
__device__ __forceinline__ void widen16(const uint4& q, float2 (&f)[2]) {
  f[0] = make_float2(__uint_as_float(q.x), __uint_as_float(q.y));
  f[1] = make_float2(__uint_as_float(q.z), __uint_as_float(q.w));
}
__device__ __forceinline__ uint4 narrow16(const float2 (&f)[4]) {
  return make_uint4(pack_bf16x2(f[0].x, f[0].y), pack_bf16x2(f[1].x, f[1].y), pack_bf16x2(f[2].x, f[2].y),
                    pack_bf16x2(f[3].x, f[3].y));
}
__device__ __forceinline__ uint4 narrow16(const float2 (&f)[2]) {
  return make_uint4(__float_as_uint(f[0].x), __float_as_uint(f[0].y), __float_as_uint(f[1].x),
                    __float_as_uint(f[1].y));
}

// N: 16-byte pieces of the row a thread holds, widened; 0: any width and alignment, read twice
template <typename T, int N>
__global__ void __launch_bounds__(1024) poly_norm_kernel(const PolyArgs p) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[2][96];
  const T* z = reinterpret_cast<const T*>(p.z);
  const T* bias = reinterpret_cast<const T*>(p.bias);
  T* out = reinterpret_cast<T*>(p.out);
  const float rf = 1.f / (float)p.ff;
  const float ca = p.coef[0], cb = p.coef[1], cc = p.coef[2], e = p.coef[3];
  float fa = 0.f, fb = 0.f, fc = 0.f;
  int turn = 0;
  auto factors = [&](float3 s) {   // from the thread's sums of z^2, z^4, z^6
    s = block_sum3(s, red[turn]);  // (what the row before left is still being read)
    turn ^= 1;
    fa = ca / sqrtf(s.x * rf + p.eps);
    fb = cb / sqrtf(s.y * rf + p.eps);
    fc = cc / sqrtf(s.z * rf + p.eps);
  };
  if constexpr (N > 0) {
    constexpr int V = 16 / sizeof(T);
    uint4 raw[N];
    float2 v[N][V / 2];
    const float2 zero = make_float2(0.f, 0.f);
    auto fetch = [&](long long row) {
#pragma unroll
      for (int j = 0; j < N; ++j) {
        const int i = (threadIdx.x + j * blockDim.x) * V;
        raw[j] = make_uint4(0, 0, 0, 0);
        if (row < p.rows && i < p.n) raw[j] = *reinterpret_cast<const uint4*>(z + row * p.n + i);
      }
    };
    fetch(blockIdx.x);
    for (long long row = blockIdx.x; row < p.rows; row += gridDim.x) {
      float2 s2 = zero, s4 = zero, s6 = zero;
#pragma unroll
      for (int j = 0; j < N; ++j) {
        const int i = (threadIdx.x + j * blockDim.x) * V;
        widen16(raw[j], v[j]);
        if (i < p.n) {
          float2 w[V / 2];
          widen16(*reinterpret_cast<const uint4*>(bias + i), w);
#pragma unroll
          for (int k = 0; k < V / 2; ++k) add2(v[j][k], w[k]);
          if (i + V > p.ff) {   // the columns beyond count nothing
#pragma unroll
            for (int k = 0; k < V / 2; ++k) {
              if (i + 2 * k >= p.ff) v[j][k].x = 0.f;
              if (i + 2 * k + 1 >= p.ff) v[j][k].y = 0.f;
            }
          }
        }
#pragma unroll
        for (int k = 0; k < V / 2; ++k) {
          const float2 x = v[j][k];
          float2 q = x, r;
          fma2(s2, x, x);
          mul2(q, x);
          r = q;
          mul2(r, q);
          add2(s4, r);
          fma2(s6, r, q);
        }
      }
      fetch(row + gridDim.x);
      factors(make_float3(s2.x + s2.y, s4.x + s4.y, s6.x + s6.y));
      const float2 A = make_float2(fa, fa), B = make_float2(fb, fb), C = make_float2(fc, fc),
                   E = make_float2(e, e);
#pragma unroll
      for (int j = 0; j < N; ++j) {
        const int i = (threadIdx.x + j * blockDim.x) * V;
        if (i >= p.n) continue;
#pragma unroll
        for (int k = 0; k < V / 2; ++k) {   // ((c v + b) v + a) v + e
          float2 y = B, u = A, x = v[j][k];
          fma2(y, C, x);
          fma2(u, y, x);
          y = E;
          fma2(y, u, x);
          v[j][k] = y;
        }
        if (i + V > p.ff) {
#pragma unroll
          for (int k = 0; k < V / 2; ++k) {
            if (i + 2 * k >= p.ff) v[j][k].x = 0.f;
            if (i + 2 * k + 1 >= p.ff) v[j][k].y = 0.f;
          }
        }
        *reinterpret_cast<uint4*>(out + row * p.n + i) = narrow16(v[j]);
      }
    }
  } else {
    for (long long row = blockIdx.x; row < p.rows; row += gridDim.x) {
      const T* z_row = z + row * p.n;
      auto at = [&](int i) { return to_f32<T>(z_row[i]) + to_f32<T>(bias[i]); };
      float3 s = make_float3(0.f, 0.f, 0.f);
      for (int i = threadIdx.x; i < p.ff; i += blockDim.x) {
        const float x = at(i), q = x * x, r = q * q;
        s.x += q;
        s.y += r;
        s.z = fmaf(r, q, s.z);
      }
      factors(s);
      for (int i = threadIdx.x; i < p.n; i += blockDim.x) {
        const float x = i < p.ff ? at(i) : 0.f;
        out[row * p.n + i] = from_f32<T>(i < p.ff ? fmaf(x, fmaf(x, fmaf(x, fc, fb), fa), e) : 0.f);
      }
    }
  }
}

template <typename T>
static int launch_poly_norm(const PolyArgs& a, long long T_rows, cudaStream_t stream) {
  constexpr int V = 16 / sizeof(T);
  const bool vec = a.n % V == 0 &&
                   ((reinterpret_cast<uintptr_t>(a.z) | reinterpret_cast<uintptr_t>(a.bias) |
                     reinterpret_cast<uintptr_t>(a.out)) & 15) == 0;
  const int pieces = a.n / V;
  auto k = poly_norm_kernel<T, 0>;
  int threads = 512;
  if (vec && pieces <= 1024 * 4) {
    const int most = T_rows <= 148 ? 1 : 4;   // few rows: more threads on each
    threads = 64;
    while (threads < 1024 && pieces > threads * most) threads *= 2;
    const int per = (pieces + threads - 1) / threads;
    k = per <= 1   ? poly_norm_kernel<T, 1>
        : per <= 2 ? poly_norm_kernel<T, 2>
        : per <= 3 ? poly_norm_kernel<T, 3>
                   : poly_norm_kernel<T, 4>;
  }
  const long long blocks = 148 * (threads >= 1024 ? 1 : threads >= 512 ? 2 : 1024 / threads);
  return launch_pdl(k, dim3((unsigned)(T_rows < blocks ? T_rows : blocks)), dim3(threads), 0, stream, a) ==
                 cudaSuccess
             ? 0
             : -5;
}

template <typename T>
__global__ void __launch_bounds__(256)
soft_cap_kernel(const T* __restrict__ z, long long ld, float* __restrict__ out, int V, float cap, int vec) {
  pdl_wait();
  pdl_trigger();
  const long long t = blockIdx.y;
  const T* src = z + t * ld;
  float* dst = out + t * V;
  const float inv = 1.f / cap;
  const int at = blockIdx.x * blockDim.x + threadIdx.x, step = gridDim.x * blockDim.x;
  if (vec) {
    for (int i = at * 4; i < V; i += step * 4) {
      const float4 v = load4(src + i);
      store4(dst + i, make_float4(cap * tanhf(v.x * inv), cap * tanhf(v.y * inv), cap * tanhf(v.z * inv),
                                  cap * tanhf(v.w * inv)));
    }
  } else {
    for (int i = at; i < V; i += step) dst[i] = cap * tanhf(to_f32<T>(src[i]) * inv);
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
gated_act_kernel(const T* __restrict__ gu, T* __restrict__ out, long long n, int ff, int act,
                 const GateParams gp) {
  pdl_wait();
  pdl_trigger();
  // four outputs per thread: they share a block of kGateBlock
  for (long long i = (blockIdx.x * (long long)blockDim.x + threadIdx.x) * 4; i < n;
       i += (long long)gridDim.x * blockDim.x * 4) {
    const long long t = i / ff;
    const int c = (int)(i - t * ff);
    const T* g = gu + t * 2 * ff + (c / kGateBlock) * (2 * kGateBlock) + c % kGateBlock;
    const float4 a = load4(g), b = load4(g + kGateBlock);
    store4(out + i, make_float4(gated(act, gp, a.x, b.x), gated(act, gp, a.y, b.y),
                                gated(act, gp, a.z, b.z), gated(act, gp, a.w, b.w)));
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
// x fp32 [T, W] = table[ids] * scale, plus, with `prev` int64 [T], the row of `second` [buckets + 1, W]
// that (prev * mul_prev + id * mul_cur) mod buckets names (prev < 0: the last one). act (may be null): x in
// the element type; keep (may be null): another copy of x.
int ab200_stream_embedding(const void* ids, const void* table, void* x, void* act, void* keep, float scale,
                           long long T, int W, long long vocab, const void* prev, const void* second,
                           long long buckets, long long mul_prev, long long mul_cur, int dtype,
                           int* status, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (prev != nullptr && (second == nullptr || buckets < 1)) return -2;
  const PairArgs pairs = {reinterpret_cast<const long long*>(prev), second, buckets, mul_prev, mul_cur};
  cudaError_t e;
  if (dtype == 0)
    e = launch_pdl(stream_embedding_kernel<bf16>, dim3((unsigned)T), dim3(256), 0, stream,
                   reinterpret_cast<const long long*>(ids), reinterpret_cast<const bf16*>(table),
                   reinterpret_cast<float*>(x), reinterpret_cast<bf16*>(act),
                   reinterpret_cast<float*>(keep), scale, W, vocab, pairs, status);
  else
    e = launch_pdl(stream_embedding_kernel<float>, dim3((unsigned)T), dim3(256), 0, stream,
                   reinterpret_cast<const long long*>(ids), reinterpret_cast<const float*>(table),
                   reinterpret_cast<float*>(x), reinterpret_cast<float*>(act),
                   reinterpret_cast<float*>(keep), scale, W, vocab, pairs, status);
  return e == cudaSuccess ? 0 : -5;
}

// In place on x [T, W]: x += mult * f, where f is y + bias (bias may be null) or, with y_rows int32 and
// y_weights fp32 [T, top], the weighted sum of these rows of y, plus `shared`'s rows (may be null);
// x += base (fp32 [T, W]) and += step (fp32 [W]) if given; act = norm(x) * w_in if act. All may be null.
int ab200_stream_pre(void* x, const void* y, long long ldy, const void* bias, const void* y_rows,
                     const void* y_weights, int top, const void* shared, long long ld_shared,
                     float mult, const void* base, const void* step, const void* w_in, int w_scalar,
                     void* act, float eps, long long T, int W, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if ((y_rows != nullptr && (y_weights == nullptr || y == nullptr)) || (act != nullptr && w_in == nullptr) ||
      (y == nullptr && (bias != nullptr || shared != nullptr)))
    return -2;
  StreamPreArgs a;
  a.x = reinterpret_cast<float*>(x);
  a.y = y; a.ldy = ldy;
  a.bias = reinterpret_cast<const float*>(bias);
  a.y_rows = reinterpret_cast<const int*>(y_rows);
  a.y_weights = reinterpret_cast<const float*>(y_weights);
  a.top = top;
  a.shared = shared; a.ld_shared = ld_shared;
  a.mult = mult;
  a.base = reinterpret_cast<const float*>(base);
  a.step = reinterpret_cast<const float*>(step);
  a.w_in = reinterpret_cast<const float*>(w_in);
  a.w_scalar = w_scalar && w_in != nullptr;
  a.act = act;
  a.eps = eps;
  a.W = W;
  return dtype == 0 ? launch_stream_pre<bf16>(a, T, stream) : launch_stream_pre<float>(a, T, stream);
}

// z, out [T, n] (element type by dtype), of whose columns the first ff count (the others become zero):
// a N(z') + b N(z'^2) + c N(z'^3) + e with z' = z + bias; bias [n], coef fp32 [4] (a, b, c, e)
int ab200_poly_norm(const void* z, const void* bias, const void* coef, void* out, long long T, int n,
                    int ff, float eps, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (ff < 1 || ff > n) return -2;
  const PolyArgs a = {z, bias, reinterpret_cast<const float*>(coef), out, T, n, ff, eps};
  return dtype == 0 ? launch_poly_norm<bf16>(a, T, stream) : launch_poly_norm<float>(a, T, stream);
}

// out fp32 [T, V] = cap * tanh(z / cap), z [T, ld]
int ab200_soft_cap(const void* z, long long ld, void* out, long long T, int V, float cap, int dtype,
                   cudaStream_t stream) {
  if (T <= 0 || V <= 0) return 0;
  if (!(cap > 0.f) || T > 65535) return -2;
  const int vec = V % 4 == 0 && ld % 4 == 0 &&
                  ((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
  const int per = (V + 1023) / 1024;
  const dim3 grid((unsigned)(per < 64 ? per : 64), (unsigned)T);
  const cudaError_t e =
      dtype == 0 ? launch_pdl(soft_cap_kernel<bf16>, grid, dim3(256), 0, stream,
                              reinterpret_cast<const bf16*>(z), ld, reinterpret_cast<float*>(out), V, cap, vec)
                 : launch_pdl(soft_cap_kernel<float>, grid, dim3(256), 0, stream,
                              reinterpret_cast<const float*>(z), ld, reinterpret_cast<float*>(out), V, cap, vec);
  return e == cudaSuccess ? 0 : -5;
}

// out rows t < T: norm(alpha * x[rows ? rows[t] : t] + y[t]) * (offset + weight). x_out may be x itself
// when rows is null (each block owns its row).
int ab200_stream_norm(const void* x, const void* rows, const void* y, long long ldy,
                      const void* y_rows, const void* y_weights, int top, const void* weight,
                      float alpha, float eps, float offset, void* x_out, void* act_out,
                      long long T, int W, int dtype, cudaStream_t stream) {
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
  a.offset = offset;
  a.x_out = reinterpret_cast<float*>(x_out);
  a.act_out = act_out;
  a.W = W;
  return dtype == 0 ? launch_stream_norm<bf16>(a, T, stream) : launch_stream_norm<float>(a, T, stream);
}

// In place on x [T, W]: x += norm(y) * (offset + w_out) if y, += step if step; act = norm(x) *
// (offset + w_in) if act.
int ab200_stream_sandwich(void* x, const void* y, long long ldy, const void* w_out, const void* step,
                          const void* w_in, void* act, float eps, float offset, long long T, int W,
                          int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if ((y != nullptr && w_out == nullptr) || (act != nullptr && w_in == nullptr)) return -2;
  SandwichArgs a;
  a.x = reinterpret_cast<float*>(x);
  a.y = y;
  a.ldy = ldy;
  a.w_out = reinterpret_cast<const float*>(w_out);
  a.step = reinterpret_cast<const float*>(step);
  a.w_in = reinterpret_cast<const float*>(w_in);
  a.act = act;
  a.eps = eps;
  a.offset = offset;
  a.W = W;
  return dtype == 0 ? launch_stream_sandwich<bf16>(a, T, stream)
                    : launch_stream_sandwich<float>(a, T, stream);
}

// In place on x [T, W]: x += norm(y) * w; act (may be null): the new x. y: rows of a sublayer's output;
// with y2: half of norm(y) * wy + norm(y2) * wy2; with y_rows int32 and y_weights fp32 [T, top]: the
// weighted sum of these rows (row -1: the token's own x, before the update) plus `shared`'s (may be null).
int ab200_stream_add(void* x, void* act, const void* w, const void* y, long long ldy, const void* wy,
                     const void* y2, long long ldy2, const void* wy2, const void* y_rows,
                     const void* y_weights, int top, const void* shared, long long ld_shared,
                     float eps, long long T, int W, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if ((y2 != nullptr && (wy == nullptr || wy2 == nullptr)) ||
      (y_rows != nullptr && (y_weights == nullptr || y2 != nullptr)))
    return -2;
  StreamAddArgs a;
  a.x = reinterpret_cast<float*>(x);
  a.act = act;
  a.w = reinterpret_cast<const float*>(w);
  a.y = y; a.ldy = ldy;
  a.wy = reinterpret_cast<const float*>(wy);
  a.y2 = y2; a.ldy2 = ldy2;
  a.wy2 = reinterpret_cast<const float*>(wy2);
  a.y_rows = reinterpret_cast<const int*>(y_rows);
  a.y_weights = reinterpret_cast<const float*>(y_weights);
  a.top = top;
  a.shared = shared; a.ld_shared = ld_shared;
  a.eps = eps;
  a.W = W;
  return dtype == 0 ? launch_stream_add<bf16>(a, T, stream) : launch_stream_add<float>(a, T, stream);
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
int ab200_gated_act(const void* gu, void* out, long long T, int ff, int act, float limit,
                    float alpha, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (ff % kGateBlock || act < kActSilu || act > kActClampedSwish) return -2;
  const GateParams gp = {limit, alpha};
  const long long n = T * ff;
  long long blocks = (n / 4 + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  cudaError_t e;
  if (dtype == 0)
    e = launch_pdl(gated_act_kernel<bf16>, dim3((unsigned)blocks), dim3(256), 0, stream,
                   reinterpret_cast<const bf16*>(gu), reinterpret_cast<bf16*>(out), n, ff, act, gp);
  else
    e = launch_pdl(gated_act_kernel<float>, dim3((unsigned)blocks), dim3(256), 0, stream,
                   reinterpret_cast<const float*>(gu), reinterpret_cast<float*>(out), n, ff, act, gp);
  return e == cudaSuccess ? 0 : -5;
}

}  // extern "C"
