// Mixture-of-experts routing, all on the device (no host round trip, so decode steps stay
// capturable):
//
//   moe_route    fp32 router logits x * W^T + b (a block keeps a few tokens' rows in shared
//                memory, so router weights are read once per block), the `top` largest per token
//                and the softmax over those
//   moe_plan     rows per expert, each expert's first row among the rows sorted by expert, and
//                the list of 128-row tiles the grouped matrix products walk
//   moe_permute  row of every (token, choice) and the copy of the token's activations there
//
// The weighted sum of the experts' outputs is taken by the norm kernel that follows (stream.cu).

#include <float.h>

#include "api.h"
#include "common/elem.cuh"
#include "common/pdl.cuh"

namespace ab200 {

constexpr int kRouteThreads = 256;
constexpr int kTileRows = 128;

// Router weights of type T; TB tokens per block. Shared memory: x rows [TB][W], logits [TB][E].
template <typename T, int TB>
__global__ void __launch_bounds__(kRouteThreads)
moe_route_kernel(const float* __restrict__ x, const T* __restrict__ w, const float* __restrict__ b,
                 long long n, int W, int E, int top, int* __restrict__ ids,
                 float* __restrict__ weights) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(16) float sm[];
  float* xs = sm;
  float* z = sm + (size_t)TB * W;
  const long long t0 = (long long)blockIdx.x * TB;
  const int nt = (int)min((long long)TB, n - t0);
  for (int i = threadIdx.x; i < TB * W; i += kRouteThreads)
    xs[i] = i / W < nt ? x[t0 * W + i] : 0.f;
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  constexpr int EB = 4;   // experts a warp takes at a time
  for (int e0 = warp * EB; e0 < E; e0 += (kRouteThreads / 32) * EB) {
    float acc[TB][EB];
#pragma unroll
    for (int t = 0; t < TB; ++t)
#pragma unroll
      for (int j = 0; j < EB; ++j) acc[t][j] = 0.f;
    for (int i = lane; i < W; i += 32) {
      float wv[EB];
#pragma unroll
      for (int j = 0; j < EB; ++j)
        wv[j] = e0 + j < E ? to_f32<T>(w[(long long)(e0 + j) * W + i]) : 0.f;
#pragma unroll
      for (int t = 0; t < TB; ++t) {
        const float xv = xs[t * W + i];
#pragma unroll
        for (int j = 0; j < EB; ++j) acc[t][j] = fmaf(xv, wv[j], acc[t][j]);
      }
    }
#pragma unroll
    for (int t = 0; t < TB; ++t)
#pragma unroll
      for (int j = 0; j < EB; ++j) {
        const float s = warp_sum(acc[t][j]);
        if (lane == 0 && e0 + j < E) z[t * E + e0 + j] = s + b[e0 + j];
      }
  }
  __syncthreads();
  // a warp per token picks the largest logit `top` times (ties: the lower expert)
  for (int t = warp; t < nt; t += kRouteThreads / 32) {
    float* zt = z + t * E;
    float first = 0.f, sum = 0.f;
    int* my_ids = ids + (t0 + t) * top;
    float* my_w = weights + (t0 + t) * top;
    for (int j = 0; j < top; ++j) {
      float best = -INFINITY;
      int bi = 0x7fffffff;
      for (int e = lane; e < E; e += 32) {
        const float v = zt[e];
        if (v > best || bi == 0x7fffffff) {
          best = v;
          bi = e;
        }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, best, o);
        const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
        if (ov > best || (ov == best && oi < bi)) {
          best = ov;
          bi = oi;
        }
      }
      bi = min(bi, E - 1);   // (a row of NaNs must still name an expert)
      if (j == 0) first = best;
      const float ex = expf(best - first);
      sum += ex;
      if (lane == 0) {
        my_ids[j] = bi;
        my_w[j] = ex;
        zt[bi] = -INFINITY;
      }
      __syncwarp();
    }
    const float inv = 1.f / sum;
    for (int j = lane; j < top; j += 32) my_w[j] *= inv;
  }
}

// One block. Rows per expert -> first rows (cursor), 128-row tiles.
__global__ void __launch_bounds__(1024)
moe_plan_kernel(const int* __restrict__ ids, long long n, int E, int* __restrict__ cursor,
                int4* __restrict__ tiles, int* __restrict__ num_tiles) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ int sh[];
  int* count = sh;            // [E]
  int* first = sh + E;        // [E]
  int* tile0 = sh + 2 * E;    // [E]
  for (int e = threadIdx.x; e < E; e += blockDim.x) count[e] = 0;
  __syncthreads();
  for (long long i = threadIdx.x; i < n; i += blockDim.x) atomicAdd(&count[ids[i]], 1);
  __syncthreads();
  if (threadIdx.x < 32) {
    int row = 0, tile = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + threadIdx.x;
      const int c = e < E ? count[e] : 0;
      const int k = (c + kTileRows - 1) / kTileRows;
      int rs = c, ts = k;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int a = __shfl_up_sync(0xffffffffu, rs, o);
        const int d = __shfl_up_sync(0xffffffffu, ts, o);
        if ((int)threadIdx.x >= o) {
          rs += a;
          ts += d;
        }
      }
      if (e < E) {
        first[e] = row + rs - c;
        tile0[e] = tile + ts - k;
      }
      row += __shfl_sync(0xffffffffu, rs, 31);
      tile += __shfl_sync(0xffffffffu, ts, 31);
    }
    if (threadIdx.x == 0) *num_tiles = tile;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) {
    cursor[e] = first[e];
    for (int r = 0, k = 0; r < count[e]; r += kTileRows, ++k)
      tiles[tile0[e] + k] = make_int4(e, first[e] + r, min(kTileRows, count[e] - r), 0);
  }
}

// A block per (token, choice): takes the next row of its expert and copies the activations.
template <typename T>
__global__ void __launch_bounds__(128)
moe_permute_kernel(const T* __restrict__ x, const int* __restrict__ ids, int* __restrict__ cursor,
                   int* __restrict__ rows, T* __restrict__ xp, int W, int top) {
  pdl_wait();
  pdl_trigger();
  __shared__ int row;
  const long long i = blockIdx.x;
  if (threadIdx.x == 0) {
    row = atomicAdd(&cursor[ids[i]], 1);
    rows[i] = row;
  }
  __syncthreads();
  const T* src = x + (i / top) * W;
  T* dst = xp + (long long)row * W;
  constexpr int V = 16 / sizeof(T);
  if (W % V == 0) {
    for (int c = threadIdx.x; c < W / V; c += blockDim.x)
      reinterpret_cast<uint4*>(dst)[c] = reinterpret_cast<const uint4*>(src)[c];
  } else {
    for (int c = threadIdx.x; c < W; c += blockDim.x) dst[c] = src[c];
  }
}

template <typename T, int TB>
static int launch_route(const void* x, const void* w, const void* b, long long n, int W, int E,
                        int top, void* ids, void* weights, cudaStream_t stream) {
  const size_t smem = ((size_t)TB * W + (size_t)TB * E) * sizeof(float);
  if (smem > 220 * 1024) return -6;
  auto k = moe_route_kernel<T, TB>;
  if (smem > 48 * 1024 &&
      cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return -3;
  return launch_pdl(k, dim3((unsigned)((n + TB - 1) / TB)), dim3(kRouteThreads), smem, stream,
                    reinterpret_cast<const float*>(x), reinterpret_cast<const T*>(w),
                    reinterpret_cast<const float*>(b), n, W, E, top, reinterpret_cast<int*>(ids),
                    reinterpret_cast<float*>(weights)) == cudaSuccess
             ? 0
             : -5;
}

}  // namespace ab200

using namespace ab200;
typedef __nv_bfloat16 bf16;

extern "C" {

// x fp32 [T, W]; w [E, W] (dtype 0 = bf16, 1 = fp32); b fp32 [E]; ids int32 and weights fp32 [T, top]
int ab200_moe_route(const void* x, const void* w, const void* b, long long T, int W, int E, int top,
                    void* ids, void* weights, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (top < 1 || top > E) return -2;
  // many tokens: several per block, so that the router's weights are read less often
  const bool wide = T >= 148 * 8 && (size_t)8 * (W + E) * 4 <= 110 * 1024;
  if (dtype == 0)
    return wide ? launch_route<bf16, 8>(x, w, b, T, W, E, top, ids, weights, stream)
                : launch_route<bf16, 1>(x, w, b, T, W, E, top, ids, weights, stream);
  return wide ? launch_route<float, 8>(x, w, b, T, W, E, top, ids, weights, stream)
              : launch_route<float, 1>(x, w, b, T, W, E, top, ids, weights, stream);
}

// ids int32 [n]; cursor int32 [E]; tiles int32 x 4 [n / 128 + E at most]; num_tiles int32 [1]
int ab200_moe_plan(const void* ids, long long n, int E, void* cursor, void* tiles, void* num_tiles,
                   cudaStream_t stream) {
  if (E <= 0 || E > 4096) return -6;
  return launch_pdl(moe_plan_kernel, dim3(1), dim3(1024), (size_t)3 * E * sizeof(int), stream,
                    reinterpret_cast<const int*>(ids), n, E, reinterpret_cast<int*>(cursor),
                    reinterpret_cast<int4*>(tiles), reinterpret_cast<int*>(num_tiles)) == cudaSuccess
             ? 0
             : -5;
}

int ab200_moe_permute(const void* x, const void* ids, void* cursor, void* rows, void* xp,
                      long long T, int W, int top, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  const dim3 grid((unsigned)(T * top));
  const cudaError_t e =
      dtype == 0
          ? launch_pdl(moe_permute_kernel<bf16>, grid, dim3(128), 0, stream,
                       reinterpret_cast<const bf16*>(x), reinterpret_cast<const int*>(ids),
                       reinterpret_cast<int*>(cursor), reinterpret_cast<int*>(rows),
                       reinterpret_cast<bf16*>(xp), W, top)
          : launch_pdl(moe_permute_kernel<float>, grid, dim3(128), 0, stream,
                       reinterpret_cast<const float*>(x), reinterpret_cast<const int*>(ids),
                       reinterpret_cast<int*>(cursor), reinterpret_cast<int*>(rows),
                       reinterpret_cast<float*>(xp), W, top);
  return e == cudaSuccess ? 0 : -5;
}

}  // extern "C"
