// Mixture-of-experts routing, all on the device (no host round trip, so decode steps stay
// capturable):
//
//   moe_route    fp32 router logits x * W^T + b (a block keeps a few tokens' rows in shared
//                memory, so router weights are read once per block), the `top` largest per token
//                and the softmax over those; rows per expert are counted on the way, and the
//                block that finishes last turns the counts into each expert's first row among
//                the rows sorted by expert and into the list of 128-row tiles the grouped matrix
//                products walk. Or, scoring over all outputs: the softmax over all of them, the
//                choice by score plus a correction, the chosen scores times a scale as weights;
//                outputs beyond the experts are identity experts, which get no rows. Or sigmoid
//                scores: the choice among the experts of the best groups of neighbours (by the sum
//                of a group's two best), the chosen scores normalised to the sum `scale`
//   moe_permute  row of every (token, choice) and the copy of the token's activations there
//
// The weighted sum of the experts' outputs is taken by the norm kernel that follows (stream.cu).

#include <float.h>

#include <type_traits>

#include "api.h"
#include "common/elem.cuh"
#include "common/pdl.cuh"

namespace ab200 {

constexpr int kTileRows = 128;

// Four elements as they lie in memory, widened when they are used.
template <typename T>
struct Raw4;
template <>
struct Raw4<float> {
  float4 q;
  __device__ __forceinline__ void load(const float* p) { q = load4(p); }
  __device__ __forceinline__ float4 get() const { return q; }
};
template <>
struct Raw4<__nv_bfloat16> {
  uint2 q;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { q = *reinterpret_cast<const uint2*>(p); }
  __device__ __forceinline__ float4 get() const {
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.y));
    return make_float4(a.x, a.y, b.x, b.y);
  }
};

enum RouteMode : int { kRouteChosen = 0, kRouteAll = 1, kRouteSigmoid = 2 };

struct RouteArgs {
  const void* x;       // [n][W]: fp32, or (x_act) in the router weights' element type
  int x_act;
  const void* w;       // [E][W]
  const float* b;      // [E] bias of the logits, or correction of the choice; may be null
  long long n;
  int W, E, top;       // E: router outputs
  int experts;         // of them the experts' (the others: identity)
  int mode;            // RouteMode: softmax over the chosen logits or over all, or sigmoids
  float scale;         // of the weights (all), their sum (sigmoids)
  int groups, keep;    // sigmoids: equal groups of experts, how many of them can be chosen from
  int* ids;            // [n][top]
  float* weights;      // [n][top]
  int* state;          // [E] counts and [1] finished blocks; zero before and after every launch
  int* cursor;         // [E] first row of each expert
  int4* tiles;
  int* num_tiles;
};

// Run by the last block: counts -> first rows and tiles; leaves the counts at zero.
__device__ void moe_plan(const RouteArgs& p, int* sh) {
  const int E = p.experts;
  int* count = sh;            // [E]
  int* first = sh + E;        // [E]
  int* tile0 = sh + 2 * E;    // [E]
  for (int e = threadIdx.x; e < E; e += blockDim.x) {
    count[e] = __ldcg(p.state + e);
    p.state[e] = 0;
  }
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
    if (threadIdx.x == 0) *p.num_tiles = tile;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) {
    p.cursor[e] = first[e];
    for (int r = 0, k = 0; r < count[e]; r += kTileRows, ++k)
      p.tiles[tile0[e] + k] = make_int4(e, first[e] + r, min(kTileRows, count[e] - r), 0);
  }
}

// The largest of n values (ties, NaNs: the lower index), by a warp; `best` its value
__device__ __forceinline__ int warp_argmax(const float* v, int n, float& best) {
  const int lane = threadIdx.x & 31;
  best = -INFINITY;
  int bi = 0x7fffffff;
  for (int e = lane; e < n; e += 32)
    if (v[e] > best || bi == 0x7fffffff) {
      best = v[e];
      bi = e;
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
  return min(bi, n - 1);   // (a row of NaNs must still name one)
}

// Router weights of type T; TB tokens per block. Shared memory: x rows [TB][W], logits [TB][E],
// at least 3 * E words for the plan.
template <typename T, int TB, int kRouteThreads>
__global__ void __launch_bounds__(kRouteThreads) moe_route_kernel(const RouteArgs p) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(16) float sm[];
  __shared__ int last;
  const int W = p.W, E = p.E, top = p.top;
  float* xs = sm;
  float* z = sm + (size_t)TB * W;
  const T* w = reinterpret_cast<const T*>(p.w);
  const long long t0 = (long long)blockIdx.x * TB;
  const int nt = (int)min((long long)TB, p.n - t0);
  const bool vec = W % 4 == 0;
  auto fill = [&](const auto* x) {
    typedef typename std::remove_const<typename std::remove_pointer<decltype(x)>::type>::type X;
    if (vec) {
      for (int i = threadIdx.x * 4; i < TB * W; i += kRouteThreads * 4)
        store4(xs + i, i / W < nt ? load4(x + t0 * W + i) : make_float4(0.f, 0.f, 0.f, 0.f));
    } else {
      for (int i = threadIdx.x; i < TB * W; i += kRouteThreads)
        xs[i] = i / W < nt ? to_f32<X>(x[t0 * W + i]) : 0.f;
    }
  };
  if (p.x_act) fill(reinterpret_cast<const T*>(p.x));
  else fill(reinterpret_cast<const float*>(p.x));
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  constexpr int EB = 4;   // experts a warp takes at a time
  for (int e0 = warp * EB; e0 < E; e0 += (kRouteThreads / 32) * EB) {
    float acc[TB][EB];
#pragma unroll
    for (int t = 0; t < TB; ++t)
#pragma unroll
      for (int j = 0; j < EB; ++j) acc[t][j] = 0.f;
    if (vec) {
      // Two pieces of four consecutive elements per lane and step (conflict-free in shared
      // memory); the next step's weights are on their way while this one's are multiplied.
      const T* we[EB];
#pragma unroll
      for (int j = 0; j < EB; ++j) we[j] = w + (long long)min(e0 + j, E - 1) * W;
      Raw4<T> nxt[EB][2];
      auto fetch = [&](int i) {
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int k = min(i + 128 * h, W - 4);
#pragma unroll
          for (int j = 0; j < EB; ++j) nxt[j][h].load(we[j] + k);
        }
      };
      fetch(lane * 4);
      for (int i = lane * 4; i < W; i += 256) {
        float4 wv[2][EB];
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int j = 0; j < EB; ++j) wv[h][j] = nxt[j][h].get();
        fetch(i + 256);
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          if (i + 128 * h >= W) break;
#pragma unroll
          for (int t = 0; t < TB; ++t) {
            const float4 xv = load4(xs + t * W + i + 128 * h);
#pragma unroll
            for (int j = 0; j < EB; ++j) {
              acc[t][j] = fmaf(xv.x, wv[h][j].x, acc[t][j]);
              acc[t][j] = fmaf(xv.y, wv[h][j].y, acc[t][j]);
              acc[t][j] = fmaf(xv.z, wv[h][j].z, acc[t][j]);
              acc[t][j] = fmaf(xv.w, wv[h][j].w, acc[t][j]);
            }
          }
        }
      }
    } else {
      for (int i = lane; i < W; i += 32) {
#pragma unroll
        for (int j = 0; j < EB; ++j) {
          const float wv = to_f32<T>(w[(long long)min(e0 + j, E - 1) * W + i]);
#pragma unroll
          for (int t = 0; t < TB; ++t) acc[t][j] = fmaf(xs[t * W + i], wv, acc[t][j]);
        }
      }
    }
#pragma unroll
    for (int t = 0; t < TB; ++t)
#pragma unroll
      for (int j = 0; j < EB; ++j) {
        const float s = warp_sum(acc[t][j]);
        if (lane == 0 && e0 + j < E)
          z[t * E + e0 + j] = p.b != nullptr && p.mode == kRouteChosen ? s + p.b[e0 + j] : s;
      }
  }
  __syncthreads();
  // a warp per token picks the largest logit `top` times (ties: the lower expert)
  for (int t = warp; t < nt; t += kRouteThreads / 32) {
    float* zt = z + t * E;
    float first = 0.f, sum = 0.f;
    if (p.mode == kRouteSigmoid) {
      for (int e = lane; e < E; e += 32) zt[e] = 1.f / (1.f + expf(-zt[e]));
      __syncwarp();
      if (p.keep < p.groups) {
        float* gs = zt + E * TB;   // scores of the groups, -inf once kept
        const int size = E / p.groups;
        for (int g = lane; g < p.groups; g += 32) {
          float a = -INFINITY, b = -INFINITY;   // the two best
          for (int e = g * size; e < (g + 1) * size; ++e) {
            b = fmaxf(b, fminf(a, zt[e]));
            a = fmaxf(a, zt[e]);
          }
          gs[g] = size > 1 ? a + b : a;
        }
        __syncwarp();
        for (int k = 0; k < p.keep; ++k) {
          float best;
          const int g = warp_argmax(gs, p.groups, best);
          __syncwarp();
          if (lane == 0) gs[g] = -INFINITY;
          __syncwarp();
        }
        for (int e = lane; e < E; e += 32)
          if (gs[e / size] != -INFINITY) zt[e] = -INFINITY;
        __syncwarp();
      }
    }
    if (p.mode == kRouteAll) {   // logits -> scores plus correction
      float mx = -INFINITY;
      for (int e = lane; e < E; e += 32) mx = fmaxf(mx, zt[e]);
      mx = warp_max(mx);
      for (int e = lane; e < E; e += 32) {
        const float ex = expf(zt[e] - mx);
        sum += ex;
        zt[e] = ex;
      }
      const float inv = 1.f / warp_sum(sum);
      for (int e = lane; e < E; e += 32) {
        zt[E * TB + e] = zt[e] * inv;
        zt[e] = zt[e] * inv + (p.b != nullptr ? p.b[e] : 0.f);
      }
      __syncwarp();
    }
    int* my_ids = p.ids + (t0 + t) * top;
    float* my_w = p.weights + (t0 + t) * top;
    for (int j = 0; j < top; ++j) {
      float best;
      const int bi = warp_argmax(zt, E, best);
      if (j == 0) first = best;
      const float ex = p.mode == kRouteAll       ? zt[E * TB + bi] * p.scale
                       : p.mode == kRouteSigmoid ? best
                                                 : expf(best - first);
      sum += ex;
      __syncwarp();
      if (lane == 0) {
        my_ids[j] = bi;
        my_w[j] = ex;
        zt[bi] = -INFINITY;
        if (bi < p.experts) atomicAdd(p.state + bi, 1);
      }
      __syncwarp();
    }
    if (p.mode == kRouteAll) continue;
    const float inv = p.mode == kRouteSigmoid ? p.scale / (sum + 1e-20f) : 1.f / sum;
    for (int j = lane; j < top; j += 32) my_w[j] *= inv;
  }
  // every block counts itself done after its counts are visible; the last one plans
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    last = atomicAdd(p.state + p.experts, 1) == (int)gridDim.x - 1;
    if (last) p.state[p.experts] = 0;
  }
  __syncthreads();
  if (last) {
    __threadfence();
    moe_plan(p, reinterpret_cast<int*>(sm));
  }
}

// A block per token: takes the next row of each of its experts and copies the activations there.
template <typename T>
__global__ void __launch_bounds__(256)
moe_permute_kernel(const T* __restrict__ x, const int* __restrict__ ids, int* __restrict__ cursor,
                   int* __restrict__ rows, T* __restrict__ xp, int W, int top, int experts) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ int row[];
  const long long t = blockIdx.x;
  for (int j = threadIdx.x; j < top; j += blockDim.x) {
    const int e = ids[t * top + j];
    row[j] = e < experts ? atomicAdd(&cursor[e], 1) : -1;   // (an identity expert has no rows)
    rows[t * top + j] = row[j];
  }
  __syncthreads();
  const T* src = x + t * W;
  constexpr int V = 16 / sizeof(T);
  if (W % V == 0) {
    for (int c = threadIdx.x; c < W / V; c += blockDim.x) {
      const uint4 v = reinterpret_cast<const uint4*>(src)[c];
      for (int j = 0; j < top; ++j)
        if (row[j] >= 0) reinterpret_cast<uint4*>(xp + (long long)row[j] * W)[c] = v;
    }
  } else {
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
      const T v = src[c];
      for (int j = 0; j < top; ++j)
        if (row[j] >= 0) xp[(long long)row[j] * W + c] = v;
    }
  }
}

template <typename T, int TB>
static int launch_route(const RouteArgs& a, cudaStream_t stream) {
  size_t smem = ((size_t)TB * a.W + (size_t)TB * a.E * (a.mode == kRouteChosen ? 1 : 2)) * sizeof(float);
  if (smem < (size_t)3 * a.E * sizeof(int)) smem = (size_t)3 * a.E * sizeof(int);
  if (smem > 220 * 1024) return -6;
  // few tokens: more warps per block, so that each has few experts to go through
  constexpr int kRouteThreads = TB == 1 ? 512 : 256;
  auto k = moe_route_kernel<T, TB, kRouteThreads>;
  if (smem > 48 * 1024 &&
      cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return -3;
  return launch_pdl(k, dim3((unsigned)((a.n + TB - 1) / TB)), dim3(kRouteThreads), smem, stream,
                    a) == cudaSuccess
             ? 0
             : -5;
}

}  // namespace ab200

using namespace ab200;
typedef __nv_bfloat16 bf16;

extern "C" {

// x [T, W] (x_dtype 0 = bf16, 1 = fp32: fp32, or what w has); w [E, W] (dtype likewise); b fp32 [E] or
// null; the first `experts` of the E outputs are experts, the others the identity; mode, scale, groups,
// keep: see RouteArgs. ids int32 and weights fp32
// [T, top]; state int32 [experts + 1], zero; cursor int32 [experts]; tiles int32 x 4 [T * top / 128 +
// experts at most]; num_tiles int32 [1]
int ab200_moe_route(const void* x, int x_dtype, const void* w, const void* b, long long T, int W, int E,
                    int experts, int top, int mode, float scale, int groups, int keep, void* ids,
                    void* weights, void* state, void* cursor, void* tiles, void* num_tiles, int dtype,
                    cudaStream_t stream) {
  if (T <= 0) return 0;
  if (top < 1 || top > E || experts < 1 || experts > E) return -2;
  if (mode < kRouteChosen || mode > kRouteSigmoid || (x_dtype != 1 && x_dtype != dtype)) return -2;
  if (mode == kRouteSigmoid && (groups < 1 || E % groups || keep < 1 || keep > groups ||
                                top > keep * (E / groups) || experts != E || b != nullptr))
    return -2;
  RouteArgs a;
  a.x = x;
  a.x_act = x_dtype != 1;
  a.w = w;
  a.b = reinterpret_cast<const float*>(b);
  a.n = T;
  a.W = W;
  a.E = E;
  a.top = top;
  a.experts = experts;
  a.mode = mode;
  a.scale = scale;
  a.groups = groups;
  a.keep = keep;
  a.ids = reinterpret_cast<int*>(ids);
  a.weights = reinterpret_cast<float*>(weights);
  a.state = reinterpret_cast<int*>(state);
  a.cursor = reinterpret_cast<int*>(cursor);
  a.tiles = reinterpret_cast<int4*>(tiles);
  a.num_tiles = reinterpret_cast<int*>(num_tiles);
  // many tokens: several per block, so that the router's weights are read less often
  const bool wide = T >= 148 * 8 && (size_t)8 * (W + E) * 4 <= 110 * 1024;
  if (dtype == 0) return wide ? launch_route<bf16, 8>(a, stream) : launch_route<bf16, 1>(a, stream);
  return wide ? launch_route<float, 8>(a, stream) : launch_route<float, 1>(a, stream);
}

int ab200_moe_permute(const void* x, const void* ids, void* cursor, void* rows, void* xp,
                      long long T, int W, int top, int experts, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  const size_t smem = (size_t)top * sizeof(int);
  const cudaError_t e =
      dtype == 0
          ? launch_pdl(moe_permute_kernel<bf16>, dim3((unsigned)T), dim3(256), smem, stream,
                       reinterpret_cast<const bf16*>(x), reinterpret_cast<const int*>(ids),
                       reinterpret_cast<int*>(cursor), reinterpret_cast<int*>(rows),
                       reinterpret_cast<bf16*>(xp), W, top, experts)
          : launch_pdl(moe_permute_kernel<float>, dim3((unsigned)T), dim3(256), smem, stream,
                       reinterpret_cast<const float*>(x), reinterpret_cast<const int*>(ids),
                       reinterpret_cast<int*>(cursor), reinterpret_cast<int*>(rows),
                       reinterpret_cast<float*>(xp), W, top, experts);
  return e == cudaSuccess ? 0 : -5;
}

}  // extern "C"
