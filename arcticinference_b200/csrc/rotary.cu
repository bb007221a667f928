// What lies between an attention layer's input projection and its scores, for layers with
// partial rotary positions:
//
//   rotary_table       cosine and sine of every token's angles (angle = position * frequency in
//                      fp32), once per step for all layers with the same frequencies
//   head_rope_cache    RMS norm of queries and keys (optional; per head, or over all query and all
//                      key heads of a token at once), rotation of their first rot dimensions,
//                      queries in place, keys and values to the paged cache; the values may be
//                      the raw keys
//   latent_rope_cache  RMS norm of a compressed K/V projection and rotation of the key part that
//                      the heads share, both to the paged latent cache; rotation of every query
//                      head's rotary part in place
//
// A block owns a token and its warps walk the heads; norms and rotations are fp32. Pairs are
// (i, i + rot / 2). Heads of 64 or 128 bf16 columns stay in registers, four columns a lane
// and several heads in flight; a pair's other half then comes from another lane.
// T is the model's element type (bf16 or fp32).

#include "api.h"
#include "common/elem.cuh"
#include "common/pdl.cuh"

namespace ab200 {

constexpr int kRopeThreads = 256;

__global__ void __launch_bounds__(256)
rotary_table_kernel(const long long* __restrict__ positions, const float* __restrict__ freq,
                    float2* __restrict__ table, int half, long long n) {
  pdl_wait();
  pdl_trigger();
  const long long k = blockIdx.x * (long long)blockDim.x + threadIdx.x;
  if (k >= n) return;
  const long long t = k / half;
  float s, c;
  sincosf((float)positions[t] * freq[k - t * half], &s, &c);
  table[k] = make_float2(c, s);
}

// cs[2 * i], cs[2 * i + 1]: cosine and sine of pair i
__device__ __forceinline__ float rotated(const float* row, const float* cs, int half, int i) {
  if (i < half) return row[i] * cs[2 * i] - row[i + half] * cs[2 * i + 1];
  if (i < 2 * half) return row[i] * cs[2 * (i - half)] + row[i - half] * cs[2 * (i - half) + 1];
  return row[i];
}

struct HeadRopeArgs {
  void* proj;               // [T][ld]: Hq query heads, Hkv key heads of D, Hkv value heads of Dv
  long long ld;
  const float* table;       // [T][half][2]
  const long long* slots;
  const float* wq;          // [D], with `whole` [Hq * D]; null: no norm
  const float* wk;
  int whole;                // the norm's mean is over all heads' columns
  int shared_kv;            // no value heads in proj: the unnormed, unrotated keys are the values
  void* k_cache;            // [num_blocks][Hkv][block_size][D]
  void* v_cache;            // [num_blocks][Hkv][block_size][Dv]
  long long num_slots;
  int Hq, Hkv, D, Dv, half, block_size;
  float rdim, rdim_k, eps;  // 1 / (dimensions the norm's mean is over; columns beyond are zero)
  int* status;
};

// Sums of the squares of a token's query and key columns, for norms over the whole projection.
template <typename T>
__device__ __forceinline__ float2 projection_squares(const T* base, int nq, int nk, bool vec) {
  __shared__ float red[2][32];
  float q = 0.f, k = 0.f;
  if (vec) {
    for (int i = threadIdx.x * 4; i < nq + nk; i += kRopeThreads * 4) {
      const float4 v = load4(base + i);
      const float s = v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
      if (i < nq) q += s;
      else k += s;
    }
  } else {
    for (int i = threadIdx.x; i < nq + nk; i += kRopeThreads) {
      const float v = to_f32<T>(base[i]);
      if (i < nq) q += v * v;
      else k += v * v;
    }
  }
  q = warp_sum(q);
  k = warp_sum(k);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (lane == 0) {
    red[0][warp] = q;
    red[1][warp] = k;
  }
  __syncthreads();
  q = lane < kRopeThreads / 32 ? red[0][lane] : 0.f;
  k = lane < kRopeThreads / 32 ? red[1][lane] : 0.f;   // (all columns have been read)
  return make_float2(warp_sum(q), warp_sum(k));
}

template <typename T, bool VEC>
__global__ void __launch_bounds__(kRopeThreads) head_rope_cache_kernel(const HeadRopeArgs p) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(16) float sm[];
  const long long t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* cs = sm + (kRopeThreads / 32) * p.D;
  float* row = sm + warp * p.D;
  for (int i = threadIdx.x; i < 2 * p.half; i += blockDim.x) cs[i] = p.table[t * 2 * p.half + i];
  __syncthreads();
  long long slot = p.slots[t];
  if (slot >= p.num_slots) {
    if (threadIdx.x == 0) report_error(p.status, kErrBounds, 43, (int)t);
    slot = -1;
  }
  const long long blk = slot >= 0 ? slot / p.block_size : 0;
  const long long off = slot >= 0 ? slot % p.block_size : 0;
  T* base = reinterpret_cast<T*>(p.proj) + t * p.ld;
  float inv_q = 1.f, inv_k = 1.f;
  if (p.whole) {
    const float2 ss = projection_squares(base, p.Hq * p.D, p.Hkv * p.D, VEC);
    inv_q = 1.f / sqrtf(ss.x * p.rdim + p.eps);
    inv_k = 1.f / sqrtf(ss.y * p.rdim_k + p.eps);
  }
  for (int j = warp; j < p.Hq + 2 * p.Hkv; j += kRopeThreads / 32) {
    const bool is_q = j < p.Hq, is_v = j >= p.Hq + p.Hkv;
    if (!is_q && slot < 0) continue;   // padding token: no key, no value
    if (is_v) {
      const int g = j - p.Hq - p.Hkv;
      const T* src = base + (long long)(p.shared_kv ? p.Hq : p.Hq + p.Hkv) * p.D + (long long)g * p.Dv;
      T* dst = reinterpret_cast<T*>(p.v_cache) + ((blk * p.Hkv + g) * p.block_size + off) * p.Dv;
      if (VEC) {
        for (int i = lane * 4; i < p.Dv; i += 128) store4(dst + i, load4(src + i));
      } else {
        for (int i = lane; i < p.Dv; i += 32) dst[i] = src[i];
      }
      continue;
    }
    T* src = base + (long long)j * p.D;
    const float* w = is_q ? p.wq : p.wk;
    float inv = 1.f;
    if (p.whole) {
      w += (long long)(is_q ? j : j - p.Hq) * p.D;
      inv = is_q ? inv_q : inv_k;
    } else if (w != nullptr) {
      float ss = 0.f;
      if (VEC) {
        for (int i = lane * 4; i < p.D; i += 128) {
          const float4 v = load4(src + i);
          ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
      } else {
        for (int i = lane; i < p.D; i += 32) {
          const float v = to_f32<T>(src[i]);
          ss += v * v;
        }
      }
      inv = 1.f / sqrtf(warp_sum(ss) * p.rdim + p.eps);
    }
    __syncwarp();   // the last head's row has been read
    if (VEC) {
      for (int i = lane * 4; i < p.D; i += 128) {
        float4 v = load4(src + i);
        if (w != nullptr) {
          const float4 g = load4(w + i);
          v = make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w);
        }
        store4(row + i, v);
      }
    } else {
      for (int i = lane; i < p.D; i += 32)
        row[i] = w != nullptr ? to_f32<T>(src[i]) * inv * w[i] : to_f32<T>(src[i]);
    }
    __syncwarp();
    T* dst = src;
    if (!is_q)
      dst = reinterpret_cast<T*>(p.k_cache) +
            ((blk * p.Hkv + (j - p.Hq)) * p.block_size + off) * p.D;
    if (VEC) {
      for (int i = lane * 4; i < p.D; i += 128)
        store4(dst + i, make_float4(rotated(row, cs, p.half, i), rotated(row, cs, p.half, i + 1),
                                    rotated(row, cs, p.half, i + 2), rotated(row, cs, p.half, i + 3)));
    } else {
      for (int i = lane; i < p.D; i += 32) dst[i] = from_f32<T>(rotated(row, cs, p.half, i));
    }
  }
}

// D = Dv = 64 or 128, half a multiple of 4
template <int D>
__global__ void __launch_bounds__(kRopeThreads, 4) head_rope_cache_wide_kernel(const HeadRopeArgs p) {
  pdl_wait();
  pdl_trigger();
  constexpr int kLanes = D / 4;                 // per head
  constexpr int kPer = 32 / kLanes;             // heads per warp
  constexpr int kStep = kPer * kRopeThreads / 32;
  constexpr int kFlight = 6;                    // heads per lane in flight
  const long long t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int i0 = (lane % kLanes) * 4;           // this lane's columns
  const int j0 = warp * kPer + lane / kLanes;   // its first head
  const int heads = p.Hq + 2 * p.Hkv;
  const int v_back = p.shared_kv ? p.Hkv : 0;   // value heads read the key heads' columns
  __nv_bfloat16* base = reinterpret_cast<__nv_bfloat16*>(p.proj) + t * p.ld + i0;
  const int side = i0 < p.half ? 0 : i0 < 2 * p.half ? 1 : 2;   // first, second of a pair, neither
  const int other = side == 0 ? lane + p.half / 4 : side == 1 ? lane - p.half / 4 : lane;
  float4 v[kFlight];
  auto load = [&](int first) {
#pragma unroll
    for (int f = 0; f < kFlight; ++f) {
      const int j = first + f * kStep + j0;
      v[f] = j < heads ? load4(base + (long long)(j < p.Hq + p.Hkv ? j : j - v_back) * D)
                       : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  float inv_q = 1.f, inv_k = 1.f;
  if (p.whole) {
    const float2 ss = projection_squares(base - i0, p.Hq * D, p.Hkv * D, true);
    inv_q = rsqrtf(ss.x * p.rdim + p.eps);
    inv_k = rsqrtf(ss.y * p.rdim_k + p.eps);
  }
  load(0);
  const long long slot = p.slots[t];
  float4 c = make_float4(1.f, 1.f, 1.f, 1.f), sn = make_float4(0.f, 0.f, 0.f, 0.f);
  if (side < 2) {
    const float* cs = p.table + (t * p.half + i0 - side * p.half) * 2;
    const float4 a = load4(cs), b = load4(cs + 4);
    const float sg = side == 0 ? -1.f : 1.f;
    c = make_float4(a.x, a.z, b.x, b.z);
    sn = make_float4(sg * a.y, sg * a.w, sg * b.y, sg * b.w);
  }
  float4 wq = make_float4(1.f, 1.f, 1.f, 1.f), wk = wq;
  if (p.wq != nullptr && !p.whole) {
    wq = load4(p.wq + i0);
    wk = load4(p.wk + i0);
  }
  long long row0 = -1;   // cache row of K/V head 0 (-1: padding token)
  if (slot >= p.num_slots) {
    if (threadIdx.x == 0) report_error(p.status, kErrBounds, 43, (int)t);
  } else if (slot >= 0) {   // (fewer than 2^31 slots)
    const unsigned blk = (unsigned)slot / (unsigned)p.block_size;
    row0 = (long long)blk * p.Hkv * p.block_size + ((unsigned)slot - blk * p.block_size);
  }
  for (int first = 0; first < heads; first += kStep * kFlight) {
    if (first > 0) load(first);
#pragma unroll
    for (int f = 0; f < kFlight; ++f) {
      if (first + f * kStep >= heads) break;
      const int j = first + f * kStep + j0;
      const bool is_v = j >= p.Hq + p.Hkv;
      float4 x = v[f];
      if (first + f * kStep + warp * kPer < p.Hq + p.Hkv) {   // (else all of the warp's are values)
        float4 z = x;
        if (p.whole) {
          if (j < p.Hq + p.Hkv) {
            const float4 w = j < p.Hq ? load4(p.wq + (long long)j * D + i0)
                                      : load4(p.wk + (long long)(j - p.Hq) * D + i0);
            const float inv = j < p.Hq ? inv_q : inv_k;
            z = make_float4(x.x * inv * w.x, x.y * inv * w.y, x.z * inv * w.z, x.w * inv * w.w);
          }
        } else if (p.wq != nullptr) {
          float ss = x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
#pragma unroll
          for (int o = kLanes / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
          const float inv = rsqrtf(ss * p.rdim + p.eps);
          const float4 w = j < p.Hq ? wq : wk;
          z = make_float4(x.x * inv * w.x, x.y * inv * w.y, x.z * inv * w.z, x.w * inv * w.w);
        }
        const float4 y = make_float4(
            __shfl_sync(0xffffffffu, z.x, other), __shfl_sync(0xffffffffu, z.y, other),
            __shfl_sync(0xffffffffu, z.z, other), __shfl_sync(0xffffffffu, z.w, other));
        if (!is_v)
          x = make_float4(z.x * c.x + y.x * sn.x, z.y * c.y + y.y * sn.y, z.z * c.z + y.z * sn.z,
                          z.w * c.w + y.w * sn.w);
      }
      if (j < p.Hq) {
        store4(base + (long long)j * D, x);
      } else if (j < heads && row0 >= 0) {
        const int g = is_v ? j - p.Hq - p.Hkv : j - p.Hq;
        __nv_bfloat16* cache = reinterpret_cast<__nv_bfloat16*>(is_v ? p.v_cache : p.k_cache);
        store4(cache + (row0 + g * p.block_size) * D + i0, x);
      }
    }
  }
}

struct LatentRopeArgs {
  void* q;                  // [T][ld]: H heads of dq columns, the rotary part from column dim
  const void* ckv;          // [T][ld]: R latent columns, then 2 * half rotary ones
  long long ld;
  const float* table;       // [T][half][2]
  const long long* slots;
  const float* weight;      // [R]
  void* cache;              // rows of `width` columns, the rotary key part from column rot_at
  long long num_slots;
  int H, dq, dim, R, half, width, rot_at;
  int vec;                  // four columns at a time are aligned
  float eps;
  int* status;
};

template <typename T>
__global__ void __launch_bounds__(kRopeThreads) latent_rope_cache_kernel(const LatentRopeArgs p) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(16) float cs[];
  __shared__ float red[32];
  const long long t = blockIdx.x;
  for (int i = threadIdx.x; i < 2 * p.half; i += blockDim.x) cs[i] = p.table[t * 2 * p.half + i];
  const T* c = reinterpret_cast<const T*>(p.ckv) + t * p.ld;
  float ss = 0.f;
  for (int i = threadIdx.x; i < p.R; i += blockDim.x) {
    const float v = to_f32<T>(c[i]);
    ss += v * v;
  }
  const float inv = 1.f / sqrtf(block_sum_all(ss, red) / (float)p.R + p.eps);   // (publishes cs)
  const long long slot = p.slots[t];
  if (slot >= p.num_slots) {
    if (threadIdx.x == 0) report_error(p.status, kErrBounds, 44, (int)t);
  } else if (slot >= 0) {
    T* dst = reinterpret_cast<T*>(p.cache) + slot * p.width;
    for (int i = threadIdx.x; i < p.R; i += blockDim.x)
      dst[i] = from_f32<T>(to_f32<T>(c[i]) * inv * p.weight[i]);
    for (int i = threadIdx.x; i < p.half; i += blockDim.x) {
      const float u = to_f32<T>(c[p.R + i]), v = to_f32<T>(c[p.R + p.half + i]);
      dst[p.rot_at + i] = from_f32<T>(u * cs[2 * i] - v * cs[2 * i + 1]);
      dst[p.rot_at + p.half + i] = from_f32<T>(v * cs[2 * i] + u * cs[2 * i + 1]);
    }
  }
  T* q = reinterpret_cast<T*>(p.q) + t * p.ld;
  if (p.vec) {   // four pairs a thread
    const int quads = p.half / 4, n = p.H * quads;
    for (int k = threadIdx.x; k < n; k += blockDim.x) {
      const int h = k / quads, i = (k - h * quads) * 4;
      T* a = q + (long long)h * p.dq + p.dim + i;
      const float4 u = load4(a), v = load4(a + p.half);
      const float* g = cs + 2 * i;
      store4(a, make_float4(u.x * g[0] - v.x * g[1], u.y * g[2] - v.y * g[3], u.z * g[4] - v.z * g[5],
                            u.w * g[6] - v.w * g[7]));
      store4(a + p.half, make_float4(v.x * g[0] + u.x * g[1], v.y * g[2] + u.y * g[3],
                                     v.z * g[4] + u.z * g[5], v.w * g[6] + u.w * g[7]));
    }
    return;
  }
  const int n = p.H * p.half;
  for (int k = threadIdx.x; k < n; k += blockDim.x) {
    const int h = k / p.half, i = k - h * p.half;
    T* a = q + (long long)h * p.dq + p.dim + i;
    const float u = to_f32<T>(a[0]), v = to_f32<T>(a[p.half]);
    a[0] = from_f32<T>(u * cs[2 * i] - v * cs[2 * i + 1]);
    a[p.half] = from_f32<T>(v * cs[2 * i] + u * cs[2 * i + 1]);
  }
}

template <typename T>
static int launch_head_rope(const HeadRopeArgs& a, long long n, cudaStream_t stream) {
  const size_t smem = ((size_t)(kRopeThreads / 32) * a.D + 2 * (size_t)a.half) * sizeof(float);
  if (smem > 200 * 1024) return -6;
  const bool vec = a.D % 4 == 0 && a.Dv % 4 == 0 && a.ld % 4 == 0 &&
                   ((reinterpret_cast<uintptr_t>(a.proj) | reinterpret_cast<uintptr_t>(a.wq) |
                     reinterpret_cast<uintptr_t>(a.wk) | reinterpret_cast<uintptr_t>(a.k_cache) |
                     reinterpret_cast<uintptr_t>(a.v_cache)) & 15) == 0;
  if (sizeof(T) == 2 && vec && a.D == a.Dv && (a.D == 64 || a.D == 128) && a.half % 4 == 0 &&
      a.num_slots <= 0x7fffffffll && (a.wq == nullptr || a.wk != nullptr))
    return launch_pdl(a.D == 128 ? head_rope_cache_wide_kernel<128> : head_rope_cache_wide_kernel<64>,
                      dim3((unsigned)n), dim3(kRopeThreads), 0, stream, a) == cudaSuccess
               ? 0
               : -5;
  auto k = vec ? head_rope_cache_kernel<T, true> : head_rope_cache_kernel<T, false>;
  if (smem > 48 * 1024 &&
      cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return -3;
  return launch_pdl(k, dim3((unsigned)n), dim3(kRopeThreads), smem, stream, a) == cudaSuccess ? 0 : -5;
}

}  // namespace ab200

using namespace ab200;
typedef __nv_bfloat16 bf16;

extern "C" {

// positions int64 [T], freq fp32 [half] -> table fp32 [T, half, 2]: cosine, sine
int ab200_rotary_table(const void* positions, const void* freq, void* table, long long T, int half,
                       cudaStream_t stream) {
  const long long n = T * half;
  if (n <= 0) return 0;
  if (n > (1ll << 38)) return -6;
  return launch_pdl(rotary_table_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, stream,
                    reinterpret_cast<const long long*>(positions),
                    reinterpret_cast<const float*>(freq), reinterpret_cast<float2*>(table), half,
                    n) == cudaSuccess
             ? 0
             : -5;
}

// proj [T, ld] holds Hq query and Hkv key heads of D columns, then Hkv value heads of Dv, of which
// the first `dim` (query, key) columns are in use and the others zero; wq, wk fp32 [D] or null, with
// `whole` fp32 [Hq * D] and [Hkv * D] for a norm over all heads at once; table fp32 [T, half, 2]:
// cosines and sines of the pairs (i, i + half). shared_kv: there are no value heads, the key heads as
// they come are the values (Dv = D).
int ab200_head_rope_cache(void* proj, long long ld, const void* table, int half,
                          const void* slots, const void* wq, const void* wk, void* k_cache,
                          void* v_cache, long long T, int Hq, int Hkv, int D, int dim, int Dv,
                          int block_size, long long num_slots, float eps, int whole, int shared_kv,
                          int dtype, int* status, cudaStream_t stream) {
  if (T <= 0) return 0;
  if ((whole && (wq == nullptr || wk == nullptr)) || (shared_kv && D != Dv)) return -2;
  if (dim < 1 || dim > D || 2 * half > D || half < 0 || block_size < 1 || Hq < 0 || Hkv < 0) return -2;
  if (ld < (long long)(Hq + Hkv) * D + (shared_kv ? 0ll : (long long)Hkv * Dv)) return -2;
  HeadRopeArgs a;
  a.proj = proj; a.ld = ld;
  a.table = reinterpret_cast<const float*>(table);
  a.slots = reinterpret_cast<const long long*>(slots);
  a.wq = reinterpret_cast<const float*>(wq);
  a.wk = reinterpret_cast<const float*>(wk);
  a.k_cache = k_cache; a.v_cache = v_cache;
  a.num_slots = num_slots;
  a.Hq = Hq; a.Hkv = Hkv; a.D = D; a.Dv = Dv;
  a.half = half; a.block_size = block_size;
  a.whole = whole;
  a.shared_kv = shared_kv;
  a.rdim = 1.f / (whole ? (float)Hq * (float)dim : (float)dim);
  a.rdim_k = 1.f / (whole ? (float)Hkv * (float)dim : (float)dim);
  a.eps = eps;
  a.status = status;
  return dtype == 0 ? launch_head_rope<bf16>(a, T, stream) : launch_head_rope<float>(a, T, stream);
}

// q [T, ld]: H heads of dq columns whose rotary part starts at column `dim`; ckv [T, ld]: R latent
// columns and 2 * half rotary ones; cache rows of `width` columns, the rotary part at rot_at.
int ab200_latent_rope_cache(void* q, const void* ckv, long long ld, const void* table, int half,
                            const void* slots, const void* weight, void* cache, long long T, int H, int dq, int dim, int R, int width,
                            int rot_at, long long num_slots, float eps, int dtype, int* status,
                            cudaStream_t stream) {
  if (T <= 0) return 0;
  if (half < 0 || dim + 2 * half > dq || R > rot_at || rot_at + 2 * half > width) return -2;
  LatentRopeArgs a;
  a.q = q; a.ckv = ckv; a.ld = ld;
  a.table = reinterpret_cast<const float*>(table);
  a.slots = reinterpret_cast<const long long*>(slots);
  a.weight = reinterpret_cast<const float*>(weight);
  a.cache = cache;
  a.num_slots = num_slots;
  a.H = H; a.dq = dq; a.dim = dim; a.R = R; a.half = half;
  a.width = width; a.rot_at = rot_at;
  a.eps = eps;
  a.status = status;
  a.vec = half > 0 && half % 4 == 0 && dim % 4 == 0 && dq % 4 == 0 && ld % 4 == 0 &&
          (reinterpret_cast<uintptr_t>(q) & 15) == 0;
  const size_t smem = (2 * (size_t)half + 4) * sizeof(float);
  if (smem > 48 * 1024) return -6;
  auto k = dtype == 0 ? latent_rope_cache_kernel<bf16> : latent_rope_cache_kernel<float>;
  return launch_pdl(k, dim3((unsigned)T), dim3(kRopeThreads), smem, stream, a) == cudaSuccess ? 0 : -5;
}

}  // extern "C"
