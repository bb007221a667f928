// Plain fp32-accumulating kernels without tensor cores, for models served in 32-bit and for
// 16-bit shapes the tensor-core kernels do not take (rows that are no multiple of 16 bytes,
// latents wider than 512):
//
//   linear_exact            out[g] = x[g] * w[g]^T: one matrix, one per group (heads), or one per
//                           expert over rows sorted by expert (a device-side tile list)
//   attention_exact         softmax attention over a paged cache (keys and values, or one latent
//                           row that is both), with a mask, a sink and an output gate, a block
//                           per (token, head), keys in tiles with a running maximum
//
// Every product and sum is IEEE fp32 (FMA); no reduced-precision mode is involved.

#include "api.h"
#include "common/elem.cuh"
#include "common/pdl.cuh"

namespace ab200 {

constexpr int kXM = 128, kXN = 64, kXK = 16;

struct ExactArgs {
  const void* x;
  long long ldx, x_gstride;
  const void* w;
  long long ldw, w_gstride;
  void* out;
  long long ldo, out_gstride;
  int M, N, K;
  const int4* tiles;      // optional: (group, first row, rows, -) per 128-row tile ...
  const int* num_tiles;   // ... and how many of them are in use
};

template <typename T>
__global__ void __launch_bounds__(256) linear_exact_kernel(const ExactArgs p) {
  pdl_wait();
  pdl_trigger();
  __shared__ float xs[kXK][kXM + 4];
  __shared__ float ws[kXK][kXN + 4];
  int group, row0, nrows;
  if (p.tiles != nullptr) {
    if ((int)blockIdx.y >= *p.num_tiles) return;
    const int4 t = p.tiles[blockIdx.y];
    group = t.x;
    row0 = t.y;
    nrows = t.z;
  } else {
    group = blockIdx.z;
    row0 = blockIdx.y * kXM;
    nrows = min(kXM, p.M - row0);
  }
  const int n0 = blockIdx.x * kXN;
  const T* x = reinterpret_cast<const T*>(p.x) + group * p.x_gstride;
  const T* w = reinterpret_cast<const T*>(p.w) + group * p.w_gstride;
  T* out = reinterpret_cast<T*>(p.out) + group * p.out_gstride;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;   // 16 x 16 threads, 8 x 4 outputs each
  float acc[8][4];
#pragma unroll
  for (int i = 0; i < 8; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < p.K; k0 += kXK) {
    for (int i = threadIdx.x; i < kXM * kXK; i += 256) {
      const int r = i / kXK, k = i % kXK;
      xs[k][r] = (r < nrows && k0 + k < p.K) ? to_f32<T>(x[(long long)(row0 + r) * p.ldx + k0 + k]) : 0.f;
    }
    for (int i = threadIdx.x; i < kXN * kXK; i += 256) {
      const int n = i / kXK, k = i % kXK;
      ws[k][n] = (n0 + n < p.N && k0 + k < p.K) ? to_f32<T>(w[(long long)(n0 + n) * p.ldw + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kXK; ++k) {
      float a[8], b[4];
#pragma unroll
      for (int i = 0; i < 8; ++i) a[i] = xs[k][ty + 16 * i];
#pragma unroll
      for (int j = 0; j < 4; ++j) b[j] = ws[k][tx + 16 * j];
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int r = ty + 16 * i;
    if (r >= nrows) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx + 16 * j;
      if (n < p.N) out[(long long)(row0 + r) * p.ldo + n] = from_f32<T>(acc[i][j]);
    }
  }
}

constexpr int kAttnKeys = 128;

struct ExactAttnArgs {
  const void* q;            // [T][ldq], head h at column h * Dk
  long long ldq;
  // cache row of (block, kv head, offset): ((block * Hkv + head) * block_size + offset) * row
  const void* k;
  const void* v;
  int k_row, v_row;
  const int* block_tables;
  int max_blocks, block_size;
  const int* tok_seq;       // [T] sequence (row of block_tables) of each token
  const long long* positions;
  const float* sink;        // [H] or null
  const void* gate;         // [T][ldg], head h at column h * Dv (gate_head: at column h, one), or null
  long long ldg;
  int gate_head;
  void* out;                // [T][ldo], head h at column h * Dv
  long long ldo;
  int H, Hkv, Dk, Dv, num_blocks;
  int mask_kind, mask_size;
  float scale, softcap;     // softcap > 0: scores become softcap * tanh(score / softcap)
  int* status;
};

// Shared memory: q[Dk], the accumulator[Dv]; the tile's cache rows and weights.
template <typename T>
__global__ void __launch_bounds__(kAttnKeys) attention_exact_kernel(const ExactAttnArgs p) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[32];
  __shared__ float pw[kAttnKeys];
  __shared__ long long rowp[kAttnKeys];
  float* q = sm;
  float* acc = sm + p.Dk;
  const long long t = blockIdx.x;
  const int h = blockIdx.y;
  const int kvh = h / (p.H / p.Hkv);
  const int tid = threadIdx.x;
  const T* qr = reinterpret_cast<const T*>(p.q) + t * p.ldq + (long long)h * p.Dk;
  for (int i = tid; i < p.Dk; i += kAttnKeys) q[i] = to_f32<T>(qr[i]);
  for (int i = tid; i < p.Dv; i += kAttnKeys) acc[i] = 0.f;
  const long long n_keys = p.positions[t] + 1;
  const int* bt = p.block_tables + (long long)p.tok_seq[t] * p.max_blocks;
  const T* kc = reinterpret_cast<const T*>(p.k);
  const T* vc = reinterpret_cast<const T*>(p.v);
  float m = -INFINITY, l = 0.f;
  for (long long k0 = first_visible(p.mask_kind, p.mask_size, (int)(n_keys - 1)); k0 < n_keys;
       k0 += kAttnKeys) {
    __syncthreads();   // q and acc are set; the last tile's weights have been read
    const long long key = k0 + tid;
    float s = -INFINITY;
    if (key < n_keys) {
      const long long b = key / p.block_size;
      const int blk = b < p.max_blocks ? bt[b] : -1;
      if (blk >= 0 && blk < p.num_blocks) {
        const long long row = ((long long)blk * p.Hkv + kvh) * p.block_size + key % p.block_size;
        rowp[tid] = row * p.v_row;
        const T* kr = kc + row * p.k_row;
        float d = 0.f;
        for (int i = 0; i < p.Dk; ++i) d = fmaf(q[i], to_f32<T>(kr[i]), d);
        s = d * p.scale;
        if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
      } else {
        rowp[tid] = 0;
        report_error(p.status, kErrBounds, 42, (int)t);
      }
    }
    const float m_new = fmaxf(m, block_max_all(s, red));
    const float w = s == -INFINITY ? 0.f : expf(s - m_new);
    pw[tid] = w;
    const float sum = block_sum_all(w, red);   // (its barriers also publish pw and rowp)
    const float keep = m == -INFINITY ? 0.f : expf(m - m_new);
    l = l * keep + sum;
    m = m_new;
    const int n = (int)min((long long)kAttnKeys, n_keys - k0);
    for (int i = tid; i < p.Dv; i += kAttnKeys) {
      float a = acc[i] * keep;
      for (int j = 0; j < n; ++j) a = fmaf(pw[j], to_f32<T>(vc[rowp[j] + i]), a);
      acc[i] = a;
    }
  }
  if (p.sink != nullptr && m != -INFINITY) l += expf(p.sink[h] - m);
  T* o = reinterpret_cast<T*>(p.out) + t * p.ldo + (long long)h * p.Dv;
  const T* gate = p.gate ? reinterpret_cast<const T*>(p.gate) + t * p.ldg +
                               (long long)h * (p.gate_head ? 1 : p.Dv) : nullptr;
  const float inv = l > 0.f ? 1.f / l : 0.f;
  for (int i = tid; i < p.Dv; i += kAttnKeys) {   // own columns
    float v = acc[i] * inv;
    if (gate != nullptr) v /= 1.f + expf(-to_f32<T>(gate[p.gate_head ? 0 : i]));
    o[i] = from_f32<T>(v);
  }
}

}  // namespace ab200

using namespace ab200;
typedef __nv_bfloat16 bf16;

extern "C" {

// Strides in elements. With `tiles` (int32 x 4 per tile) x and out hold the rows of all groups
// one after the other and M is ignored; else every group has M rows at its own x / out offset.
int ab200_linear_exact(const void* x, long long ldx, long long x_gstride, const void* w,
                       long long ldw, long long w_gstride, void* out, long long ldo,
                       long long out_gstride, int M, int N, int K, int groups, const void* tiles,
                       const void* num_tiles, int max_tiles, int dtype, cudaStream_t stream) {
  if (N <= 0 || K <= 0 || groups <= 0 || (tiles == nullptr ? M : max_tiles) <= 0) return 0;
  if (tiles != nullptr && num_tiles == nullptr) return -2;
  ExactArgs a;
  a.x = x; a.ldx = ldx; a.x_gstride = x_gstride;
  a.w = w; a.ldw = ldw; a.w_gstride = w_gstride;
  a.out = out; a.ldo = ldo; a.out_gstride = out_gstride;
  a.M = M; a.N = N; a.K = K;
  a.tiles = reinterpret_cast<const int4*>(tiles);
  a.num_tiles = reinterpret_cast<const int*>(num_tiles);
  const long long ny = tiles ? max_tiles : (M + kXM - 1) / kXM;
  if (ny > 65535 || groups > 65535) return -6;
  const dim3 grid((unsigned)((N + kXN - 1) / kXN), (unsigned)ny, tiles ? 1u : (unsigned)groups);
  const cudaError_t e = dtype == 0
                            ? launch_pdl(linear_exact_kernel<bf16>, grid, dim3(256), 0, stream, a)
                            : launch_pdl(linear_exact_kernel<float>, grid, dim3(256), 0, stream, a);
  return e == cudaSuccess ? 0 : -5;
}

// k: [num_blocks, Hkv, block_size, k_row] of which the first Dk columns count, v likewise (it may
// be the same tensor); sink fp32 [H] and gate [T, ldg] (a number per column, or with gate_head one per
// head) may be null.
int ab200_attention_exact(const void* q, long long ldq, const void* k, int k_row, const void* v,
                          int v_row, int num_blocks, int block_size, const void* block_tables,
                          int max_blocks, const void* tok_seq, const void* positions,
                          const void* sink, const void* gate, long long ldg, int gate_head,
                          void* out, long long ldo, long long T, int H, int Hkv, int Dk, int Dv,
                          int mask_kind, int mask_size, float scale, float softcap, int dtype,
                          int* status, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H < 1 || Hkv < 1 || H % Hkv || Dk > k_row || Dv > v_row || block_size < 1) return -2;
  if (mask_kind < kMaskCausal || mask_kind > kMaskChunk || (mask_kind != kMaskCausal && mask_size < 1))
    return -2;
  const size_t smem = ((size_t)Dk + Dv) * sizeof(float);
  if (H > 65535 || smem > 200 * 1024) return -6;
  ExactAttnArgs a;
  a.q = q; a.ldq = ldq;
  a.k = k; a.v = v;
  a.k_row = k_row; a.v_row = v_row;
  a.block_tables = reinterpret_cast<const int*>(block_tables);
  a.max_blocks = max_blocks; a.block_size = block_size;
  a.tok_seq = reinterpret_cast<const int*>(tok_seq);
  a.positions = reinterpret_cast<const long long*>(positions);
  a.sink = reinterpret_cast<const float*>(sink);
  a.gate = gate; a.ldg = ldg; a.gate_head = gate_head;
  a.out = out; a.ldo = ldo;
  a.H = H; a.Hkv = Hkv; a.Dk = Dk; a.Dv = Dv;
  a.num_blocks = num_blocks;
  a.mask_kind = mask_kind; a.mask_size = mask_size;
  a.scale = scale;
  a.softcap = softcap;
  a.status = status;
  const dim3 grid((unsigned)T, (unsigned)H);
  auto kern = dtype == 0 ? attention_exact_kernel<bf16> : attention_exact_kernel<float>;
  if (smem > 40 * 1024 &&
      cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return -3;
  return launch_pdl(kern, grid, dim3(kAttnKeys), smem, stream, a) == cudaSuccess ? 0 : -5;
}

}  // extern "C"
