// Recurrent mixers: layers that carry a [dim, vdim] matrix per head from token to token.
//
//   delta rule      q, k, v through a short causal convolution and silu; q and k to unit length; a
//                   decay g per key channel and a step size beta per head:
//                       S <- g * S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//   matrix memory   log gates i, f per head with a running maximum m (m' = max(f + m, i)):
//                       S <- exp(f + m - m') S + exp(i - m') k v^T,  z likewise with k alone;
//                       o = S^T q / (max(|z . q|, exp(-m')) + 1e-6)
//                   z is kept as one more column of S, whose value is always 1.
//
// Both are followed by the RMS norm of each head's o, a weight and an output gate. Everything that
// enters the recurrence is fp32, and so is its arithmetic (FMAs on pairs of rows).
//
// A block owns a sequence's head, or some of the head's columns, which do not depend on one another,
// and keeps its part of S in registers for all of the sequence's tokens in this step: a lane holds
// DP / 8 rows by kCols columns. Tokens come in tiles. Per tile the block first prepares the vectors
// the recurrence needs in shared memory (convolution, norms, gates, decays), then runs the
// recurrence B tokens at a time, then writes the tile's normed and gated outputs.
//
// Within a tile S is held undecayed: S = G * Z with G the product of the tile's decays so far (per
// row), so that a token costs three multiply-adds per element and not four,
//     Z^T (G k), Z^T (G q) and Z <- Z + (k / G) u^T,
// and B tokens need no exchange but their scalar products: with a = G k, b = k / G, c = G q
//     u_i = beta_i (v_i - Z^T a_i - sum_{j<i} (a_i . b_j) u_j),  o_i = Z^T c_i + sum_{j<=i} (c_i . b_j) u_j
// where Z is the one before the first of them. G goes back to 1 at a tile's end, and after every B
// tokens when a channel decays so much within the tile that 1 / G would leave fp32's range.
//
// What a sequence carries over lies in its slot: S in fp32; the convolution's last inputs and m twice,
// for even and odd steps of the sequence (`phase`), so that blocks which read them never race with the
// block that writes them. A sequence that starts at position 0 reads nothing from its slot.

#include "api.h"
#include "common/elem.cuh"
#include "common/pdl.cuh"

namespace ab200 {

constexpr int kScanMaxWarps = 10;
constexpr float kMinLogDecay = -20.f;     // per token: a factor below 2e-9 is as good as that
constexpr float kTileLogDecay = -60.f;    // a tile whose decays multiply to less is cut
constexpr int kStepInts = 5;              // first row, rows, slot, start position, phase

struct ScanArgs {
  const void* proj;          // [T][ld]: projections of the layer's input (element type T)
  long long ld;
  int q_at, k_at, v_at;      // columns of head 0's query, key and value
  int b_at;                  // delta: step sizes [heads]
  int i_at, f_at;            // memory: gates [heads]
  const void* decay;         // delta: [T][ld_decay], head h's channels at column h * dim
  long long ld_decay;
  const void* gate;          // output gate [T][ld_gate], head h at column h * vdim
  long long ld_gate;
  const float* conv;         // delta: [taps][channels]: queries', keys', values' weights
  const float* a_exp;        // delta: [heads] exp(A_log)
  const float* dt_bias;      // delta: [heads][dim]
  const float* i_bias;       // memory: [heads]
  const float* f_bias;
  const float* norm;         // head h's weights at h * norm_step
  int norm_step;
  float* state;              // [slots][heads][dim][state_cols]
  int state_cols;
  void* conv_state;          // delta: [slots][2][taps - 1][channels] (element type T)
  float* max_state;          // memory: [slots][2][heads]
  const int* steps;          // [n][kStepInts]
  void* out;                 // [T][ldo], head h at column h * vdim (one block per head) ...
  long long ldo;
  float* raw;                // ... or [T][heads][raw_cols] unnormed, for scan_output
  int raw_cols;
  int num_slots, heads, group, dim, vdim, ncols, taps, channels;
  int slices, nc;            // blocks per head, columns of each
  int vec;                   // four channels at a time are aligned
  float q_scale, cap, eps;
  int* status;
};

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

__device__ __forceinline__ float softplus_f(float z) {
  return fmaxf(z, 0.f) + log1pf(__expf(-fabsf(z)));
}
__device__ __forceinline__ float silu_f(float z) { return __fdividef(z, 1.f + __expf(-z)); }
__device__ __forceinline__ float sigmoid_f(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }

// DP: rows (dim, zero-padded); B tokens at a time, TT per tile
template <int DP>
struct ScanShape {
  static constexpr int kRows = DP / 8;                  // per lane, in chunks of four
  static constexpr int kCols = DP <= 128 ? 4 : 2;
  static constexpr int kWarpCols = 4 * kCols;
};

template <int DP, int TT, int B, bool DELTA>
struct ScanSmem {   // offsets in floats
  static constexpr int kB = 0, kC = kB + TT * DP, kA = kC + TT * DP, kG = kA + (DELTA ? TT * DP : 0);
  static constexpr int kDotB = kG + TT / B * DP, kDotC = kDotB + TT * B, kBeta = kDotC + TT * B;
  static constexpr int kInvQ = kBeta + TT, kInvK = kInvQ + TT, kMax = kInvK + TT, kV = (kMax + TT + 2 + 3) / 4 * 4;
  static constexpr int total(int nc) { return kV + TT * nc; }
};

template <typename T, int DP, int TT, int B, bool DELTA>
__global__ void __launch_bounds__(kScanMaxWarps * 32, 1) scan_kernel(const ScanArgs p) {
  using Sh = ScanShape<DP>;
  using Sm = ScanSmem<DP, TT, B, DELTA>;
  constexpr int kRows = Sh::kRows, kCols = Sh::kCols, kChunks = kRows / 4;
  extern __shared__ __align__(16) float sm[];
  float* sB = sm + Sm::kB;       // keys, then k / G
  float* sC = sm + Sm::kC;       // queries, then G q
  float* sA = sm + Sm::kA;       // G k
  float* sG = sm + Sm::kG;
  float* dotB = sm + Sm::kDotB;  // [token][earlier token of its group]: a . b
  float* dotC = sm + Sm::kDotC;  // c . b
  float* sBeta = sm + Sm::kBeta; // delta: step size; memory: log of the input factor
  float* invQ = sm + Sm::kInvQ;  // memory: cumulative log decay
  float* invK = sm + Sm::kInvK;
  float* sMax = sm + Sm::kMax;   // memory: m per token; [TT]: m carried over, [TT + 1]: flag
  float* sV = sm + Sm::kV;       // values, then outputs [TT][nc]
  pdl_wait();
  pdl_trigger();

  const int slice = blockIdx.x % p.slices;
  const int h = blockIdx.x / p.slices % p.heads;
  const int* step = p.steps + (long long)(blockIdx.x / p.slices / p.heads) * kStepInts;
  const long long first = step[0];
  const int n = step[1], slot = step[2], start = step[3], phase = step[4] & 1;
  if (n <= 0) return;
  const int tid = threadIdx.x, threads = blockDim.x, warp = tid >> 5, lane = tid & 31;
  const int warps = threads >> 5;
  const int nc = p.nc, c_first = slice * nc;
  const int hv = h;                                // value head
  const int hk = DELTA ? h / p.group : h;          // query / key head
  const T* proj = reinterpret_cast<const T*>(p.proj);
  if (slot <= 0 || slot >= p.num_slots) {          // padding rows: finite outputs, no state
    if (slot >= p.num_slots && tid == 0) report_error(p.status, kErrBounds, 50, slot);
    for (int t = 0; t < n; ++t) {
      if (p.raw != nullptr) {
        float* dst = p.raw + ((first + t) * p.heads + h) * p.raw_cols;
        for (int c = c_first + tid; c < min(c_first + nc, p.raw_cols); c += threads) dst[c] = 0.f;
        if (!DELTA && slice == 0 && tid == 0) dst[p.ncols] = 1.f;
      } else {
        T* dst = reinterpret_cast<T*>(p.out) + (first + t) * p.ldo + (long long)h * p.vdim;
        for (int c = tid; c < p.vdim; c += threads) dst[c] = from_f32<T>(0.f);
      }
    }
    return;
  }

  // ---- this lane's part of the state
  const int rl = lane & 7;
  const int c_local = warp * Sh::kWarpCols + (lane >> 3) * kCols;   // of the block's columns
  const int c0 = c_first + c_local;
  float* state = p.state + ((long long)slot * p.heads + h) * p.dim * p.state_cols;
  float2 S[kRows / 2][kCols];   // row pairs
  const bool mine = c0 < p.state_cols;
#pragma unroll
  for (int j = 0; j < kChunks; ++j) {
    const int r = j * 32 + rl * 4;
    float f[4][kCols];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
#pragma unroll
      for (int c = 0; c < kCols; ++c) f[i][c] = 0.f;
      if (start > 0 && mine && r + i < p.dim) {
        const float* src = state + (long long)(r + i) * p.state_cols + c0;
        if constexpr (kCols == 4) {
          const float4 v = load4(src);
          f[i][0] = v.x; f[i][1] = v.y; f[i][2] = v.z; f[i][3] = v.w;
        } else {
          const float2 v = *reinterpret_cast<const float2*>(src);
          f[i][0] = v.x; f[i][1] = v.y;
        }
      }
    }
#pragma unroll
    for (int c = 0; c < kCols; ++c) {
      S[2 * j][c] = make_float2(f[0][c], f[1][c]);
      S[2 * j + 1][c] = make_float2(f[2][c], f[3][c]);
    }
  }
  if (!DELTA && tid == 0)
    sMax[TT] = start > 0 ? p.max_state[((long long)slot * 2 + phase) * p.heads + h] : 0.f;

  // ---- inputs: the projection's value of a channel at token t of this step (t < 0: earlier)
  const int back = DELTA ? p.taps - 1 : 0;
  const T* old_inputs = DELTA ? reinterpret_cast<const T*>(p.conv_state) +
                                    ((long long)slot * 2 + phase) * back * p.channels
                              : nullptr;
  auto raw1 = [&](int t, int col, int ch) -> float {
    if (t >= 0) return to_f32<T>(proj[(first + t) * p.ld + col]);
    return start + t >= 0 ? to_f32<T>(old_inputs[(long long)(back + t) * p.channels + ch]) : 0.f;
  };
  auto raw4 = [&](int t, int col, int ch) -> float4 {
    if (t >= 0) return load4(proj + (first + t) * p.ld + col);
    return start + t >= 0 ? load4(old_inputs + (long long)(back + t) * p.channels + ch)
                          : make_float4(0.f, 0.f, 0.f, 0.f);
  };
  const int q_col = p.q_at + hk * p.dim, k_col = p.k_at + hk * p.dim, v_col = p.v_at + hv * p.vdim;
  const int q_ch = hk * p.dim, k_ch = (p.heads / p.group + hk) * p.dim;
  const int v_ch = 2 * (p.heads / p.group) * p.dim + hv * p.vdim;
  const int nv = min(nc, p.vdim - c_first);   // value columns of this block (the rest: zeros or 1)

  for (int t0 = 0; t0 < n; t0 += TT) {
    const int nt = min(TT, n - t0);
    __syncthreads();   // the last tile's outputs have been read
    // ---- 1. queries, keys and values (convolved)
    {
      const int step4 = p.vec ? 4 : 1;
      const int per = (2 * DP + nc) / step4;
      for (int it = tid; it < TT * per; it += threads) {
        const int t = it / per, x = (it - t * per) * step4;
        const int part = x < DP ? 0 : x < 2 * DP ? 1 : 2;
        const int d = part == 0 ? x : part == 1 ? x - DP : x - 2 * DP;
        const int limit = part == 2 ? nv : p.dim;
        const int col = (part == 0 ? q_col : part == 1 ? k_col : v_col + c_first) + d;
        const int ch = (part == 0 ? q_ch : part == 1 ? k_ch : v_ch + c_first) + d;
        float* dst = (part == 0 ? sC + t * DP : part == 1 ? sB + t * DP : sV + t * nc) + d;
        if (p.vec) {
          float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
          if (t < nt && d < limit) {
            if (DELTA) {
              for (int j = 0; j < p.taps; ++j) {
                const float4 w = load4(p.conv + (long long)j * p.channels + ch);
                const float4 v = raw4(t0 + t - back + j, col, ch);
                y.x = fmaf(w.x, v.x, y.x); y.y = fmaf(w.y, v.y, y.y);
                y.z = fmaf(w.z, v.z, y.z); y.w = fmaf(w.w, v.w, y.w);
              }
              y = make_float4(silu_f(y.x), silu_f(y.y), silu_f(y.z), silu_f(y.w));
            } else {
              y = raw4(t0 + t, col, 0);
            }
          }
          if (!DELTA && part == 2) {   // the normaliser's column
            const int one = p.vdim - c_first - d;
            if (one == 0) y.x = 1.f;
            if (one == 1) y.y = 1.f;
            if (one == 2) y.z = 1.f;
            if (one == 3) y.w = 1.f;
          }
          store4(dst, y);
        } else {
          float y = 0.f;
          if (t < nt && d < limit) {
            if (DELTA) {
              for (int j = 0; j < p.taps; ++j)
                y = fmaf(p.conv[(long long)j * p.channels + ch], raw1(t0 + t - back + j, col, ch), y);
              y = silu_f(y);
            } else {
              y = raw1(t0 + t, col, 0);
            }
          }
          if (!DELTA && part == 2 && d == p.vdim - c_first) y = 1.f;
          *dst = y;
        }
      }
    }
    if (!DELTA && tid < 32) {
      // m' = max(f + m, i) of the tile's tokens one after the other; lane t holds token t's logs
      float gi = 0.f, gf = 0.f;
      if (lane < nt) {
        const T* r = proj + (first + t0 + lane) * p.ld;
        gi = p.cap * tanhf((to_f32<T>(r[p.i_at + h]) + p.i_bias[h]) / p.cap);
        const float z = p.cap * tanhf((to_f32<T>(r[p.f_at + h]) + p.f_bias[h]) / p.cap);
        gf = fminf(z, 0.f) - log1pf(expf(-fabsf(z)));
      }
      float m = sMax[TT], cum = 0.f;
      for (int t = 0; t < nt; ++t) {
        const float i = __shfl_sync(0xffffffffu, gi, t), f = __shfl_sync(0xffffffffu, gf, t);
        const float m_new = fmaxf(f + m, i);
        cum += fmaxf(f + m - m_new, kMinLogDecay);
        if (lane == 0) {
          sBeta[t] = i - m_new;
          invQ[t] = cum;
          sMax[t] = m_new;
        }
        m = m_new;
      }
      if (lane == 0) {
        for (int t = nt; t < TT; ++t) {
          sBeta[t] = 0.f;
          invQ[t] = cum;
        }
        sMax[TT] = m;
      }
    }
    __syncthreads();
    // ---- 2. unit length, step sizes
    if (DELTA) {
      for (int t = warp; t < TT; t += warps) {
        float a = 0.f, b = 0.f;
        for (int d = lane; d < DP; d += 32) {
          const float q = sC[t * DP + d], k = sB[t * DP + d];
          a = fmaf(q, q, a);
          b = fmaf(k, k, b);
        }
        a = warp_sum(a);
        b = warp_sum(b);
        if (lane == 0) {
          invQ[t] = p.q_scale / sqrtf(a + 1e-6f);
          invK[t] = 1.f / sqrtf(b + 1e-6f);
          sBeta[t] = t < nt ? 1.f / (1.f + expf(-to_f32<T>(proj[(first + t0 + t) * p.ld + p.b_at + h])))
                            : 0.f;
        }
      }
      __syncthreads();
    }
    // ---- 3. decays; a, b, c
    bool strong = false;
    if (DELTA) {
      // a thread owns a channel (blocks of fewer threads than channels: several, one after the
      // other); its cumulative logs of the tile go through sA
      bool deep = false;
      for (int d = tid; d < DP; d += threads) {
        float cum = 0.f;
        if (d < p.dim) {
          const T* z = reinterpret_cast<const T*>(p.decay) + (first + t0) * p.ld_decay + h * p.dim + d;
          const float ae = p.a_exp[h], bias = p.dt_bias[h * p.dim + d];
          float raw[TT];
#pragma unroll
          for (int t = 0; t < TT; ++t) raw[t] = t < nt ? to_f32<T>(z[(long long)t * p.ld_decay]) : 0.f;
#pragma unroll
          for (int t = 0; t < TT; ++t) {
            if (t < nt) cum += fmaxf(-ae * softplus_f(raw[t] + bias), kMinLogDecay);
            sA[t * DP + d] = cum;
          }
        } else {
          for (int t = 0; t < TT; ++t) sA[t * DP + d] = 0.f;
        }
        deep |= cum < kTileLogDecay;
      }
      strong = TT > B && __syncthreads_or(deep);
      for (int d = tid; d < DP; d += threads) {
        float base = 0.f;
        for (int t = 0; t < TT; ++t) {
          const float cum = sA[t * DP + d] - base;
          const float g = __expf(cum), k = sB[t * DP + d] * invK[t];
          sA[t * DP + d] = k * g;
          sB[t * DP + d] = k * __expf(-cum);
          sC[t * DP + d] *= invQ[t] * g;
          if (t % B == B - 1) {
            sG[t / B * DP + d] = g;
            if (strong) base += cum;
          }
        }
      }
    } else {
      strong = TT > B && invQ[TT - 1] < kTileLogDecay;
      for (int it = tid; it < TT * DP; it += threads) {
        const int t = it / DP;
        const float base = strong && t >= B ? invQ[t / B * B - 1] : 0.f;
        const float cum = invQ[t] - base;
        sB[it] *= __expf(sBeta[t] - cum);
        sC[it] *= p.q_scale * __expf(cum);
        if (t % B == B - 1) sG[t / B * DP + it - t * DP] = __expf(cum);
      }
    }
    __syncthreads();
    // ---- 4. scalar products within groups of B tokens
    for (int i = warp; i < TT; i += warps) {
      const int g0 = i / B * B;
      float a[B], c[B];
#pragma unroll
      for (int j = 0; j < B; ++j) a[j] = c[j] = 0.f;
      for (int d = lane; d < DP; d += 32) {
        const float ai = DELTA ? sA[i * DP + d] : 0.f, ci = sC[i * DP + d];
#pragma unroll
        for (int j = 0; j < B; ++j) {
          const float b = sB[(g0 + j) * DP + d];
          if (DELTA) a[j] = fmaf(ai, b, a[j]);
          c[j] = fmaf(ci, b, c[j]);
        }
      }
#pragma unroll
      for (int j = 0; j < B; ++j) {
        const float x = DELTA ? warp_sum(a[j]) : 0.f, y = warp_sum(c[j]);
        if (lane == 0) {
          dotB[i * B + j] = x;
          dotC[i * B + j] = y;
        }
      }
    }
    __syncthreads();
    // ---- 5. the recurrence
    if (c_local < nc) {
      for (int g0 = 0; g0 < nt; g0 += B) {
        constexpr int kKinds = DELTA ? 2 : 1;
        float2 acc[kKinds][kCols][B];
#pragma unroll
        for (int e = 0; e < kKinds; ++e)
#pragma unroll
          for (int c = 0; c < kCols; ++c)
#pragma unroll
            for (int i = 0; i < B; ++i) acc[e][c][i] = make_float2(0.f, 0.f);
#pragma unroll
        for (int j = 0; j < kChunks; ++j) {
          const int r = j * 32 + rl * 4;
#pragma unroll
          for (int i = 0; i < B; ++i) {
            const float4 vc = load4(sC + (g0 + i) * DP + r);
            if constexpr (DELTA) {
              const float4 va = load4(sA + (g0 + i) * DP + r);
#pragma unroll
              for (int c = 0; c < kCols; ++c) {
                fma2(acc[0][c][i], S[2 * j][c], make_float2(va.x, va.y));
                fma2(acc[0][c][i], S[2 * j + 1][c], make_float2(va.z, va.w));
              }
            }
#pragma unroll
            for (int c = 0; c < kCols; ++c) {
              fma2(acc[kKinds - 1][c][i], S[2 * j][c], make_float2(vc.x, vc.y));
              fma2(acc[kKinds - 1][c][i], S[2 * j + 1][c], make_float2(vc.z, vc.w));
            }
          }
        }
        // Sums over the eight lanes of a column: each exchange halves what a lane still carries, so
        // that in the end it has one kind (delta: lanes 0 - 3 Z^T a, 4 - 7 Z^T c) of one column.
        float my[B];
        int my_c;
        if constexpr (DELTA) {
          float v[kCols][B];
          const bool hi = lane & 4;
#pragma unroll
          for (int c = 0; c < kCols; ++c)
#pragma unroll
            for (int i = 0; i < B; ++i) {
              const float x = acc[0][c][i].x + acc[0][c][i].y, y = acc[1][c][i].x + acc[1][c][i].y;
              const float got = __shfl_xor_sync(0xffffffffu, hi ? x : y, 4);
              v[c][i] = (hi ? y : x) + got;
            }
          if constexpr (kCols == 4) {
            const bool c2 = lane & 2, c1 = lane & 1;
            float w[2][B];
#pragma unroll
            for (int c = 0; c < 2; ++c)
#pragma unroll
              for (int i = 0; i < B; ++i) {
                const float got = __shfl_xor_sync(0xffffffffu, c2 ? v[c][i] : v[c + 2][i], 2);
                w[c][i] = (c2 ? v[c + 2][i] : v[c][i]) + got;
              }
#pragma unroll
            for (int i = 0; i < B; ++i) {
              const float got = __shfl_xor_sync(0xffffffffu, c1 ? w[0][i] : w[1][i], 1);
              my[i] = (c1 ? w[1][i] : w[0][i]) + got;
            }
            my_c = lane & 3;
          } else {
            const bool c1 = lane & 1;
#pragma unroll
            for (int i = 0; i < B; ++i) {
              const float got = __shfl_xor_sync(0xffffffffu, c1 ? v[0][i] : v[1][i], 1);
              const float x = (c1 ? v[1][i] : v[0][i]) + got;
              my[i] = x + __shfl_xor_sync(0xffffffffu, x, 2);
            }
            my_c = lane & 1;
          }
        } else {
          if constexpr (kCols == 4) {
            const bool c2 = lane & 2, c1 = lane & 1;
            float w[2][B];
#pragma unroll
            for (int c = 0; c < 2; ++c)
#pragma unroll
              for (int i = 0; i < B; ++i) {
                const float x = acc[0][c][i].x + acc[0][c][i].y, y = acc[0][c + 2][i].x + acc[0][c + 2][i].y;
                const float got = __shfl_xor_sync(0xffffffffu, c2 ? x : y, 2);
                w[c][i] = (c2 ? y : x) + got;
              }
#pragma unroll
            for (int i = 0; i < B; ++i) {
              const float got = __shfl_xor_sync(0xffffffffu, c1 ? w[0][i] : w[1][i], 1);
              const float x = (c1 ? w[1][i] : w[0][i]) + got;
              my[i] = x + __shfl_xor_sync(0xffffffffu, x, 4);
            }
            my_c = lane & 3;
          } else {
            const bool c1 = lane & 1;
#pragma unroll
            for (int i = 0; i < B; ++i) {
              const float a = acc[0][0][i].x + acc[0][0][i].y, b = acc[0][1][i].x + acc[0][1][i].y;
              const float got = __shfl_xor_sync(0xffffffffu, c1 ? a : b, 1);
              float x = (c1 ? b : a) + got;
              x += __shfl_xor_sync(0xffffffffu, x, 2);
              my[i] = x + __shfl_xor_sync(0xffffffffu, x, 4);
            }
            my_c = lane & 1;
          }
        }
        // u of every token and column; o
        float u[B];
#pragma unroll
        for (int i = 0; i < B; ++i) {
          const float v = sV[(g0 + i) * nc + c_local + my_c];
          u[i] = v;
          if constexpr (DELTA) {
            float x = v - my[i];
#pragma unroll
            for (int j = 0; j < B; ++j)
              if (j < i) x = fmaf(-dotB[(g0 + i) * B + j], u[j], x);
            u[i] = sBeta[g0 + i] * x;   // (of use in lanes 0 - 3)
          }
        }
        float U[B][kCols];
        if constexpr (DELTA) {
#pragma unroll
          for (int i = 0; i < B; ++i) {
#pragma unroll
            for (int c = 0; c < kCols; ++c) U[i][c] = __shfl_sync(0xffffffffu, u[i], (lane & 24) | c);
            u[i] = __shfl_sync(0xffffffffu, u[i], (lane & 24) | my_c);
          }
        } else {
#pragma unroll
          for (int i = 0; i < B; ++i)
#pragma unroll
            for (int c = 0; c < kCols; ++c) U[i][c] = sV[(g0 + i) * nc + c_local + c];
        }
        __syncwarp();   // the values of these tokens have been read: the outputs take their place
#pragma unroll
        for (int i = 0; i < B; ++i) {
          float o = my[i];
#pragma unroll
          for (int j = 0; j < B; ++j)
            if (j <= i) o = fmaf(dotC[(g0 + i) * B + j], u[j], o);
          if (rl >= 4 && rl < 4 + kCols) sV[(g0 + i) * nc + c_local + my_c] = o;
        }
        const bool renorm = strong || g0 + B >= nt;
        const float* ge = sG + (strong ? g0 / B : TT / B - 1) * DP;
#pragma unroll
        for (int j = 0; j < kChunks; ++j) {
          const int r = j * 32 + rl * 4;
#pragma unroll
          for (int i = 0; i < B; ++i) {
            const float4 b = load4(sB + (g0 + i) * DP + r);
#pragma unroll
            for (int c = 0; c < kCols; ++c) {
              const float2 uu = make_float2(U[i][c], U[i][c]);
              fma2(S[2 * j][c], make_float2(b.x, b.y), uu);
              fma2(S[2 * j + 1][c], make_float2(b.z, b.w), uu);
            }
          }
          if (renorm) {
            const float4 g = load4(ge + r);
#pragma unroll
            for (int c = 0; c < kCols; ++c) {
              mul2(S[2 * j][c], make_float2(g.x, g.y));
              mul2(S[2 * j + 1][c], make_float2(g.z, g.w));
            }
          }
        }
      }
    }
    __syncthreads();
    // ---- 6. outputs
    for (int t = warp; t < nt; t += warps) {
      const float* o = sV + t * nc;
      const long long row = first + t0 + t;
      if (p.raw != nullptr) {
        float* dst = p.raw + (row * p.heads + h) * p.raw_cols + c_first;
        for (int c = lane; c < min(nc, p.ncols - c_first); c += 32) dst[c] = o[c];
        if (!DELTA && slice == 0 && lane == 0) dst[p.ncols] = expf(-sMax[t]);
        continue;
      }
      float scale = 1.f, ss = 0.f;
      if (!DELTA) scale = 1.f / (fmaxf(fabsf(o[p.vdim]), expf(-sMax[t])) + 1e-6f);
      for (int c = lane; c < p.vdim; c += 32) {
        const float x = o[c] * scale;
        ss = fmaf(x, x, ss);
      }
      scale *= 1.f / sqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
      const T* g = reinterpret_cast<const T*>(p.gate) + row * p.ld_gate + (long long)h * p.vdim;
      const float* w = p.norm + (long long)h * p.norm_step;
      T* dst = reinterpret_cast<T*>(p.out) + row * p.ldo + (long long)h * p.vdim;
      for (int c = lane; c < p.vdim; c += 32)
        dst[c] = from_f32<T>(o[c] * scale * w[c] * sigmoid_f(to_f32<T>(g[c])));
    }
  }

  // ---- what the sequence's next step starts from
#pragma unroll
  for (int j = 0; j < kChunks; ++j) {
    const int r = j * 32 + rl * 4;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      if (!mine || c_local >= nc || r + i >= p.dim) continue;
      float* dst = state + (long long)(r + i) * p.state_cols + c0;
      auto at = [&](int c) { return (i & 1) ? S[2 * j + i / 2][c].y : S[2 * j + i / 2][c].x; };
      if constexpr (kCols == 4)
        store4(dst, make_float4(at(0), at(1), at(2), at(3)));
      else
        *reinterpret_cast<float2*>(dst) = make_float2(at(0), at(1));
    }
  }
  if (DELTA) {
    T* next = reinterpret_cast<T*>(p.conv_state) + ((long long)slot * 2 + (phase ^ 1)) * back * p.channels;
    const bool qk = slice == 0 && h % p.group == 0;
    for (int it = tid; it < back * (2 * p.dim + nv); it += threads) {
      const int j = it / (2 * p.dim + nv), x = it - j * (2 * p.dim + nv);
      if (x < 2 * p.dim && !qk) continue;
      const int col = x < p.dim ? q_col + x : x < 2 * p.dim ? k_col + x - p.dim : v_col + c_first + x - 2 * p.dim;
      const int ch = x < p.dim ? q_ch + x : x < 2 * p.dim ? k_ch + x - p.dim : v_ch + c_first + x - 2 * p.dim;
      next[(long long)j * p.channels + ch] = from_f32<T>(raw1(n - back + j, col, ch));
    }
  } else if (slice == 0 && tid == 0) {
    p.max_state[((long long)slot * 2 + (phase ^ 1)) * p.heads + h] = sMax[TT];
  }
}

// Heads whose columns several blocks share: norm, weight and gate of the raw outputs. A warp per
// (token, head).
template <typename T, bool DELTA>
__global__ void __launch_bounds__(256) scan_output_kernel(const ScanArgs p, long long n) {
  pdl_wait();
  pdl_trigger();
  const long long k = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (k >= n) return;
  const long long row = k / p.heads;
  const int h = (int)(k - row * p.heads);
  const float* o = p.raw + k * p.raw_cols;
  float scale = 1.f, ss = 0.f;
  if (!DELTA) scale = 1.f / (fmaxf(fabsf(o[p.vdim]), o[p.vdim + 1]) + 1e-6f);
  for (int c = lane; c < p.vdim; c += 32) {
    const float x = o[c] * scale;
    ss = fmaf(x, x, ss);
  }
  scale *= 1.f / sqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
  const T* g = reinterpret_cast<const T*>(p.gate) + row * p.ld_gate + (long long)h * p.vdim;
  const float* w = p.norm + (long long)h * p.norm_step;
  T* dst = reinterpret_cast<T*>(p.out) + row * p.ldo + (long long)h * p.vdim;
  for (int c = lane; c < p.vdim; c += 32)
    dst[c] = from_f32<T>(o[c] * scale * w[c] * sigmoid_f(to_f32<T>(g[c])));
}

template <typename T, int DP, int TT, int B, bool DELTA>
static int launch_scan(ScanArgs a, int n_seq, cudaStream_t stream) {
  constexpr int wc = ScanShape<DP>::kWarpCols;
  a.nc = (a.ncols + a.slices - 1) / a.slices;
  a.nc = (a.nc + wc - 1) / wc * wc;
  if (a.nc / wc > kScanMaxWarps || (long long)a.nc * (a.slices - 1) >= a.ncols) return -2;
  const size_t smem = (size_t)ScanSmem<DP, TT, B, DELTA>::total(a.nc) * sizeof(float);
  if (smem > 220 * 1024) return -6;
  auto k = scan_kernel<T, DP, TT, B, DELTA>;
  if (smem > 48 * 1024 &&
      cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return -3;
  const long long blocks = (long long)n_seq * a.heads * a.slices;
  if (blocks > 0x7fffffffll) return -6;
  return launch_pdl(k, dim3((unsigned)blocks), dim3(a.nc / wc * 32), smem, stream, a) == cudaSuccess ? 0 : -5;
}

template <typename T, bool DELTA>
static int run_scan(ScanArgs a, int n_seq, int max_rows, long long rows, cudaStream_t stream) {
  int rc = -6;
#define AB200_SCAN(DP)                                                             \
  rc = max_rows == 1 ? launch_scan<T, DP, 1, 1, DELTA>(a, n_seq, stream)           \
                     : launch_scan<T, DP, 16, 4, DELTA>(a, n_seq, stream)
  if (a.dim <= 32) AB200_SCAN(32);
  else if (a.dim <= 64) AB200_SCAN(64);
  else if (a.dim <= 128) AB200_SCAN(128);
  else if (a.dim <= 256) AB200_SCAN(256);
#undef AB200_SCAN
  if (rc != 0 || a.raw == nullptr) return rc;
  const long long n = rows * a.heads;
  return launch_pdl(scan_output_kernel<T, DELTA>, dim3((unsigned)((n + 7) / 8)), dim3(256), 0, stream, a,
                    n) == cudaSuccess
             ? 0
             : -5;
}

static int aligned4(const void* p, long long ld, int dtype) {
  return ld % 4 == 0 && (reinterpret_cast<uintptr_t>(p) & (dtype == 0 ? 7 : 15)) == 0;
}

}  // namespace ab200

using namespace ab200;
typedef __nv_bfloat16 bf16;

extern "C" {

// Blocks per head so that each block's columns fit: 0 if dim is beyond the kernel's.
int ab200_scan_min_slices(int dim, int ncols) {
  if (dim < 1 || dim > 256) return 0;
  const int most = kScanMaxWarps * (dim <= 128 ? 16 : 8);
  return (ncols + most - 1) / most;
}

// Gated delta rule over n_seq sequences. proj [T, ld]: query and key heads of dim at q_at, k_at, value
// heads of vdim at v_at, step sizes at b_at. steps int32 [n_seq, 5]: first row, rows, slot (0: padding),
// start position, phase. raw fp32 [T, heads, vdim] when slices > 1. See ScanArgs.
int ab200_delta_scan(const void* proj, long long ld, int q_at, int k_at, int v_at, int b_at,
                     const void* decay, long long ld_decay, const void* gate, long long ld_gate,
                     const void* conv, int taps, const void* a_exp, const void* dt_bias,
                     const void* norm, void* state, int state_cols, void* conv_state, int num_slots,
                     const void* steps, int n_seq, int max_rows, long long T, int heads, int kv_heads,
                     int dim, int vdim, int slices, float eps, void* raw, void* out, long long ldo,
                     int dtype, int* status, cudaStream_t stream) {
  if (T <= 0 || n_seq <= 0) return 0;
  if (heads < 1 || kv_heads < 1 || heads % kv_heads || dim < 1 || vdim < 1 || taps < 1 || slices < 1 ||
      state_cols < vdim || state_cols % 4 || (slices > 1 && raw == nullptr))
    return -2;
  ScanArgs a = {};
  a.proj = proj; a.ld = ld;
  a.q_at = q_at; a.k_at = k_at; a.v_at = v_at; a.b_at = b_at;
  a.decay = decay; a.ld_decay = ld_decay;
  a.gate = gate; a.ld_gate = ld_gate;
  a.conv = reinterpret_cast<const float*>(conv);
  a.a_exp = reinterpret_cast<const float*>(a_exp);
  a.dt_bias = reinterpret_cast<const float*>(dt_bias);
  a.norm = reinterpret_cast<const float*>(norm);
  a.state = reinterpret_cast<float*>(state);
  a.state_cols = state_cols;
  a.conv_state = conv_state;
  a.num_slots = num_slots;
  a.steps = reinterpret_cast<const int*>(steps);
  a.heads = heads; a.group = heads / kv_heads; a.dim = dim; a.vdim = vdim; a.ncols = vdim;
  a.taps = taps;
  a.channels = 2 * kv_heads * dim + heads * vdim;
  a.slices = slices;
  a.q_scale = 1.f / sqrtf((float)dim);
  a.eps = eps;
  a.raw = slices > 1 ? reinterpret_cast<float*>(raw) : nullptr;
  a.raw_cols = vdim;
  a.out = out; a.ldo = ldo;
  a.status = status;
  a.vec = dim % 4 == 0 && vdim % 4 == 0 && q_at % 4 == 0 && k_at % 4 == 0 && v_at % 4 == 0 &&
          aligned4(proj, ld, dtype) && aligned4(conv_state, 0, dtype) && aligned4(conv, 0, 1);
  return dtype == 0 ? run_scan<bf16, true>(a, n_seq, max_rows, T, stream)
                    : run_scan<float, true>(a, n_seq, max_rows, T, stream);
}

// Matrix memory: query and key heads of dim, value heads of vdim, gates at i_at and f_at; state
// [slots, heads, dim, state_cols] with the normaliser in column vdim; max_state fp32 [slots, 2, heads];
// raw fp32 [T, heads, vdim + 2] when slices > 1.
int ab200_memory_scan(const void* proj, long long ld, int q_at, int k_at, int v_at, int i_at, int f_at,
                      const void* gate, long long ld_gate, const void* i_bias, const void* f_bias,
                      float cap, const void* norm, void* state, int state_cols, void* max_state,
                      int num_slots, const void* steps, int n_seq, int max_rows, long long T, int heads,
                      int dim, int vdim, int slices, float eps, void* raw, void* out, long long ldo,
                      int dtype, int* status, cudaStream_t stream) {
  if (T <= 0 || n_seq <= 0) return 0;
  if (heads < 1 || dim < 1 || vdim < 1 || slices < 1 || state_cols < vdim + 1 || state_cols % 4 ||
      !(cap > 0.f) || (slices > 1 && raw == nullptr))
    return -2;
  ScanArgs a = {};
  a.proj = proj; a.ld = ld;
  a.q_at = q_at; a.k_at = k_at; a.v_at = v_at; a.i_at = i_at; a.f_at = f_at;
  a.gate = gate; a.ld_gate = ld_gate;
  a.i_bias = reinterpret_cast<const float*>(i_bias);
  a.f_bias = reinterpret_cast<const float*>(f_bias);
  a.cap = cap;
  a.norm = reinterpret_cast<const float*>(norm);
  a.norm_step = vdim;
  a.state = reinterpret_cast<float*>(state);
  a.state_cols = state_cols;
  a.max_state = reinterpret_cast<float*>(max_state);
  a.num_slots = num_slots;
  a.steps = reinterpret_cast<const int*>(steps);
  a.heads = heads; a.group = 1; a.dim = dim; a.vdim = vdim; a.ncols = vdim + 1;
  a.taps = 1;
  a.slices = slices;
  a.q_scale = 1.f / sqrtf((float)dim);
  a.eps = eps;
  a.raw = slices > 1 ? reinterpret_cast<float*>(raw) : nullptr;
  a.raw_cols = vdim + 2;
  a.out = out; a.ldo = ldo;
  a.status = status;
  a.vec = dim % 4 == 0 && vdim % 4 == 0 && q_at % 4 == 0 && k_at % 4 == 0 && v_at % 4 == 0 &&
          aligned4(proj, ld, dtype);
  return dtype == 0 ? run_scan<bf16, false>(a, n_seq, max_rows, T, stream)
                    : run_scan<float, false>(a, n_seq, max_rows, T, stream);
}

}  // extern "C"
