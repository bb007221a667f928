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
//   forget scan     (HGRN2) a forget gate f per channel, which also decides what is written:
//                       S <- f * S + (1 - f) v^T;  o = S^T q,  q through silu
//
// They are followed by the RMS norm of each head's o, a weight and (but for the forget scan) an output
// gate. Everything that enters the recurrence is fp32, and so is its arithmetic (FMAs on pairs of rows).
//
// Steps of one token per sequence run in one kernel (step_kernel): a block owns a sequence's head, or
// some of the head's columns, which do not depend on one another.
//
// Longer portions take two. tile_kernel prepares, for tiles of 16 tokens and all of them at once, the
// vectors that the recurrence needs (convolution, norms, gates, decays) as records in memory;
// scan_kernel then walks a sequence's records with a head's part of S in registers (a lane holds DP / 8
// rows by kCols columns), four tokens at a time, the next records on their way to shared memory.
// Within a tile S is held undecayed: S = G * Z with G the product of the tile's decays so far (per
// row), so that a token costs three multiply-adds per element and not four,
//     Z^T (G k), Z^T (G q) and Z <- Z + (k / G) u^T,
// and a group of tokens needs no exchange but its scalar products: with a = G k, b = k / G, c = G q
//     u_i = beta_i (v_i - Z^T a_i - sum_{j<i} (a_i . b_j) u_j),  o_i = Z^T c_i + sum_{j<=i} (c_i . b_j) u_j
// where Z is the one before the group. G goes back to 1 at a tile's end, and after every group when a
// channel decays so much within the tile that 1 / G would leave fp32's range. (Without the delta rule u is
// the value; the forget scan's k is 1 - f, its decays f.)
//
// For 16-bit models the products of a tile run on the tensor cores (recurrent_mma.cu); 32-bit models use
// fp32 multiply-adds.
//
// What a sequence carries over lies in its slot: S in fp32; the convolution's last inputs and m twice,
// for even and odd steps of the sequence (`phase`), so that blocks which read them never race with the
// block that writes them. A sequence that starts at position 0 reads nothing from its slot.

#include "api.h"
#include "common/recurrent.cuh"

namespace ab200 {

// DP: rows (dim, zero-padded)
template <int DP>
struct ScanShape {
  static constexpr int kRows = DP / 8;                  // per lane, in chunks of four
  static constexpr int kCols = DP <= 128 ? 4 : 2;
  static constexpr int kWarpCols = 4 * kCols;
};

// A record: offsets in floats. Its values [kTT][value columns] follow.
template <int DP, bool DELTA>
struct Record {
  static constexpr int kKeys = 0, kQ = kTT * DP, kA = 2 * kTT * DP, kG = (DELTA ? 3 : 2) * kTT * DP;
  static constexpr int kDotB = kG + kTT / kB * DP, kDotC = kDotB + kTT * kB;
  static constexpr int kBeta = kDotC + kTT * kB;    // memory: exp(-m)
  static constexpr int kStrong = kBeta + kTT, kV = kStrong + 4;
};

// Lane's part of the state: rows j * 32 + rl * 4 + {0 .. 3}, kCols columns from c0, in row pairs
template <int DP>
__device__ __forceinline__ void load_state(float2 (&S)[ScanShape<DP>::kRows / 2][ScanShape<DP>::kCols],
                                           const float* state, const ScanArgs& p, int rl, int c0,
                                           bool any) {
  constexpr int kCols = ScanShape<DP>::kCols;
#pragma unroll
  for (int j = 0; j < ScanShape<DP>::kRows / 4; ++j) {
    const int r = j * 32 + rl * 4;
    float f[4][kCols];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
#pragma unroll
      for (int c = 0; c < kCols; ++c) f[i][c] = 0.f;
      if (any && c0 < p.state_cols && r + i < p.dim) {
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
}
template <int DP>
__device__ __forceinline__ void store_state(const float2 (&S)[ScanShape<DP>::kRows / 2][ScanShape<DP>::kCols],
                                            float* state, const ScanArgs& p, int rl, int c0) {
  constexpr int kCols = ScanShape<DP>::kCols;
#pragma unroll
  for (int j = 0; j < ScanShape<DP>::kRows / 4; ++j) {
    const int r = j * 32 + rl * 4;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      if (c0 >= p.state_cols || r + i >= p.dim) continue;
      float* dst = state + (long long)(r + i) * p.state_cols + c0;
      auto at = [&](int c) { return (i & 1) ? S[2 * j + i / 2][c].y : S[2 * j + i / 2][c].x; };
      if constexpr (kCols == 4)
        store4(dst, make_float4(at(0), at(1), at(2), at(3)));
      else
        *reinterpret_cast<float2*>(dst) = make_float2(at(0), at(1));
    }
  }
}

// Sums of acc over the eight lanes of a column group. Each exchange halves what a lane still carries,
// so that in the end it has one kind (two kinds: lanes 0 - 3 the first, 4 - 7 the second) of one
// column, which is returned.
template <int KINDS, int COLS, int N>
__device__ __forceinline__ int reduce_columns(const float2 (&acc)[KINDS][COLS][N], float (&my)[N]) {
  const int lane = threadIdx.x & 31;
  const bool hi = lane & 4, c2 = lane & 2, c1 = lane & 1;
  float v[COLS][N];
#pragma unroll
  for (int c = 0; c < COLS; ++c)
#pragma unroll
    for (int i = 0; i < N; ++i) {
      v[c][i] = acc[0][c][i].x + acc[0][c][i].y;
      if constexpr (KINDS == 2) {
        const float y = acc[1][c][i].x + acc[1][c][i].y;
        const float got = __shfl_xor_sync(0xffffffffu, hi ? v[c][i] : y, 4);
        v[c][i] = (hi ? y : v[c][i]) + got;
      }
    }
  float w[2][N];
#pragma unroll
  for (int c = 0; c < 2; ++c)
#pragma unroll
    for (int i = 0; i < N; ++i) {
      if constexpr (COLS == 4) {
        const float got = __shfl_xor_sync(0xffffffffu, c2 ? v[c][i] : v[c + 2][i], 2);
        w[c][i] = (c2 ? v[c + 2][i] : v[c][i]) + got;
      } else {
        w[c][i] = v[c][i];
      }
    }
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const float got = __shfl_xor_sync(0xffffffffu, c1 ? w[0][i] : w[1][i], 1);
    my[i] = (c1 ? w[1][i] : w[0][i]) + got;
    if constexpr (COLS == 2) my[i] += __shfl_xor_sync(0xffffffffu, my[i], 2);
    if constexpr (KINDS == 1) my[i] += __shfl_xor_sync(0xffffffffu, my[i], 4);
  }
  return lane & (COLS - 1);
}

// ------------------------------------------------------------------ one token per sequence
// A thread holds four neighbouring columns of kRows consecutive rows, so that a warp reads and writes
// whole rows of the state; nc / 4 threads side by side, kGroups groups of rows.
template <int DP>
struct StepShape {
  static constexpr int kGroups = DP <= 128 ? 8 : 16, kRows = DP / kGroups;
  static constexpr int max_threads(int rule) { return kGroups * max_warps(rule) * 4; }
  static constexpr int smem_floats(int nc) { return 3 * DP + nc + 2 * kGroups * nc; }
};

template <typename T, int DP, int RULE>
__global__ void __launch_bounds__(StepShape<DP>::max_threads(RULE), DP <= 128 ? 2 : 1)
step_kernel(const ScanArgs p) {
  using Sh = StepShape<DP>;
  constexpr bool DELTA = RULE == kDelta, MEMORY = RULE == kMemory, FORGET = RULE == kForget;
  constexpr int kRows = Sh::kRows;
  extern __shared__ __align__(16) float sm[];
  float* sQ = sm;              // query, key (before their norms), decay, values / outputs
  float* sK = sm + DP;
  float* sG = sm + 2 * DP;
  float* sV = sm + 3 * DP;
  float* sP = sV + p.nc;       // [kGroups][nc]: S^T k of a group's rows; then what is put
  float* sR = sP + Sh::kGroups * p.nc;   // S^T q
  pdl_wait();
  pdl_trigger();
  const int slice = blockIdx.x % p.slices, h = blockIdx.x / p.slices % p.heads;
  const Seq s(p.steps + (long long)(blockIdx.x / p.slices / p.heads) * kStepInts);
  if (s.n <= 0) return;
  if (s.slot <= 0 || s.slot >= p.num_slots) {
    put_zeros<T, RULE>(p, s, h, slice);
    return;
  }
  const int tid = threadIdx.x, threads = blockDim.x, lane = tid & 31;
  const int quads = p.nc / 4, group = tid / quads, c_local = (tid - group * quads) * 4;
  const int c_first = slice * p.nc, r0 = group * kRows;
  float* state = p.state + ((long long)s.slot * p.heads + h) * p.dim * p.state_cols +
                 (long long)r0 * p.state_cols + c_first + c_local;
  const bool mine = c_first + c_local < p.state_cols;
  float4 S[kRows];
  const int rows = mine ? p.dim - r0 : 0, rows_in = s.start > 0 ? rows : 0;   // of the thread's, in use
  float* row = state;
#pragma unroll
  for (int i = 0; i < kRows; ++i, row += p.state_cols)
    S[i] = i < rows_in ? load4(row) : make_float4(0.f, 0.f, 0.f, 0.f);

  const Inputs<T> in(p, s, h, DELTA);
  const int nv = min(p.nc, p.vdim - c_first);
  float keep = 0.f, put = 0.f, m_new = 0.f, beta = 0.f, a_exp = 0.f;
  if (DELTA) {
    a_exp = p.a_exp[h];
    beta = sigmoid_f(to_f32<T>(in.proj[p.b_at + h]));
  } else if (MEMORY) {
    const float2 g = memory_log_gates(to_f32<T>(in.proj[p.i_at + h]) + p.i_bias[h],
                                      to_f32<T>(in.proj[p.f_at + h]) + p.f_bias[h], p.cap);
    const float m = s.start > 0 ? p.max_state[((long long)s.slot * 2 + s.phase) * p.heads + h] : 0.f;
    m_new = fmaxf(g.y + m, g.x);
    keep = expf(g.y + m - m_new);
    put = expf(g.x - m_new);
  }
  // a thread's output columns: gate and norm weight, ahead
  const T* gate = reinterpret_cast<const T*>(p.gate) + s.first * p.ld_gate + (long long)h * p.vdim;
  const float* norm = p.norm + (long long)h * p.norm_step;
  T gate0 = from_f32<T>(0.f);
  float norm0 = 0.f;
  if (p.raw == nullptr && tid < p.vdim) {
    if (!FORGET) gate0 = gate[tid];
    norm0 = norm[tid];
  }
  // a channel a thread and turn, two turns' loads at once
  const bool qk_block = DELTA && slice == 0 && h % p.group == 0;   // saves the queries' and keys' inputs
  T* next = reinterpret_cast<T*>(p.conv_state) + ((long long)s.slot * 2 + (s.phase ^ 1)) * in.back * p.channels;
  struct Channel {   // the inputs as they lie in memory: earlier ones, the token's own
    T old[kTaps - 1], x, z;
    float w[kTaps], bias;
  };
  const T* decay = reinterpret_cast<const T*>(p.decay) + s.first * p.ld_decay + h * p.dim;
  const long long last_tap = (long long)in.back * p.channels;
  constexpr int kKeyed = FORGET ? DP : 2 * DP;   // (the forget scan's keys come with the queries)
  const int channels = kKeyed + p.nc;
  auto place = [&](int x, int& part, int& d) {
    part = x < DP ? 0 : x < kKeyed ? 1 : 2;
    d = part == 2 ? x - kKeyed + c_first : x - part * DP;
    return x < channels && (part == 2 ? d < c_first + nv : d < p.dim);
  };
  auto fetch = [&](int x, Channel& c) {
    int part, d;
    if (!place(x, part, d)) return;
    if (DELTA) {
      const float* w = p.conv + in.ch(part) + d;
      const T* o = in.old + in.ch(part) + d;
      c.x = in.proj[in.col(part) + d];
      c.w[kTaps - 1] = w[last_tap];
#pragma unroll
      for (int j = 0; j < kTaps - 1; ++j, w += p.channels, o += p.channels) {
        c.w[j] = j < in.back ? *w : 0.f;
        c.old[j] = j < in.back && s.start + j >= in.back ? *o : from_f32<T>(0.f);
      }
      if (part == 0) {
        c.z = decay[d];
        c.bias = p.dt_bias[h * p.dim + d];
      }
    } else {
      c.x = in.proj[in.col(part) + d];
      if (FORGET && part == 0) {
        c.z = decay[d];
        c.bias = p.dt_bias[h * p.dim + d];
        c.w[0] = p.lower[h * p.dim + d];
      }
    }
  };
  auto finish = [&](int x, const Channel& c) {
    int part, d;
    const bool ok = place(x, part, d);
    if (x >= channels) return;
    float y = 0.f;
    if (DELTA && ok) {
      y = c.w[kTaps - 1] * to_f32<T>(c.x);
#pragma unroll
      for (int j = 0; j < kTaps - 1; ++j) y = fmaf(c.w[j], to_f32<T>(c.old[j]), y);
      if (p.taps > kTaps) {   // (the first ones are there)
        const float* w = p.conv + in.ch(part) + d;
        for (int j = kTaps - 1; j < in.back; ++j)
          y = fmaf(w[(long long)j * p.channels], in.one(part, d, j - in.back), y);
      } else if (part == 2 || qk_block) {
        T* o = next + in.ch(part) + d;
#pragma unroll
        for (int j = 0; j < kTaps - 1; ++j, o += p.channels)
          if (j < in.back) *o = j == in.back - 1 ? c.x : c.old[j + 1 < kTaps - 1 ? j + 1 : j];
      }
      y = silu_f(y);
    } else if (MEMORY) {
      y = ok ? to_f32<T>(c.x) : part == 2 && d == p.vdim ? 1.f : 0.f;
    } else if (FORGET) {
      y = ok ? to_f32<T>(c.x) : 0.f;
      if (part == 0) {
        const float z = ok ? to_f32<T>(c.z) + c.bias : 0.f;
        y = silu_f(y);
        sG[d] = ok ? forget_keep(z, c.w[0]) : 1.f;
        sK[d] = ok ? forget_put(z, c.w[0]) : 0.f;
      }
    }
    if (DELTA && part == 0) sG[d] = ok ? exp2_fast(-kLog2e * a_exp * softplus_f(to_f32<T>(c.z) + c.bias)) : 1.f;
    (part == 0 ? sQ : part == 1 ? sK : sV)[part == 2 ? d - c_first : d] = y;
  };
  for (int x = tid; x < channels; x += 2 * threads) {
    Channel a, b;
    fetch(x, a);
    fetch(x + threads, b);
    finish(x, a);
    finish(x + threads, b);
  }
  __syncthreads();
  // every warp: norms and the product of query and key
  float qq = 0.f, kk = 0.f, qk = 0.f;
  for (int d = lane; d < DP; d += 32) {
    const float q = sQ[d], k = sK[d];
    qq = fmaf(q, q, qq);
    kk = fmaf(k, k, kk);
    qk = fmaf(q, k, qk);
  }
  qk = warp_sum(qk);
  float fq = p.q_scale, fk = 1.f;
  if (DELTA) {
    fq /= sqrtf(warp_sum(qq) + 1e-6f);
    fk = 1.f / sqrtf(warp_sum(kk) + 1e-6f);
  }
  qk *= fq * fk * (MEMORY ? put : 1.f);
  float4 P = make_float4(0.f, 0.f, 0.f, 0.f), Q = P;
#pragma unroll
  for (int i = 0; i < kRows; i += 4) {
    const float4 q = load4(sQ + r0 + i), k = load4(sK + r0 + i), g = load4(sG + r0 + i);   // (g: not memory)
    const float qs[4] = {q.x, q.y, q.z, q.w}, ks[4] = {k.x, k.y, k.z, k.w}, gs[4] = {g.x, g.y, g.z, g.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {   // S <- g * S; S^T k, S^T q
      float4& x = S[i + e];
      const float f = MEMORY ? keep : gs[e];
      x = make_float4(x.x * f, x.y * f, x.z * f, x.w * f);
      if (DELTA) axpy4(P, make_float4(ks[e], ks[e], ks[e], ks[e]), x);
      axpy4(Q, make_float4(qs[e], qs[e], qs[e], qs[e]), x);
    }
  }
  if (DELTA) store4(sP + group * p.nc + c_local, P);
  store4(sR + group * p.nc + c_local, Q);
  __syncthreads();
  for (int c = tid; c < p.nc; c += threads) {
    float pk = 0.f, o = 0.f, u = sV[c];
#pragma unroll
    for (int g = 0; g < Sh::kGroups; ++g) {
      if (DELTA) pk += sP[g * p.nc + c];
      o += sR[g * p.nc + c];
    }
    if (DELTA) u = beta * (u - fk * pk);
    sV[c] = fmaf(qk, u, fq * o);
    sP[c] = u * (MEMORY ? put : fk);   // what the rows' keys are multiplied by
  }
  __syncthreads();
  const float4 u = load4(sP + c_local);
  row = state;
#pragma unroll
  for (int i = 0; i < kRows; i += 4) {
    const float4 k = load4(sK + r0 + i);
    const float ks[4] = {k.x, k.y, k.z, k.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      axpy4(S[i + e], make_float4(ks[e], ks[e], ks[e], ks[e]), u);
      if (i + e < rows) store4(row, S[i + e]);
      row += p.state_cols;
    }
  }
  if (p.raw != nullptr) {
    float* dst = p.raw + (s.first * p.heads + h) * p.raw_cols + c_first;
    for (int c = tid; c < min(p.nc, p.ncols - c_first); c += threads) dst[c] = sV[c];
    if (MEMORY && slice == 0 && tid == 0) dst[p.ncols] = expf(-m_new);
  } else {   // every warp the norm, then its own columns
    float scale = !MEMORY ? 1.f : 1.f / (fmaxf(fabsf(sV[p.vdim]), expf(-m_new)) + 1e-6f), ss = 0.f;
    for (int c = lane; c < p.vdim; c += 32) {
      const float x = sV[c] * scale;
      ss = fmaf(x, x, ss);
    }
    scale *= 1.f / sqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
    T* dst = reinterpret_cast<T*>(p.out) + s.first * p.ldo + (long long)h * p.vdim;
    for (int c = tid; c < p.vdim; c += threads)
      dst[c] = from_f32<T>(sV[c] * scale * (c == tid ? norm0 : norm[c]) *
                           (FORGET ? 1.f : sigmoid_f(to_f32<T>(c == tid ? gate0 : gate[c]))));
  }
  if (DELTA) {
    if (p.taps > kTaps) save_inputs<T>(p, s, in, qk_block, c_first, max(0, nv));
  } else if (MEMORY && slice == 0 && tid == 0)
    p.max_state[((long long)s.slot * 2 + (s.phase ^ 1)) * p.heads + h] = m_new;
}

// ------------------------------------------------------------------ portions of several tokens
// Gates of the matrix memory: m' = max(f + m, i) composes as (F, I) -> max(F + m, I), so a block scans
// a head's tokens 1024 at a time.
template <typename T>
__global__ void __launch_bounds__(1024) memory_gates_kernel(const ScanArgs p) {
  pdl_wait();
  pdl_trigger();
  __shared__ float2 part[32];
  __shared__ float carry;
  const int h = blockIdx.x % p.heads;
  const Seq s(p.steps + (long long)(blockIdx.x / p.heads) * kStepInts);
  if (s.n <= 0 || s.slot <= 0 || s.slot >= p.num_slots) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  float m0 = s.start > 0 ? p.max_state[((long long)s.slot * 2 + s.phase) * p.heads + h] : 0.f;
  const T* proj = reinterpret_cast<const T*>(p.proj) + s.first * p.ld;
  for (int t0 = 0; t0 < s.n; t0 += blockDim.x) {
    const int t = t0 + tid;
    float2 g = make_float2(-INFINITY, 0.f);   // i, f: neither puts nor forgets
    if (t < s.n)
      g = memory_log_gates(to_f32<T>(proj[t * p.ld + p.i_at + h]) + p.i_bias[h],
                           to_f32<T>(proj[t * p.ld + p.f_at + h]) + p.f_bias[h], p.cap);
    float I = g.x, F = g.y;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float i1 = __shfl_up_sync(0xffffffffu, I, o), f1 = __shfl_up_sync(0xffffffffu, F, o);
      if (lane >= o) {
        I = fmaxf(i1 + F, I);
        F += f1;
      }
    }
    if (lane == 31) part[warp] = make_float2(I, F);
    __syncthreads();
    float m = m0;                              // the maximum before this warp's tokens
    for (int w = 0; w < warp; ++w) m = fmaxf(m + part[w].y, part[w].x);
    const float m_new = fmaxf(F + m, I);
    float m_old = __shfl_up_sync(0xffffffffu, m_new, 1);
    if (lane == 0) m_old = m;
    if (t < s.n) {
      float* dst = p.gates + ((s.first + t) * p.heads + h) * 3;
      dst[0] = fmaxf(g.y + m_old - m_new, kMinLogDecay);
      dst[1] = g.x - m_new;
      dst[2] = m_new;
    }
    if (tid == blockDim.x - 1) carry = m_new;
    __syncthreads();
    m0 = carry;
    __syncthreads();
  }
  if (tid == 0) p.max_state[((long long)s.slot * 2 + (s.phase ^ 1)) * p.heads + h] = m0;
}

// A tile's records of a head: queries, keys, values (convolved), unit lengths, decays, products.
template <typename T, int DP, int RULE>
__global__ void __launch_bounds__(DP <= 128 ? 128 : 256) tile_kernel(const ScanArgs p) {
  constexpr bool DELTA = RULE == kDelta, MEMORY = RULE == kMemory, FORGET = RULE == kForget;
  using R = Record<DP, DELTA>;
  constexpr int kThreads = DP <= 128 ? 128 : 256, kWarps = kThreads / 32;
  constexpr int kOwn = (DP + kThreads - 1) / kThreads;
  static_assert(kOwn == 1, "a thread owns a channel");
  extern __shared__ __align__(16) float sm[];
  float* sB = sm;                                // keys, then k / G
  float* sC = sm + kTT * DP;                     // queries, then G q
  float* sA = sm + 2 * kTT * DP;                 // delta: G k
  __shared__ float invQ[kTT], invK[kTT];         // memory: log decay (cumulative), log input factor
  pdl_wait();
  pdl_trigger();
  const int h = blockIdx.x % p.heads;
  const long long tile = blockIdx.x / p.heads;
  const int* tl = p.tiles + tile * 2;
  const Seq s(p.steps + (long long)tl[0] * kStepInts);
  if (s.slot <= 0 || s.slot >= p.num_slots) return;
  const int t0 = tl[1], nt = min(kTT, s.n - t0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  float* rec = p.records + (tile * p.heads + h) * p.record;
  const Inputs<T> in(p, s, h, DELTA);
  const int vcols = p.slices * p.nc;

  // this thread's channel of the decays, on its way
  float z[kTT];
  if (!MEMORY) {
    const T* src = reinterpret_cast<const T*>(p.decay) + (s.first + t0) * p.ld_decay + h * p.dim + tid;
#pragma unroll
    for (int t = 0; t < kTT; ++t)
      z[t] = tid < p.dim && t < nt ? to_f32<T>(src[(long long)t * p.ld_decay]) : 0.f;
  } else if (tid < kTT) {
    const float* g = p.gates + ((s.first + t0 + tid) * p.heads + h) * 3;
    const bool ok = tid < nt;
    invQ[tid] = ok ? g[0] : 0.f;
    invK[tid] = ok ? g[1] : 0.f;
    rec[R::kBeta + tid] = ok ? expf(-g[2]) : 1.f;
  }
  if (DELTA && tid < kTT)
    rec[R::kBeta + tid] =
        tid < nt ? sigmoid_f(to_f32<T>(in.proj[(long long)(t0 + tid) * p.ld + p.b_at + h])) : 0.f;

  // ---- 1. four channels and all of the tile's tokens a thread
  auto put = [&](int part, int d, int t, const float4& y) {
    if (part == 2) store4(rec + R::kV + t * vcols + d, y);
    else store4((part == 0 ? sC : sB) + t * DP + d, y);
  };
  for (int x = tid * 4; x < 2 * DP + vcols; x += kThreads * 4) {
    const int part = x < DP ? 0 : x < 2 * DP ? 1 : 2;
    if (FORGET && part == 1) continue;   // (keys: with the decays)
    const int d = x - part * DP, limit = part == 2 ? p.vdim : p.dim;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    if (p.vec && (!DELTA || p.taps <= kTaps)) {
      const bool ok = d < limit;
      if constexpr (DELTA) {
        float4 w[kTaps], v[kTaps + 3];
#pragma unroll
        for (int j = 0; j < kTaps; ++j) {   // the last tap is the current token's
          const int k = j - (kTaps - p.taps);
          w[j] = ok && k >= 0 ? load4(p.conv + (long long)k * p.channels + in.ch(part) + d) : zero;
        }
#pragma unroll
        for (int j = 0; j < kTaps - 1; ++j)
          v[j] = ok && j >= kTaps - p.taps ? in.four(part, d, t0 + j - (kTaps - 1)) : zero;
#pragma unroll
        for (int tb = 0; tb < kTT; tb += 4) {
#pragma unroll
          for (int t = 0; t < 4; ++t)
            v[kTaps - 1 + t] = ok && tb + t < nt ? in.four(part, d, t0 + tb + t) : zero;
#pragma unroll
          for (int t = 0; t < 4; ++t) {
            float4 y = zero;
#pragma unroll
            for (int j = 0; j < kTaps; ++j) axpy4(y, w[j], v[t + j]);
            put(part, d, tb + t, tb + t < nt ? silu4(y) : zero);
          }
#pragma unroll
          for (int j = 0; j < kTaps - 1; ++j) v[j] = v[4 + j];
        }
      } else {
        const int one = MEMORY && part == 2 ? p.vdim - d : -1;   // the normaliser's column
#pragma unroll
        for (int t = 0; t < kTT; ++t) {
          float4 y = ok && t < nt ? in.four(part, d, t0 + t) : zero;
          if (FORGET && part == 0) y = silu4(y);
          if (one == 0) y.x = 1.f;
          if (one == 1) y.y = 1.f;
          if (one == 2) y.z = 1.f;
          if (one == 3) y.w = 1.f;
          put(part, d, t, y);
        }
      }
      continue;
    }
    for (int t = 0; t < kTT; ++t) {
      float y[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        y[e] = 0.f;
        if (t < nt && d + e < limit) {
          if (DELTA) {
            const float* w = p.conv + in.ch(part) + d + e;
            for (int j = 0; j < p.taps; ++j)
              y[e] = fmaf(w[(long long)j * p.channels], in.one(part, d + e, t0 + t - in.back + j), y[e]);
            y[e] = silu_f(y[e]);
          } else {
            y[e] = in.one(part, d + e, t0 + t);
            if (FORGET && part == 0) y[e] = silu_f(y[e]);
          }
        }
        if (MEMORY && part == 2 && d + e == p.vdim) y[e] = 1.f;
      }
      put(part, d, t, make_float4(y[0], y[1], y[2], y[3]));
    }
  }
  __syncthreads();

  // ---- 2. unit length
  if (DELTA) {
    for (int t = warp; t < kTT; t += kWarps) {
      float a = 0.f, b = 0.f;
      for (int d = lane * 4; d < DP; d += 128) {
        const float4 q = load4(sC + t * DP + d), k = load4(sB + t * DP + d);
        a = dot4(q, q, a);
        b = dot4(k, k, b);
      }
      a = warp_sum(a);
      b = warp_sum(b);
      if (lane == 0) {
        invQ[t] = p.q_scale / sqrtf(a + 1e-6f);
        invK[t] = 1.f / sqrtf(b + 1e-6f);
      }
    }
  }
  // ---- 3. decays; a, b, c
  float cum = 0.f;
  if (DELTA) {
    const float ae = tid < p.dim ? p.a_exp[h] : 0.f;
    const float bias = tid < p.dim ? p.dt_bias[h * p.dim + tid] : 0.f;
#pragma unroll
    for (int t = 0; t < kTT; ++t) {
      if (t < nt) cum += fmaxf(-ae * softplus_f(z[t] + bias), kMinLogDecay);
      z[t] = cum;
    }
  } else if (FORGET) {
    if (tid < DP) {
      const bool ok = tid < p.dim;
      const float bias = ok ? p.dt_bias[h * p.dim + tid] : 0.f, lower = ok ? p.lower[h * p.dim + tid] : 0.f;
#pragma unroll
      for (int t = 0; t < kTT; ++t) {
        const float k = ok && t < nt ? (1.f - lower) / (1.f + expf(z[t] + bias)) : 0.f;
        const float f = lower + (1.f - lower) / (1.f + expf(-z[t] - bias));
        if (ok && t < nt) cum += fmaxf(k < 0.5f ? log1pf(-k) : logf(f), kMinLogDecay);
        sB[t * DP + tid] = k;
        z[t] = cum;
      }
    }
  } else {
#pragma unroll
    for (int t = 0; t < kTT; ++t) {
      cum += invQ[t];
      z[t] = cum;
    }
  }
  const bool strong = __syncthreads_or(cum < kTileLogDecay);
  if (tid == 0) rec[R::kStrong] = strong ? 1.f : 0.f;
  if (tid < DP) {
    float base = 0.f;
#pragma unroll
    for (int t = 0; t < kTT; ++t) {
      const float l = z[t] - base, g = __expf(l);
      const float k = sB[t * DP + tid], q = sC[t * DP + tid];
      const float kn = DELTA ? k * invK[t] : k;
      const float b = kn * __expf((MEMORY ? invK[t] : 0.f) - l);
      const float c = q * g * (DELTA ? invQ[t] : p.q_scale);
      sB[t * DP + tid] = b;
      sC[t * DP + tid] = c;
      rec[R::kKeys + t * DP + tid] = b;
      rec[R::kQ + t * DP + tid] = c;
      if (DELTA) {
        sA[t * DP + tid] = kn * g;
        rec[R::kA + t * DP + tid] = kn * g;
      }
      if (t % kB == kB - 1) {
        rec[R::kG + t / kB * DP + tid] = g;
        if (strong) base += l;
      }
    }
  }
  __syncthreads();
  // ---- 4. scalar products within groups
  for (int g = warp; g < kTT / kB; g += kWarps) {
    float a[kB][kB], c[kB][kB];   // [token][earlier token]
#pragma unroll
    for (int i = 0; i < kB; ++i)
#pragma unroll
      for (int j = 0; j < kB; ++j) a[i][j] = c[i][j] = 0.f;
    for (int d = lane * 4; d < DP; d += 128) {
      float4 b[kB];
#pragma unroll
      for (int j = 0; j < kB; ++j) b[j] = load4(sB + (g * kB + j) * DP + d);
#pragma unroll
      for (int i = 0; i < kB; ++i) {
        const float4 ci = load4(sC + (g * kB + i) * DP + d);
        float4 ai = ci;
        if (DELTA) ai = load4(sA + (g * kB + i) * DP + d);
#pragma unroll
        for (int j = 0; j <= i; ++j) {
          c[i][j] = dot4(ci, b[j], c[i][j]);
          if (DELTA && j < i) a[i][j] = dot4(ai, b[j], a[i][j]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < kB; ++i)
#pragma unroll
      for (int j = 0; j <= i; ++j) {
        const float y = warp_sum(c[i][j]);
        const float x = DELTA && j < i ? warp_sum(a[i][j]) : 0.f;
        if (lane == 0) {
          rec[R::kDotC + (g * kB + i) * kB + j] = y;
          if (j < i) rec[R::kDotB + (g * kB + i) * kB + j] = x;
        }
      }
  }
  if (DELTA && t0 + nt == s.n) save_inputs<T>(p, s, in, h % p.group == 0, 0, p.vdim);
}

// Floats of a stage of scan_kernel's shared memory
template <int DP, bool DELTA>
__host__ __device__ constexpr int stage_floats(int nc) {
  return Record<DP, DELTA>::kV + kTT * nc;
}

template <typename T, int DP, int RULE, int STAGES>
__global__ void __launch_bounds__(max_warps(RULE) * 32, 1) scan_kernel(const ScanArgs p) {
  constexpr bool DELTA = RULE == kDelta;
  using Sh = ScanShape<DP>;
  using R = Record<DP, DELTA>;
  constexpr int kCols = Sh::kCols, kChunks = Sh::kRows / 4, kKinds = DELTA ? 2 : 1;
  extern __shared__ __align__(16) float sm[];
  pdl_wait();
  pdl_trigger();
  const int slice = blockIdx.x % p.slices, h = blockIdx.x / p.slices % p.heads;
  const int seq = blockIdx.x / p.slices / p.heads;
  const Seq s(p.steps + (long long)seq * kStepInts);
  if (s.n <= 0) return;
  if (s.slot <= 0 || s.slot >= p.num_slots) {
    put_zeros<T, RULE>(p, s, h, slice);
    return;
  }
  const int tid = threadIdx.x, threads = blockDim.x, warp = tid >> 5, lane = tid & 31, rl = lane & 7;
  const int nc = p.nc, c_first = slice * nc, vcols = p.slices * nc;
  const int c_local = warp * Sh::kWarpCols + (lane >> 3) * kCols;
  const int stage_size = stage_floats<DP, DELTA>(nc);
  const int tiles = (s.n + kTT - 1) / kTT;
  const float* rec0 = p.records + ((long long)p.first_tile[seq] * p.heads + h) * p.record;
  auto fetch = [&](int i) {   // (one group of copies per tile, also when there is none)
    if (i < tiles) {
      const float* src = rec0 + (long long)i * p.heads * p.record;
      float* dst = sm + i % STAGES * stage_size;
      for (int x = tid * 4; x < R::kV; x += threads * 4) copy16_async(dst + x, src + x);
      const int per = nc / 4;
      for (int x = tid; x < kTT * per; x += threads) {
        const int t = x / per, c = (x - t * per) * 4;
        copy16_async(dst + R::kV + t * nc + c, src + R::kV + t * vcols + c_first + c);
      }
    }
    copies_commit();
  };
#pragma unroll
  for (int i = 0; i < STAGES - 1; ++i) fetch(i);
  float* state = p.state + ((long long)s.slot * p.heads + h) * p.dim * p.state_cols;
  float2 S[Sh::kRows / 2][kCols];
  load_state<DP>(S, state, p, rl, c_first + c_local, s.start > 0);
  // outputs: eight columns of a token a thread, where they are a power of two
  const int lanes = p.vdim / 8;
  const T* gate = reinterpret_cast<const T*>(p.gate) + s.first * p.ld_gate + (long long)h * p.vdim;
  T* out = reinterpret_cast<T*>(p.out) + s.first * p.ldo + (long long)h * p.vdim;
  const float* w = p.norm + (long long)h * p.norm_step;
  const int o_t = p.vec_out ? tid / lanes : 0, o_c = p.vec_out ? (tid - o_t * lanes) * 8 : 0;
  float4 wa = make_float4(0.f, 0.f, 0.f, 0.f), wb = wa;
  if (p.vec_out) {
    wa = load4(w + o_c);
    wb = load4(w + o_c + 4);
  }

  for (int it = 0; it < tiles; ++it) {
    const int t0 = it * kTT, nt = min(kTT, s.n - t0);
    copies_wait<STAGES - 2>();
    __syncthreads();       // the tile's record is there; the stage of the tile before is free
    fetch(it + STAGES - 1);
    float* st = sm + it % STAGES * stage_size;
    const float* sB = st + R::kKeys;
    const float* sC = st + R::kQ;
    const float* sA = st + R::kA;
    const float* dotB = st + R::kDotB;
    const float* dotC = st + R::kDotC;
    float* sV = st + R::kV;
    const bool strong = st[R::kStrong] != 0.f;
    Raw8<T> gates = {};
    if (RULE != kForget && p.vec_out && o_t < nt)   // the first outputs' gates, ahead
      gates.load(gate + (long long)(t0 + o_t) * p.ld_gate + o_c);
    for (int q0 = 0; q0 < nt; q0 += kB) {
      float2 acc[kKinds][kCols][kB];
#pragma unroll
      for (int e = 0; e < kKinds; ++e)
#pragma unroll
        for (int c = 0; c < kCols; ++c)
#pragma unroll
          for (int i = 0; i < kB; ++i) acc[e][c][i] = make_float2(0.f, 0.f);
#pragma unroll
      for (int j = 0; j < kChunks; ++j) {
        const int r = j * 32 + rl * 4;
#pragma unroll
        for (int i = 0; i < kB; ++i) {
          const float4 vc = load4(sC + (q0 + i) * DP + r);
          if constexpr (DELTA) {
            const float4 va = load4(sA + (q0 + i) * DP + r);
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
      float my[kB];
      const int my_c = reduce_columns<kKinds, kCols, kB>(acc, my);
      // u of every token and column; o
      float u[kB], U[kB][kCols];
#pragma unroll
      for (int i = 0; i < kB; ++i) {
        u[i] = sV[(q0 + i) * nc + c_local + my_c];
        if constexpr (DELTA) {
          float x = u[i] - my[i];
#pragma unroll
          for (int j = 0; j < kB; ++j)
            if (j < i) x = fmaf(-dotB[(q0 + i) * kB + j], u[j], x);
          u[i] = st[R::kBeta + q0 + i] * x;   // (of use in lanes 0 - 3)
        }
      }
      if constexpr (DELTA) {
#pragma unroll
        for (int i = 0; i < kB; ++i) {
#pragma unroll
          for (int c = 0; c < kCols; ++c) U[i][c] = __shfl_sync(0xffffffffu, u[i], (lane & 24) | c);
          u[i] = __shfl_sync(0xffffffffu, u[i], (lane & 24) | my_c);
        }
      } else {
#pragma unroll
        for (int i = 0; i < kB; ++i)
#pragma unroll
          for (int c = 0; c < kCols; ++c) U[i][c] = sV[(q0 + i) * nc + c_local + c];
      }
      __syncwarp();   // the values of these tokens have been read: the outputs take their place
#pragma unroll
      for (int i = 0; i < kB; ++i) {
        float o = my[i];
#pragma unroll
        for (int j = 0; j < kB; ++j)
          if (j <= i) o = fmaf(dotC[(q0 + i) * kB + j], u[j], o);
        if (rl >= 4 && rl < 4 + kCols) sV[(q0 + i) * nc + c_local + my_c] = o;
      }
      const bool renorm = strong || q0 + kB >= nt;
      const float* ge = st + R::kG + (strong ? q0 / kB : kTT / kB - 1) * DP;
#pragma unroll
      for (int j = 0; j < kChunks; ++j) {
        const int r = j * 32 + rl * 4;
#pragma unroll
        for (int i = 0; i < kB; ++i) {
          const float4 b = load4(sB + (q0 + i) * DP + r);
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
    __syncthreads();   // the tile's outputs are there
    if (p.raw != nullptr) {
      for (int t = warp; t < nt; t += threads / 32) {
        float* dst = p.raw + ((s.first + t0 + t) * p.heads + h) * p.raw_cols + c_first;
        for (int c = lane; c < min(nc, p.ncols - c_first); c += 32) dst[c] = sV[t * nc + c];
        if (RULE == kMemory && slice == 0 && lane == 0) dst[p.ncols] = st[R::kBeta + t];
      }
    } else if (p.vec_out) {
      vector_outputs<T, RULE>(p, sV, nc, st + R::kBeta, nt, lanes, gate + (long long)t0 * p.ld_gate,
                               out + (long long)t0 * p.ldo, w, gates, wa, wb);
    } else {
      for (int t = warp; t < nt; t += threads / 32)
        head_output<T, RULE>(p, sV + t * nc, s.first + t0 + t, h, st[R::kBeta + t]);
    }
  }
  copies_wait<0>();
  store_state<DP>(S, state, p, rl, c_first + c_local);
}

// Heads whose columns several blocks share: norm, weight and gate of the raw outputs. A warp per
// (token, head).
template <typename T, int RULE>
__global__ void __launch_bounds__(256) scan_output_kernel(const ScanArgs p, long long n) {
  pdl_wait();
  pdl_trigger();
  const long long k = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (k >= n) return;
  const float* o = p.raw + k * p.raw_cols;
  head_output<T, RULE>(p, o, k / p.heads, (int)(k % p.heads), RULE == kMemory ? o[p.vdim + 1] : 0.f);
}

template <typename T, int DP, int RULE>
static int launch_scan(const ScanArgs& a, int n_seq, int n_tiles, int max_rows, cudaStream_t stream) {
  constexpr bool DELTA = RULE == kDelta;
  // (one-token steps and 32-bit models; on tensor cores a warp has 16 columns)
  const int wc = a.warp_cols;
  if (a.nc % wc || a.nc / wc > max_warps(RULE) || (long long)a.nc * (a.slices - 1) >= a.ncols ||
      (long long)a.nc * a.slices < a.ncols)
    return -2;
  const long long blocks = (long long)n_seq * a.heads * a.slices;
  const dim3 threads(a.nc / wc * 32);
  if (blocks > 0x7fffffffll || (long long)n_tiles * a.heads > 0x7fffffffll) return -6;
  if (max_rows == 1) {
    using Sh = StepShape<DP>;
    const size_t smem = (size_t)Sh::smem_floats(a.nc) * sizeof(float);
    const dim3 step_threads(a.nc / 4 * Sh::kGroups);
    if (step_threads.x > Sh::max_threads(RULE)) return -2;
    if (!set_smem(step_kernel<T, DP, RULE>, smem)) return -3;
    return launch_pdl(step_kernel<T, DP, RULE>, dim3((unsigned)blocks), step_threads, smem, stream, a) ==
                   cudaSuccess
               ? 0
               : -5;
  }
  if (n_tiles < 1 || a.records == nullptr || a.tiles == nullptr || a.first_tile == nullptr ||
      a.record < (sizeof(T) == 2 ? MmaRecord<DP, DELTA>::bytes(a.nc * a.slices) / 4
                                 : stage_floats<DP, DELTA>(a.nc * a.slices)))
    return -2;
  if (RULE == kMemory && launch_pdl(memory_gates_kernel<T>, dim3((unsigned)(n_seq * a.heads)),
                           dim3(max_rows <= 128 ? 128 : max_rows <= 512 ? 512 : 1024), 0, stream,
                           a) != cudaSuccess)
    return -5;
  if constexpr (sizeof(T) == 2) {
    return launch_tiles_mma(a, RULE, n_seq, n_tiles, stream);
  } else {
    const dim3 tile_grid((unsigned)(n_tiles * a.heads)), tile_threads(DP <= 128 ? 128 : 256);
    const size_t tile_smem = (size_t)(DELTA ? 3 : 2) * kTT * DP * sizeof(float);
    if (!set_smem(tile_kernel<T, DP, RULE>, tile_smem)) return -3;
    if (launch_pdl(tile_kernel<T, DP, RULE>, tile_grid, tile_threads, tile_smem, stream, a) != cudaSuccess)
      return -5;
    const size_t stage = (size_t)stage_floats<DP, DELTA>(a.nc) * sizeof(float);
    const bool three = 3 * stage <= 220 * 1024;
    auto k = three ? scan_kernel<T, DP, RULE, 3> : scan_kernel<T, DP, RULE, 2>;
    const size_t smem = (three ? 3 : 2) * stage;
    if (smem > 220 * 1024) return -6;
    if (!set_smem(k, smem)) return -3;
    return launch_pdl(k, dim3((unsigned)blocks), threads, smem, stream, a) == cudaSuccess ? 0 : -5;
  }
}

template <typename T, int RULE>
static int run_scan(const ScanArgs& a, int n_seq, int n_tiles, int max_rows, long long rows,
                    cudaStream_t stream) {
  const int rc = a.dim <= 32    ? launch_scan<T, 32, RULE>(a, n_seq, n_tiles, max_rows, stream)
                 : a.dim <= 64  ? launch_scan<T, 64, RULE>(a, n_seq, n_tiles, max_rows, stream)
                 : a.dim <= 128 ? launch_scan<T, 128, RULE>(a, n_seq, n_tiles, max_rows, stream)
                 : a.dim <= 256 ? launch_scan<T, 256, RULE>(a, n_seq, n_tiles, max_rows, stream)
                                : -6;
  if (rc != 0 || a.raw == nullptr) return rc;
  const long long n = rows * a.heads;
  return launch_pdl(scan_output_kernel<T, RULE>, dim3((unsigned)((n + 7) / 8)), dim3(256), 0, stream, a,
                    n) == cudaSuccess
             ? 0
             : -5;
}

static int aligned4(const void* p, long long ld, int dtype) {
  return ld % 4 == 0 && (reinterpret_cast<uintptr_t>(p) & (dtype == 0 ? 7 : 15)) == 0;
}

// Columns of a warp: on tensor cores (16-bit models, portions of several tokens) always 16
static int warp_cols(int dim, int dtype, bool several) {
  return dim <= 128 || (several && dtype == 0) ? 16 : 8;
}

// The common part of the entry points
static void finish_args(ScanArgs& a, int slices, int ncols, int raw_cols, void* raw, int dtype,
                        bool several) {
  a.slices = slices;
  a.ncols = ncols;
  a.warp_cols = warp_cols(a.dim, dtype, several);
  a.nc = (ncols + slices - 1) / slices;
  a.nc = (a.nc + a.warp_cols - 1) / a.warp_cols * a.warp_cols;
  a.raw = slices > 1 ? reinterpret_cast<float*>(raw) : nullptr;
  a.raw_cols = raw_cols;
  a.q_scale = 1.f / sqrtf((float)a.dim);
  const int lanes = a.vdim / 8;
  a.vec_out = slices == 1 && a.vdim % 8 == 0 && lanes <= 32 && (lanes & (lanes - 1)) == 0 &&
              aligned4(a.gate, a.ld_gate, dtype) && aligned4(a.out, a.ldo, dtype) &&
              aligned4(a.norm, a.norm_step, 1);
  a.vec = a.dim % 4 == 0 && a.vdim % 4 == 0 && a.q_at % 4 == 0 && a.k_at % 4 == 0 && a.v_at % 4 == 0 &&
          aligned4(a.proj, a.ld, dtype) && aligned4(a.conv_state, 0, dtype) && aligned4(a.conv, 0, 1) &&
          aligned4(a.decay, a.ld_decay, dtype);
}

}  // namespace ab200

using namespace ab200;
typedef __nv_bfloat16 bf16;

extern "C" {

// Blocks per head so that each block's columns fit: 0 if dim is beyond the kernel's.
int ab200_scan_min_slices(int dim, int ncols, int rule, int dtype, int several) {
  if (dim < 1 || dim > 256) return 0;
  const int most = max_warps(rule) * warp_cols(dim, dtype, several != 0);
  return (ncols + most - 1) / most;
}

// Floats of a tile's record of a head (portions of more than one token).
long long ab200_scan_record(int dim, int ncols, int slices, int rule, int dtype) {
  const bool delta = rule == kDelta;
  const int wc = warp_cols(dim, dtype, true), nc = ((ncols + slices - 1) / slices + wc - 1) / wc * wc;
  const int dp = dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : 256;
  if (dtype == 0) {
    const int cols = nc * slices;
    return (delta ? (dp == 32    ? MmaRecord<32, true>::bytes(cols)
                     : dp == 64  ? MmaRecord<64, true>::bytes(cols)
                     : dp == 128 ? MmaRecord<128, true>::bytes(cols)
                                 : MmaRecord<256, true>::bytes(cols))
                  : (dp == 32    ? MmaRecord<32, false>::bytes(cols)
                     : dp == 64  ? MmaRecord<64, false>::bytes(cols)
                     : dp == 128 ? MmaRecord<128, false>::bytes(cols)
                                 : MmaRecord<256, false>::bytes(cols))) / 4;
  }
  const int vectors = delta ? 3 * kTT + kTT / kB : 2 * kTT + kTT / kB;
  return (long long)vectors * dp + 2 * kTT * kB + kTT + 4 + (long long)kTT * nc * slices;
}

// Gated delta rule over n_seq sequences. proj [T, ld]: query and key heads of dim at q_at, k_at, value
// heads of vdim at v_at, step sizes at b_at. steps int32 [n_seq, 5]: first row, rows, slot (0: padding),
// start position, phase. When max_rows > 1: tiles int32 [n_tiles, 2] and first_tile int32 [n_seq] cut the
// sequences into tiles of 16 tokens, records fp32 [n_tiles, heads, ab200_scan_record]. raw fp32
// [T, heads, vdim] when slices > 1. See ScanArgs.
int ab200_delta_scan(const void* proj, long long ld, int q_at, int k_at, int v_at, int b_at,
                     const void* decay, long long ld_decay, const void* gate, long long ld_gate,
                     const void* conv, int taps, const void* a_exp, const void* dt_bias,
                     const void* norm, void* state, int state_cols, void* conv_state, int num_slots,
                     const void* steps, int n_seq, int max_rows, const void* tiles,
                     const void* first_tile, int n_tiles, void* records, long long T, int heads,
                     int kv_heads, int dim, int vdim, int slices, float eps, void* raw, void* out,
                     long long ldo, int dtype, int* status, cudaStream_t stream) {
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
  a.tiles = reinterpret_cast<const int*>(tiles);
  a.first_tile = reinterpret_cast<const int*>(first_tile);
  a.records = reinterpret_cast<float*>(records);
  a.record = ab200_scan_record(dim, vdim, slices, kDelta, dtype);
  a.heads = heads; a.group = heads / kv_heads; a.dim = dim; a.vdim = vdim;
  a.taps = taps;
  a.channels = 2 * kv_heads * dim + heads * vdim;
  a.eps = eps;
  a.out = out; a.ldo = ldo;
  a.status = status;
  finish_args(a, slices, vdim, vdim, raw, dtype, max_rows > 1);
  return dtype == 0 ? run_scan<bf16, kDelta>(a, n_seq, n_tiles, max_rows, T, stream)
                    : run_scan<float, kDelta>(a, n_seq, n_tiles, max_rows, T, stream);
}

// Matrix memory: query and key heads of dim, value heads of vdim, gates at i_at and f_at; state
// [slots, heads, dim, state_cols] with the normaliser in column vdim; max_state fp32 [slots, 2, heads];
// gates fp32 [T, heads, 3] when max_rows > 1; raw fp32 [T, heads, vdim + 2] when slices > 1.
int ab200_memory_scan(const void* proj, long long ld, int q_at, int k_at, int v_at, int i_at, int f_at,
                      const void* gate, long long ld_gate, const void* i_bias, const void* f_bias,
                      float cap, const void* norm, void* state, int state_cols, void* max_state,
                      int num_slots, const void* steps, int n_seq, int max_rows, const void* tiles,
                      const void* first_tile, int n_tiles, void* records, void* gates, long long T,
                      int heads, int dim, int vdim, int slices, float eps, void* raw, void* out,
                      long long ldo, int dtype, int* status, cudaStream_t stream) {
  if (T <= 0 || n_seq <= 0) return 0;
  if (heads < 1 || dim < 1 || vdim < 1 || slices < 1 || state_cols < vdim + 1 || state_cols % 4 ||
      !(cap > 0.f) || (slices > 1 && raw == nullptr) || (max_rows > 1 && gates == nullptr))
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
  a.tiles = reinterpret_cast<const int*>(tiles);
  a.first_tile = reinterpret_cast<const int*>(first_tile);
  a.records = reinterpret_cast<float*>(records);
  a.record = ab200_scan_record(dim, vdim + 1, slices, kMemory, dtype);
  a.gates = reinterpret_cast<float*>(gates);
  a.heads = heads; a.group = 1; a.dim = dim; a.vdim = vdim;
  a.taps = 1;
  a.eps = eps;
  a.out = out; a.ldo = ldo;
  a.status = status;
  finish_args(a, slices, vdim + 1, vdim + 2, raw, dtype, max_rows > 1);
  return dtype == 0 ? run_scan<bf16, kMemory>(a, n_seq, n_tiles, max_rows, T, stream)
                    : run_scan<float, kMemory>(a, n_seq, n_tiles, max_rows, T, stream);
}

// Forget scan: query heads of dim at q_at (before silu), forget gates [heads][dim] at f_at (before bias and
// sigmoid), value heads of vdim at v_at; f_bias and lower fp32 [heads, dim], norm fp32 [vdim]; state
// [slots, heads, dim, state_cols]; the rest as for ab200_delta_scan, without an output gate.
int ab200_forget_scan(const void* proj, long long ld, int q_at, int f_at, int v_at, const void* f_bias,
                      const void* lower, const void* norm, void* state, int state_cols, int num_slots,
                      const void* steps, int n_seq, int max_rows, const void* tiles,
                      const void* first_tile, int n_tiles, void* records, long long T, int heads, int dim,
                      int vdim, int slices, float eps, void* raw, void* out, long long ldo, int dtype,
                      int* status, cudaStream_t stream) {
  if (T <= 0 || n_seq <= 0) return 0;
  if (heads < 1 || dim < 1 || vdim < 1 || slices < 1 || state_cols < vdim || state_cols % 4 ||
      (slices > 1 && raw == nullptr))
    return -2;
  ScanArgs a = {};
  a.proj = proj; a.ld = ld;
  a.q_at = q_at; a.k_at = f_at; a.v_at = v_at;
  a.decay = reinterpret_cast<const char*>(proj) + (long long)f_at * (dtype == 0 ? 2 : 4);
  a.ld_decay = ld;
  a.dt_bias = reinterpret_cast<const float*>(f_bias);
  a.lower = reinterpret_cast<const float*>(lower);
  a.norm = reinterpret_cast<const float*>(norm);
  a.state = reinterpret_cast<float*>(state);
  a.state_cols = state_cols;
  a.num_slots = num_slots;
  a.steps = reinterpret_cast<const int*>(steps);
  a.tiles = reinterpret_cast<const int*>(tiles);
  a.first_tile = reinterpret_cast<const int*>(first_tile);
  a.records = reinterpret_cast<float*>(records);
  a.record = ab200_scan_record(dim, vdim, slices, kForget, dtype);
  a.heads = heads; a.group = 1; a.dim = dim; a.vdim = vdim;
  a.taps = 1;
  a.eps = eps;
  a.out = out; a.ldo = ldo;
  a.status = status;
  finish_args(a, slices, vdim, vdim, raw, dtype, max_rows > 1);
  a.q_scale = 1.f;
  return dtype == 0 ? run_scan<bf16, kForget>(a, n_seq, n_tiles, max_rows, T, stream)
                    : run_scan<float, kForget>(a, n_seq, n_tiles, max_rows, T, stream);
}

}  // extern "C"
