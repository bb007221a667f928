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
// channel decays so much within the tile that 1 / G would leave fp32's range.
//
// For 16-bit models the products of a tile run on the tensor cores (mma.sync: Z lives in the registers
// of the warps that own its columns, as the accumulator of the update and, converted in place, as the
// left operand of the read-outs; nothing but the small token-side operands passes through shared
// memory). Every operand is the sum of two bf16 numbers, so that products carry 16 significant bits,
// and sums and Z are fp32. The 16 tokens are then one group, solved with the inverse of the unit
// triangular matrix that the tile's a, b and beta form. 32-bit models use fp32 multiply-adds.
//
// What a sequence carries over lies in its slot: S in fp32; the convolution's last inputs and m twice,
// for even and odd steps of the sequence (`phase`), so that blocks which read them never race with the
// block that writes them. A sequence that starts at position 0 reads nothing from its slot.

#include "api.h"
#include "common/elem.cuh"
#include "common/pdl.cuh"

namespace ab200 {

// warps of a block: 128 columns of wide states, and the normaliser's beside them
__host__ __device__ constexpr int max_warps(bool delta) { return delta ? 8 : 9; }

constexpr int kTT = 16, kB = 4;           // tokens per tile and per group
constexpr int kTaps = 4;                  // convolutions of up to this many taps stay in registers
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
  const int* tiles;          // [n_tiles][2]: sequence, its first token of the tile; in order
  const int* first_tile;     // [n]
  float* gates;              // memory: [T][heads][3]: log decay, log input factor, m
  float* records;            // [n_tiles][heads][record]
  long long record;          // floats
  void* out;                 // [T][ldo], head h at column h * vdim (one block per head) ...
  long long ldo;
  float* raw;                // ... or [T][heads][raw_cols] unnormed, for scan_output
  int raw_cols;
  int num_slots, heads, group, dim, vdim, ncols, taps, channels;
  int slices, nc;            // blocks per head, columns of each
  int warp_cols;             // columns of a warp
  int vec;                   // four channels at a time are aligned
  int vec_out;               // eight output columns at a time are aligned, a power of two of them
  float q_scale, cap, eps;
  int* status;
};

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
__device__ __forceinline__ void copy16_async(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void copies_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void copies_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

constexpr float kLog2e = 1.4426950408889634f;
__device__ __forceinline__ float exp2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp_fast(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float log2_fast(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// log(1 + e^z); log1p's first terms where the fast logarithm would lose them
__device__ __forceinline__ float softplus_f(float z) {
  const float e = exp2_fast(-kLog2e * fabsf(z));
  const float series = e * fmaf(e, fmaf(e, fmaf(e, -0.25f, 0.33333333f), -0.5f), 1.f);
  return fmaxf(z, 0.f) + (e < 0.03f ? series : log2_fast(1.f + e) * (1.f / kLog2e));
}
__device__ __forceinline__ float sigmoid_f(float z) { return rcp_fast(1.f + exp2_fast(-kLog2e * z)); }
__device__ __forceinline__ float silu_f(float z) { return z * sigmoid_f(z); }
__device__ __forceinline__ float4 silu4(const float4& y) {
  return make_float4(silu_f(y.x), silu_f(y.y), silu_f(y.z), silu_f(y.w));
}
__device__ __forceinline__ void axpy4(float4& y, const float4& w, const float4& v) {
  y.x = fmaf(w.x, v.x, y.x);
  y.y = fmaf(w.y, v.y, y.y);
  y.z = fmaf(w.z, v.z, y.z);
  y.w = fmaf(w.w, v.w, y.w);
}
__device__ __forceinline__ float dot4(const float4& a, const float4& b, float acc) {
  return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, acc))));
}
// D[16 x 8] += A[16 x 16] B[16 x 8], bf16 operands: lane (g = lane / 4, t = lane % 4) holds D's rows g
// and g + 8, columns 2 t and 2 t + 1; A's a0 (g, 2 t ..), a1 (g + 8, 2 t ..), a2, a3 eight columns
// further; B's b0 (rows 2 t .., column g), b1 eight rows further
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void load_matrices(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void load_matrices_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
// x and y as sums of two bf16 numbers each
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  lo = pack_bf16x2(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xffff0000u));
}
// An accumulator pair [16 x 16] as a left operand
__device__ __forceinline__ void split_left(const float (&d0)[4], const float (&d1)[4], uint32_t (&hi)[4],
                                           uint32_t (&lo)[4]) {
  split2(d0[0], d0[1], hi[0], lo[0]);
  split2(d0[2], d0[3], hi[1], lo[1]);
  split2(d1[0], d1[1], hi[2], lo[2]);
  split2(d1[2], d1[3], hi[3], lo[3]);
}
// d[n] += (hi + lo) (bh + bl), n = 0, 1: right operands' registers 2 n, 2 n + 1
__device__ __forceinline__ void mma_split(float (&d)[2][4], const uint32_t (&hi)[4], const uint32_t (&lo)[4],
                                          const uint32_t (&bh)[4], const uint32_t (&bl)[4]) {
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    mma_bf16(d[n], hi, bl[2 * n], bl[2 * n + 1]);
    mma_bf16(d[n], lo, bh[2 * n], bh[2 * n + 1]);
    mma_bf16(d[n], hi, bh[2 * n], bh[2 * n + 1]);
  }
}
// Elements as they lie in memory, widened when they are used (so that nothing waits for a load early)
template <typename T>
struct Raw8;
template <>
struct Raw8<float> {
  float4 a, b;
  __device__ __forceinline__ void load(const float* p) { a = load4(p); b = load4(p + 4); }
  __device__ __forceinline__ float4 lo() const { return a; }
  __device__ __forceinline__ float4 hi() const { return b; }
};
__device__ __forceinline__ float4 widen(uint32_t x, uint32_t y) {
  return make_float4(__uint_as_float(x << 16), __uint_as_float(x & 0xffff0000u), __uint_as_float(y << 16),
                     __uint_as_float(y & 0xffff0000u));
}
template <>
struct Raw8<__nv_bfloat16> {   // (8-byte aligned)
  uint2 a, b;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) {
    a = *reinterpret_cast<const uint2*>(p);
    b = *reinterpret_cast<const uint2*>(p + 4);
  }
  __device__ __forceinline__ float4 lo() const { return widen(a.x, a.y); }
  __device__ __forceinline__ float4 hi() const { return widen(b.x, b.y); }
};
// log gates of the matrix memory
__device__ __forceinline__ float2 memory_log_gates(float zi, float zf, float cap) {
  const float z = cap * tanhf(zf / cap);
  return make_float2(cap * tanhf(zi / cap), fminf(z, 0.f) - log1pf(expf(-fabsf(z))));
}

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

// A sequence of a step and a head of it
struct Seq {
  long long first;
  int n, slot, start, phase;
  __device__ __forceinline__ explicit Seq(const int* s)
      : first(s[0]), n(s[1]), slot(s[2]), start(s[3]), phase(s[4] & 1) {}
};

// What a block reads of the projections: columns and convolution channels of its head's query, key and
// value, and the inputs of tokens before the step's.
template <typename T>
struct Inputs {
  const T* proj;
  const T* old;
  long long ld;
  int back, start, channels;
  int q_col, k_col, v_col, q_ch, k_ch, v_ch;
  __device__ __forceinline__ Inputs(const ScanArgs& p, const Seq& s, int h, bool delta) {
    const int hk = delta ? h / p.group : h, G = p.heads / p.group;
    proj = reinterpret_cast<const T*>(p.proj) + s.first * p.ld;
    ld = p.ld;
    back = delta ? p.taps - 1 : 0;
    start = s.start;
    channels = p.channels;
    old = reinterpret_cast<const T*>(p.conv_state) + ((long long)s.slot * 2 + s.phase) * back * channels;
    q_col = p.q_at + hk * p.dim;
    k_col = p.k_at + hk * p.dim;
    v_col = p.v_at + h * p.vdim;
    q_ch = hk * p.dim;
    k_ch = (G + hk) * p.dim;
    v_ch = 2 * G * p.dim + h * p.vdim;
  }
  __device__ __forceinline__ int col(int part) const { return part == 0 ? q_col : part == 1 ? k_col : v_col; }
  __device__ __forceinline__ int ch(int part) const { return part == 0 ? q_ch : part == 1 ? k_ch : v_ch; }
  // part 0 query, 1 key, 2 value; token t of the step (t < 0: an earlier one)
  __device__ __forceinline__ float one(int part, int d, int t) const {
    if (t >= 0) return to_f32<T>(proj[t * ld + col(part) + d]);
    return start + t >= 0 ? to_f32<T>(old[(long long)(back + t) * channels + ch(part) + d]) : 0.f;
  }
  __device__ __forceinline__ float4 four(int part, int d, int t) const {
    if (t >= 0) return load4(proj + t * ld + col(part) + d);
    return start + t >= 0 ? load4(old + (long long)(back + t) * channels + ch(part) + d)
                          : make_float4(0.f, 0.f, 0.f, 0.f);
  }
};

// The convolution's inputs that the sequence's next step reads, written by the blocks `qk` (queries and
// keys) and those of the value columns [v0, v0 + nv).
template <typename T>
__device__ __forceinline__ void save_inputs(const ScanArgs& p, const Seq& s, const Inputs<T>& in, bool qk,
                                            int v0, int nv) {
  T* next = reinterpret_cast<T*>(p.conv_state) +
            ((long long)s.slot * 2 + (s.phase ^ 1)) * in.back * p.channels;
  const int per = (qk ? 2 * p.dim : 0) + nv;
  for (int it = threadIdx.x; it < in.back * per; it += blockDim.x) {
    const int j = it / per;
    int x = it - j * per, part = 2;
    if (qk) {
      part = x < p.dim ? 0 : x < 2 * p.dim ? 1 : 2;
      x -= part * p.dim;
    }
    if (part == 2) x += v0;
    next[(long long)j * p.channels + in.ch(part) + x] = from_f32<T>(in.one(part, x, s.n - in.back + j));
  }
}

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

// Outputs of padding rows: finite, no state involved
template <typename T, bool DELTA>
__device__ __forceinline__ void put_zeros(const ScanArgs& p, const Seq& s, int h, int slice) {
  if (s.slot >= p.num_slots && threadIdx.x == 0) report_error(p.status, kErrBounds, 50, s.slot);
  for (int t = 0; t < s.n; ++t) {
    if (p.raw != nullptr) {
      float* dst = p.raw + ((s.first + t) * p.heads + h) * p.raw_cols;
      const int c1 = min((slice + 1) * p.nc, p.ncols);
      for (int c = slice * p.nc + threadIdx.x; c < c1; c += blockDim.x) dst[c] = 0.f;
      if (!DELTA && slice == 0 && threadIdx.x == 0) dst[p.ncols] = 1.f;
    } else {
      T* dst = reinterpret_cast<T*>(p.out) + (s.first + t) * p.ldo + (long long)h * p.vdim;
      for (int c = threadIdx.x; c < p.vdim; c += blockDim.x) dst[c] = from_f32<T>(0.f);
    }
  }
}

// A warp's token: norm, weight and gate of a head's outputs o (memory: with the normaliser's product
// in column vdim and `floor` = exp(-m)).
template <typename T, bool DELTA>
__device__ __forceinline__ void head_output(const ScanArgs& p, const float* o, long long row, int h,
                                            float floor) {
  const int lane = threadIdx.x & 31;
  const T* g = reinterpret_cast<const T*>(p.gate) + row * p.ld_gate + (long long)h * p.vdim;
  const float* w = p.norm + (long long)h * p.norm_step;
  T* dst = reinterpret_cast<T*>(p.out) + row * p.ldo + (long long)h * p.vdim;
  float scale = DELTA ? 1.f : 1.f / (fmaxf(fabsf(o[p.vdim]), floor) + 1e-6f);
  float ss = 0.f;
  for (int c = lane; c < p.vdim; c += 32) {
    const float x = o[c] * scale;
    ss = fmaf(x, x, ss);
  }
  scale *= 1.f / sqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
  for (int c = lane; c < p.vdim; c += 32)
    dst[c] = from_f32<T>(o[c] * scale * w[c] * sigmoid_f(to_f32<T>(g[c])));
}

// A block's tile: eight columns a thread, the `lanes` lanes of a token side by side. g, wa, wb: gate
// and norm weights of the thread's first columns.
template <typename T, bool DELTA>
__device__ __forceinline__ void vector_outputs(const ScanArgs& p, const float* o_tile, int ld, const float* floors,
                                               int nt, int lanes, const T* gate, T* out, const float* w,
                                               Raw8<T> g, float4 wa, float4 wb) {
  // (whole warps: the lanes of a token lie in one)
  for (int x = threadIdx.x; x < (kTT * lanes + 31) / 32 * 32; x += blockDim.x) {
    const int t = x / lanes, c = (x - t * lanes) * 8;
    const bool ok = t < nt;
    const float* o = o_tile + (ok ? t : 0) * ld;
    if (x != threadIdx.x && ok) {
      g.load(gate + t * p.ld_gate + c);
      wa = load4(w + c);
      wb = load4(w + c + 4);
    }
    const float4 a = load4(o + c), b = load4(o + c + 4);
    float f = DELTA ? 1.f : 1.f / (fmaxf(fabsf(o[p.vdim]), floors[ok ? t : 0]) + 1e-6f);
    float ss = dot4(a, a, dot4(b, b, 0.f)) * f * f;
    for (int k = lanes / 2; k > 0; k >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, k);
    f *= 1.f / sqrtf(ss / (float)p.vdim + p.eps);
    if (!ok) continue;
    const float4 g0 = g.lo(), g1 = g.hi();
    T* dst = out + t * p.ldo + c;
    store4(dst, make_float4(a.x * f * wa.x * sigmoid_f(g0.x), a.y * f * wa.y * sigmoid_f(g0.y),
                            a.z * f * wa.z * sigmoid_f(g0.z), a.w * f * wa.w * sigmoid_f(g0.w)));
    store4(dst + 4, make_float4(b.x * f * wb.x * sigmoid_f(g1.x), b.y * f * wb.y * sigmoid_f(g1.y),
                                b.z * f * wb.z * sigmoid_f(g1.z), b.w * f * wb.w * sigmoid_f(g1.w)));
  }
}

// ------------------------------------------------------------------ one token per sequence
// A thread holds four neighbouring columns of kRows consecutive rows, so that a warp reads and writes
// whole rows of the state; nc / 4 threads side by side, kGroups groups of rows.
template <int DP>
struct StepShape {
  static constexpr int kGroups = DP <= 128 ? 8 : 16, kRows = DP / kGroups;
  static constexpr int max_threads(bool delta) { return kGroups * max_warps(delta) * 4; }
  static constexpr int smem_floats(int nc) { return 3 * DP + nc + 2 * kGroups * nc; }
};

template <typename T, int DP, bool DELTA>
__global__ void __launch_bounds__(StepShape<DP>::max_threads(DELTA), DP <= 128 ? 2 : 1)
step_kernel(const ScanArgs p) {
  using Sh = StepShape<DP>;
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
    put_zeros<T, DELTA>(p, s, h, slice);
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
  } else {
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
    gate0 = gate[tid];
    norm0 = norm[tid];
  }
  // a channel a thread and turn, two turns' loads at once
  const bool qk_block = slice == 0 && h % p.group == 0;   // saves the queries' and keys' inputs
  T* next = reinterpret_cast<T*>(p.conv_state) + ((long long)s.slot * 2 + (s.phase ^ 1)) * in.back * p.channels;
  struct Channel {   // the inputs as they lie in memory: earlier ones, the token's own
    T old[kTaps - 1], x, z;
    float w[kTaps], bias;
  };
  const T* decay = reinterpret_cast<const T*>(p.decay) + s.first * p.ld_decay + h * p.dim;
  const long long last_tap = (long long)in.back * p.channels;
  const int channels = 2 * DP + p.nc;
  auto place = [&](int x, int& part, int& d) {
    part = x < DP ? 0 : x < 2 * DP ? 1 : 2;
    d = x - part * DP + (part == 2 ? c_first : 0);
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
    } else if (!DELTA) {
      y = ok ? to_f32<T>(c.x) : part == 2 && d == p.vdim ? 1.f : 0.f;
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
  qk *= fq * fk * (DELTA ? 1.f : put);
  float4 P = make_float4(0.f, 0.f, 0.f, 0.f), Q = P;
#pragma unroll
  for (int i = 0; i < kRows; i += 4) {
    const float4 q = load4(sQ + r0 + i), k = load4(sK + r0 + i), g = load4(sG + r0 + i);
    const float qs[4] = {q.x, q.y, q.z, q.w}, ks[4] = {k.x, k.y, k.z, k.w}, gs[4] = {g.x, g.y, g.z, g.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {   // S <- g * S; S^T k, S^T q
      float4& x = S[i + e];
      const float f = DELTA ? gs[e] : keep;
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
    sP[c] = u * (DELTA ? fk : put);   // what the rows' keys are multiplied by
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
    if (!DELTA && slice == 0 && tid == 0) dst[p.ncols] = expf(-m_new);
  } else {   // every warp the norm, then its own columns
    float scale = DELTA ? 1.f : 1.f / (fmaxf(fabsf(sV[p.vdim]), expf(-m_new)) + 1e-6f), ss = 0.f;
    for (int c = lane; c < p.vdim; c += 32) {
      const float x = sV[c] * scale;
      ss = fmaf(x, x, ss);
    }
    scale *= 1.f / sqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
    T* dst = reinterpret_cast<T*>(p.out) + s.first * p.ldo + (long long)h * p.vdim;
    for (int c = tid; c < p.vdim; c += threads)
      dst[c] = from_f32<T>(sV[c] * scale * (c == tid ? norm0 : norm[c]) *
                           sigmoid_f(to_f32<T>(c == tid ? gate0 : gate[c])));
  }
  if (DELTA) {
    if (p.taps > kTaps) save_inputs<T>(p, s, in, qk_block, c_first, max(0, nv));
  } else if (slice == 0 && tid == 0)
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
template <typename T, int DP, bool DELTA>
__global__ void __launch_bounds__(DP <= 128 ? 128 : 256) tile_kernel(const ScanArgs p) {
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
  if (DELTA) {
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
        const int one = part == 2 ? p.vdim - d : -1;   // the normaliser's column
#pragma unroll
        for (int t = 0; t < kTT; ++t) {
          float4 y = ok && t < nt ? in.four(part, d, t0 + t) : zero;
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
          }
        }
        if (!DELTA && part == 2 && d + e == p.vdim) y[e] = 1.f;
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
      const float b = kn * __expf((DELTA ? 0.f : invK[t]) - l);
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

template <typename T, int DP, bool DELTA, int STAGES>
__global__ void __launch_bounds__(max_warps(DELTA) * 32, 1) scan_kernel(const ScanArgs p) {
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
    put_zeros<T, DELTA>(p, s, h, slice);
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
    if (p.vec_out && o_t < nt)   // the first outputs' gates, ahead
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
        if (!DELTA && slice == 0 && lane == 0) dst[p.ncols] = st[R::kBeta + t];
      }
    } else if (p.vec_out) {
      vector_outputs<T, DELTA>(p, sV, nc, st + R::kBeta, nt, lanes, gate + (long long)t0 * p.ld_gate,
                               out + (long long)t0 * p.ldo, w, gates, wa, wb);
    } else {
      for (int t = warp; t < nt; t += threads / 32)
        head_output<T, DELTA>(p, sV + t * nc, s.first + t0 + t, h, st[R::kBeta + t]);
    }
  }
  copies_wait<0>();
  store_state<DP>(S, state, p, rl, c_first + c_local);
}

// ------------------------------------------------------------------ the same on tensor cores
// A record, in bytes: a (delta), b and c as pairs of bf16 matrices [kTT][kLd], the solving matrix
// (delta) and c . b as pairs [kTT][kLdT], decays, step sizes (memory: exp(-m)), values fp32 [kTT][vld].
template <int DP, bool DELTA>
struct MmaRecord {
  static constexpr int kLd = DP + 8, kLdT = kTT + 8;    // rows shifted over the banks
  static constexpr int kMat = kTT * kLd * 2, kSmall = kTT * kLdT * 2;
  static constexpr int kB = 0, kC = 2 * kMat, kA = 4 * kMat, kQ = (DELTA ? 6 : 4) * kMat;
  static constexpr int kT = kQ + 2 * kSmall, kG = kT + (DELTA ? 2 * kSmall : 0);
  static constexpr int kBeta = kG + 4 * DP * 4, kGroups = kBeta + kTT * 4, kV = kGroups + 16;
  __host__ __device__ static constexpr int vld(int cols) { return cols + 4; }
  __host__ __device__ static constexpr int bytes(int cols) { return kV + kTT * vld(cols) * 4; }
};

template <int DP, bool DELTA>
__global__ void __launch_bounds__(DP <= 128 ? 128 : 256, DP > 128 ? 2 : DELTA ? 4 : 6) tile_mma_kernel(const ScanArgs p) {
  typedef __nv_bfloat16 T;
  using R = MmaRecord<DP, DELTA>;
  constexpr int kThreads = DP <= 128 ? 128 : 256, kWarps = kThreads / 32, kLd = R::kLd;
  extern __shared__ __align__(16) float sm[];
  float* sB = sm;                                // keys
  float* sC = sm + kTT * DP;                     // queries
  uint8_t* mats = reinterpret_cast<uint8_t*>(sm + 2 * kTT * DP);   // the record up to its values
  constexpr int kTriLd = kTT + 4;
  float* tri = reinterpret_cast<float*>(mats + R::kV);             // [kTT][kTriLd]
  __shared__ float invQ[kTT], invK[kTT], beta[kTT];   // memory: log decay, log input factor, exp(-m)
  pdl_wait();
  pdl_trigger();
  const int h = blockIdx.x % p.heads;
  const long long tile = blockIdx.x / p.heads;
  const int* tl = p.tiles + tile * 2;
  const Seq s(p.steps + (long long)tl[0] * kStepInts);
  if (s.slot <= 0 || s.slot >= p.num_slots) return;
  const int t0 = tl[1], nt = min(kTT, s.n - t0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  uint8_t* rec = reinterpret_cast<uint8_t*>(p.records) + (tile * p.heads + h) * p.record * 4;
  const Inputs<T> in(p, s, h, DELTA);
  const int vcols = p.slices * p.nc, vld = R::vld(vcols);
  float* rec_v = reinterpret_cast<float*>(rec + R::kV);

  // Decays: a thread has two channels and eight of the tokens; lane ^ 16 has the others.
  const int d0 = 2 * ((tid & 15) + (tid >> 5) * 16), half = (tid >> 4) & 1;
  uint32_t zr[8] = {};
  float2 z[8];
  float2 bias = make_float2(0.f, 0.f);
  float ae = 0.f;
  if (DELTA) {
    if (d0 < p.dim) {
      const T* src = reinterpret_cast<const T*>(p.decay) + (s.first + t0 + half * 8) * p.ld_decay + h * p.dim + d0;
      const bool two = d0 + 1 < p.dim;
      ae = -kLog2e * p.a_exp[h];     // (logs are to base 2 from here on)
      bias.x = p.dt_bias[h * p.dim + d0];
      if (two) bias.y = p.dt_bias[h * p.dim + d0 + 1];
      const int mine = nt - half * 8;
      if (p.vec) {
#pragma unroll
        for (int t = 0; t < 8; ++t)
          if (t < mine) zr[t] = *reinterpret_cast<const uint32_t*>(src + t * p.ld_decay);
      } else {
#pragma unroll
        for (int t = 0; t < 8; ++t)
          if (t < mine)
            zr[t] = pack_bf16x2(to_f32<T>(src[t * p.ld_decay]), two ? to_f32<T>(src[t * p.ld_decay + 1]) : 0.f);
      }
    }
    if (tid < kTT)
      beta[tid] = tid < nt ? sigmoid_f(to_f32<T>(in.proj[(long long)(t0 + tid) * p.ld + p.b_at + h])) : 0.f;
  } else if (tid < kTT) {
    const float* g = p.gates + ((s.first + t0 + tid) * p.heads + h) * 3;
    const bool ok = tid < nt;
    invQ[tid] = ok ? g[0] * kLog2e : 0.f;
    invK[tid] = ok ? g[1] * kLog2e : 0.f;
    beta[tid] = ok ? expf(-g[2]) : 1.f;
  }

  // ---- 1. queries, keys, values: four channels and all of the tile's tokens a thread
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int x = tid * 4; x < 2 * DP + vcols; x += kThreads * 4) {
    const int part = x < DP ? 0 : x < 2 * DP ? 1 : 2;
    const int d = x - part * DP, limit = part == 2 ? p.vdim : p.dim;
    float* dst = part == 2 ? rec_v + d : (part == 0 ? sC : sB) + d;
    const int dst_ld = part == 2 ? vld : DP;
    if (p.vec && (!DELTA || p.taps <= kTaps)) {
      const bool ok = d < limit;
      const T* src = in.proj + (long long)t0 * p.ld + in.col(part) + (ok ? d : 0);
      if constexpr (DELTA) {
        // all loads at once: the tile's tokens, the ones before it, the taps (the last one is the
        // current token's)
        uint2 raw[kTT];
#pragma unroll
        for (int t = 0; t < kTT; ++t, src += p.ld) {
          raw[t] = make_uint2(0u, 0u);
          if (t < nt) raw[t] = *reinterpret_cast<const uint2*>(src);
        }
        float4 w[kTaps], v[kTaps + 3];
        const float* cw = p.conv + in.ch(part) + (ok ? d : 0);
#pragma unroll
        for (int j = 0; j < kTaps - 1; ++j)
          v[j] = ok && j >= kTaps - p.taps ? in.four(part, d, t0 + j - (kTaps - 1)) : zero;
#pragma unroll
        for (int j = 0; j < kTaps; ++j) {
          const int k = j - (kTaps - p.taps);
          w[j] = k >= 0 ? load4(cw + (long long)k * p.channels) : zero;
        }
#pragma unroll
        for (int tb = 0; tb < kTT; tb += 4) {
#pragma unroll
          for (int t = 0; t < 4; ++t) v[kTaps - 1 + t] = widen(raw[tb + t].x, raw[tb + t].y);
#pragma unroll
          for (int t = 0; t < 4; ++t) {
            float4 y = zero;
#pragma unroll
            for (int j = 0; j < kTaps; ++j) axpy4(y, w[j], v[t + j]);
            store4(dst, ok && tb + t < nt ? silu4(y) : zero);
            dst += dst_ld;
          }
#pragma unroll
          for (int j = 0; j < kTaps - 1; ++j) v[j] = v[4 + j];
        }
      } else {
        const int one = part == 2 ? p.vdim - d : -1;   // the normaliser's column
#pragma unroll
        for (int t = 0; t < kTT; ++t, src += p.ld, dst += dst_ld) {
          float4 y = ok && t < nt ? load4(src) : zero;
          if (one == 0) y.x = 1.f;
          if (one == 1) y.y = 1.f;
          if (one == 2) y.z = 1.f;
          if (one == 3) y.w = 1.f;
          store4(dst, y);
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
          }
        }
        if (!DELTA && part == 2 && d + e == p.vdim) y[e] = 1.f;
      }
      store4(dst + t * dst_ld, make_float4(y[0], y[1], y[2], y[3]));
    }
  }
  // cumulative log decays
  float2 cum = make_float2(0.f, 0.f);
  if (DELTA) {
#pragma unroll
    for (int t = 0; t < 8; ++t) {
      if (half * 8 + t < nt) {
        const float zx = __uint_as_float(zr[t] << 16), zy = __uint_as_float(zr[t] & 0xffff0000u);
        cum.x += fmaxf(ae * softplus_f(zx + bias.x), kMinLogDecay * kLog2e);
        cum.y += fmaxf(ae * softplus_f(zy + bias.y), kMinLogDecay * kLog2e);
      }
      z[t] = cum;
    }
    const float bx = __shfl_xor_sync(0xffffffffu, cum.x, 16), by = __shfl_xor_sync(0xffffffffu, cum.y, 16);
    if (half) {
#pragma unroll
      for (int t = 0; t < 8; ++t) z[t] = make_float2(z[t].x + bx, z[t].y + by);
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
  } else {
    float c = 0.f;
    for (int t = 0; t < half * 8; ++t) c += invQ[t];
#pragma unroll
    for (int t = 0; t < 8; ++t) {
      c += invQ[half * 8 + t];
      z[t] = make_float2(c, c);
    }
  }
  // one group of tokens, or two or four where 1 / G would leave its range
  const float2 other = make_float2(__shfl_xor_sync(0xffffffffu, z[7].x, 16),
                                   __shfl_xor_sync(0xffffffffu, z[7].y, 16));
  const float2 first = half ? other : z[7], whole = half ? z[7] : other;   // logs of the half, the tile
  const float low = kTileLogDecay * kLog2e;
  const bool deep = __syncthreads_or(fminf(whole.x, whole.y) < low);
  const bool deeper = __syncthreads_or(fminf(fminf(first.x, first.y),
                                             fminf(whole.x - first.x, whole.y - first.y)) < low);
  const int groups = !deep ? 1 : !deeper ? 2 : kTT / kB;
  // ---- 3. a, b, c and the groups' decays
  if (tid < DP) {
    float2 base = half && groups > 1 ? first : make_float2(0.f, 0.f);   // logs at the group's start
    float* G = reinterpret_cast<float*>(mats + R::kG);
#pragma unroll
    for (int t = 0; t < 8; ++t) {
      const int tok = half * 8 + t;
      const float lx = z[t].x - base.x, ly = z[t].y - base.y;
      const float gx = exp2_fast(lx), gy = exp2_fast(ly);
      const float2 k = *reinterpret_cast<const float2*>(sB + tok * DP + d0);
      const float2 q = *reinterpret_cast<const float2*>(sC + tok * DP + d0);
      const float fk = DELTA ? invK[tok] : 1.f, fq = DELTA ? invQ[tok] : p.q_scale;
      const float put = DELTA ? 0.f : invK[tok];
      const float kx = k.x * fk, ky = k.y * fk;
      auto split_to = [&](int at, float x, float y) {
        uint32_t hi, lo;
        split2(x, y, hi, lo);
        *reinterpret_cast<uint32_t*>(mats + at + (tok * kLd + d0) * 2) = hi;
        *reinterpret_cast<uint32_t*>(mats + at + R::kMat + (tok * kLd + d0) * 2) = lo;
      };
      split_to(R::kB, kx * exp2_fast(put - lx), ky * exp2_fast(put - ly));
      split_to(R::kC, q.x * fq * gx, q.y * fq * gy);
      if (DELTA) split_to(R::kA, kx * gx, ky * gy);
      if (tok % kB == kB - 1) {
        *reinterpret_cast<float2*>(G + tok / kB * DP + d0) = make_float2(gx, gy);
        if (groups == kTT / kB) base = z[t];
      }
    }
  }
  if (tid < kTT) reinterpret_cast<float*>(mats + R::kBeta)[tid] = beta[tid];
  if (tid == 0) *reinterpret_cast<float4*>(mats + R::kGroups) = make_float4((float)groups, 0.f, 0.f, 0.f);
  __syncthreads();
  // ---- 4. products of the tokens: the first warp c . b, the second a . b; the others write the rest out
  constexpr int kGram = DELTA ? 2 : 1;
  if (warp >= kGram) {
    constexpr int kSkip = (R::kG - R::kQ) / 16, kAll = R::kV / 16 - kSkip;
    for (int x = tid - kGram * 32; x < kAll; x += kThreads - kGram * 32) {
      const int y = x < R::kQ / 16 ? x : x + kSkip;
      reinterpret_cast<uint4*>(rec)[y] = reinterpret_cast<const uint4*>(mats)[y];
    }
  } else {
    const uint32_t mb = smem_u32(mats);
    const int m = lane >> 3, rr = lane & 7;
    const uint32_t la = mb + (warp == 0 ? R::kC : R::kA) + (((m & 1) * 8 + rr) * kLd + (m >> 1) * 8) * 2;
    const uint32_t lb = mb + R::kB + (((m >> 1) * 8 + rr) * kLd + (m & 1) * 8) * 2;
    float acc[2][4] = {};
#pragma unroll
    for (int k = 0; k < DP / 16; ++k) {
      uint32_t ah[4], al[4], bh[4], bl[4];
      load_matrices(ah, la + k * 32);
      load_matrices(al, la + R::kMat + k * 32);
      load_matrices(bh, lb + k * 32);
      load_matrices(bl, lb + R::kMat + k * 32);
      mma_split(acc, ah, al, bh, bl);
    }
    const int g = lane >> 2, t2 = (lane & 3) * 2;
#pragma unroll
    for (int nb = 0; nb < 2; ++nb)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int i = g + (e >> 1) * 8, j = nb * 8 + t2;
        const bool same = i * groups / kTT == j * groups / kTT;   // (j and j + 1 are of one group)
        if (warp == 0) {
          uint32_t hi, lo;
          split2(same && j <= i ? acc[nb][e] : 0.f, same && j + 1 <= i ? acc[nb][e + 1] : 0.f, hi, lo);
          *reinterpret_cast<uint32_t*>(rec + R::kQ + (i * R::kLdT + j) * 2) = hi;
          *reinterpret_cast<uint32_t*>(rec + R::kQ + R::kSmall + (i * R::kLdT + j) * 2) = lo;
        } else {
          *reinterpret_cast<float2*>(tri + i * kTriLd + j) =
              make_float2(same && j < i ? beta[i] * acc[nb][e] : 0.f,
                          same && j + 1 < i ? beta[i] * acc[nb][e + 1] : 0.f);
        }
      }
    if (DELTA && warp == 1) {   // (I + diag(beta) a b^T)^-1, a column a lane
      __syncwarp();
      const int c = lane & 15;
      float x[kTT];
#pragma unroll
      for (int i = 0; i < kTT; ++i) {
        float v0 = i == c ? 1.f : 0.f, v1 = 0.f;
#pragma unroll
        for (int j = 0; j < i; j += 4) {
          const float4 t = load4(tri + i * kTriLd + j);
          v0 = fmaf(-t.x, x[j], v0);
          if (j + 1 < i) v1 = fmaf(-t.y, x[j + 1], v1);
          if (j + 2 < i) v0 = fmaf(-t.z, x[j + 2], v0);
          if (j + 3 < i) v1 = fmaf(-t.w, x[j + 3], v1);
        }
        x[i] = v0 + v1;
      }
      // lanes 0 - 15 write the first part of the split, 16 - 31 the second
      __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(rec + R::kT + (lane >> 4) * R::kSmall) + c;
#pragma unroll
      for (int i = 0; i < kTT; ++i) {
        const __nv_bfloat16 hi = __float2bfloat16(x[i]);
        dst[i * R::kLdT] = lane < 16 ? hi : __float2bfloat16(x[i] - __bfloat162float(hi));
      }
    }
  }
  if (DELTA && t0 + nt == s.n) save_inputs<T>(p, s, in, h % p.group == 0, 0, p.vdim);
}

// Two warps own 16 columns, half of the rows each: Z transposed, as accumulators of 16 columns by 8 rows.
// They add up their read-outs through shared memory; the first one writes the outputs.
__device__ __forceinline__ void pair_sync(int pair) {
  asm volatile("bar.sync %0, 64;" ::"r"(1 + pair) : "memory");
}
// floats a lane of a pair swaps: both halves of P, one of O
__host__ __device__ constexpr int swap_floats(bool delta) { return delta ? 24 : 8; }

template <int DP, bool DELTA, int STAGES>
__global__ void __launch_bounds__(max_warps(DELTA) * 64, 1) scan_mma_kernel(const ScanArgs p) {
  typedef __nv_bfloat16 T;
  using R = MmaRecord<DP, DELTA>;
  constexpr int kSwap = swap_floats(DELTA);
  constexpr int kN = DP / 16, kSteps = DP / 32, kLd = R::kLd;   // of a warp's half of the rows
  extern __shared__ __align__(16) uint8_t smem[];
  pdl_wait();
  pdl_trigger();
  const int slice = blockIdx.x % p.slices, h = blockIdx.x / p.slices % p.heads;
  const int seq = blockIdx.x / p.slices / p.heads;
  const Seq s(p.steps + (long long)seq * kStepInts);
  if (s.n <= 0) return;
  if (s.slot <= 0 || s.slot >= p.num_slots) {
    put_zeros<T, DELTA>(p, s, h, slice);
    return;
  }
  const int tid = threadIdx.x, threads = blockDim.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t2 = (lane & 3) * 2;
  const int pairs = p.nc / 16, second = warp >= pairs, pair = warp - second * pairs;
  const int nc = p.nc, c_first = slice * nc, vld = R::vld(nc), rec_vld = R::vld(p.slices * nc);
  const int stage_size = R::bytes(nc);
  float* swap = reinterpret_cast<float*>(smem + STAGES * stage_size) + pair * kSwap * 32 + lane;
  const int tiles = (s.n + kTT - 1) / kTT;
  const uint8_t* rec0 = reinterpret_cast<const uint8_t*>(p.records) +
                        ((long long)p.first_tile[seq] * p.heads + h) * p.record * 4;
  auto copy16 = [](uint8_t* dst, const uint8_t* src) {
    copy16_async(reinterpret_cast<float*>(dst), reinterpret_cast<const float*>(src));
  };
  auto fetch = [&](int i) {   // (one group of copies per tile, also when there is none)
    if (i < tiles) {
      const uint8_t* src = rec0 + (long long)i * p.heads * p.record * 4;
      uint8_t* dst = smem + i % STAGES * stage_size;
      for (int x = tid * 16; x < R::kV; x += threads * 16) copy16(dst + x, src + x);
      const int per = nc / 4;
      for (int x = tid; x < kTT * per; x += threads) {
        const int t = x / per, c = (x - t * per) * 4;
        copy16(dst + R::kV + (t * vld + c) * 4, src + R::kV + (t * rec_vld + c_first + c) * 4);
      }
    }
    copies_commit();
  };
  // (a tile's outputs are written out while the next one's are computed: two stages are in use)
#pragma unroll
  for (int i = 0; i < STAGES - 2; ++i) fetch(i);
  // state: Z[n]: columns c and c + 8, rows r0 + 8 n + t2 and the next
  float* state = p.state + ((long long)s.slot * p.heads + h) * p.dim * p.state_cols;
  const int c0 = c_first + pair * 16 + g, r0 = second * (DP / 2);
  float Z[kN][4];
#pragma unroll
  for (int n = 0; n < kN; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = r0 + 8 * n + t2 + (e & 1), c = c0 + (e >> 1) * 8;
      Z[n][e] = s.start > 0 && r < p.dim && c < p.state_cols ? state[(long long)r * p.state_cols + c] : 0.f;
    }
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
  // ldmatrix addresses within a stage: right operands with tokens as columns, and as rows
  const int m = lane >> 3, rr = lane & 7;
  const uint32_t tok_cols = (((m >> 1) * 8 + rr) * kLd + (m & 1) * 8 + r0) * 2;
  const uint32_t tok_cols_t = (((m >> 1) * 8 + rr) * R::kLdT + (m & 1) * 8) * 2;
  const uint32_t tok_rows = (((m & 1) * 8 + rr) * kLd + (m >> 1) * 8 + r0) * 2;

  // norm, weight and gate of a tile's outputs
  Raw8<T> gates = {};
  auto put_out = [&](int it) {
    const int t0 = it * kTT, nt = min(kTT, s.n - t0);
    uint8_t* st = smem + it % STAGES * stage_size;
    const float* beta = reinterpret_cast<const float*>(st + R::kBeta);
    float* sV = reinterpret_cast<float*>(st + R::kV);
    if (p.raw != nullptr) {
      for (int t = warp; t < nt; t += threads / 32) {
        float* dst = p.raw + ((s.first + t0 + t) * p.heads + h) * p.raw_cols + c_first;
        for (int c = lane; c < min(nc, p.ncols - c_first); c += 32) dst[c] = sV[t * vld + c];
        if (!DELTA && slice == 0 && lane == 0) dst[p.ncols] = beta[t];
      }
    } else if (p.vec_out) {
      vector_outputs<T, DELTA>(p, sV, vld, beta, nt, lanes, gate + (long long)t0 * p.ld_gate,
                               out + (long long)t0 * p.ldo, w, gates, wa, wb);
    } else {
      for (int t = warp; t < nt; t += threads / 32)
        head_output<T, DELTA>(p, sV + t * vld, s.first + t0 + t, h, beta[t]);
    }
  };

  for (int it = 0; it < tiles; ++it) {
    const int t0 = it * kTT, nt = min(kTT, s.n - t0);
    copies_wait<STAGES - 3>();
    __syncthreads();       // the tile's record and the outputs of the tile before are there
    fetch(it + STAGES - 2);   // (into the stage of two tiles before, whose outputs are written)
    uint8_t* st = smem + it % STAGES * stage_size;
    const uint32_t sb = smem_u32(st);
    const float* beta = reinterpret_cast<const float*>(st + R::kBeta);
    float* sV = reinterpret_cast<float*>(st + R::kV);
    const int groups = (int)*reinterpret_cast<const float*>(st + R::kGroups);
    if (it > 0) put_out(it - 1);
    if (p.vec_out && o_t < nt)   // the first outputs' gates, ahead
      gates.load(gate + (long long)(t0 + o_t) * p.ld_gate + o_c);
    for (int grp = 0; grp < groups; ++grp) {
      // read-outs [16 columns x 16 tokens]: P, what is put (U = beta (v - P), solved), O
      float P[2][4] = {}, O[2][4] = {}, U[2][4];
      uint32_t uh[4], ul[4], bh[4], bl[4];
      auto mine = [&](int tok) { return tok * groups / kTT == grp; };   // (other groups wait)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e)
          U[n][e] = sV[(n * 8 + t2 + (e & 1)) * vld + pair * 16 + g + (e >> 1) * 8];
#pragma unroll
      for (int k = 0; k < kSteps; ++k) {
        uint32_t zh[4], zl[4];
        split_left(Z[2 * k], Z[2 * k + 1], zh, zl);
        if constexpr (DELTA) {
          load_matrices(bh, sb + R::kA + tok_cols + k * 32);
          load_matrices(bl, sb + R::kA + R::kMat + tok_cols + k * 32);
          mma_split(P, zh, zl, bh, bl);
        }
        load_matrices(bh, sb + R::kC + tok_cols + k * 32);
        load_matrices(bl, sb + R::kC + R::kMat + tok_cols + k * 32);
        mma_split(O, zh, zl, bh, bl);
      }
      // the other half's sums: both warps need P, the first one O
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          if (DELTA) swap[(second * 8 + n * 4 + e) * 32] = P[n][e];
          if (second) swap[((DELTA ? 16 : 0) + n * 4 + e) * 32] = O[n][e];
        }
      pair_sync(pair);
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          if (DELTA) P[n][e] += swap[((second ^ 1) * 8 + n * 4 + e) * 32];
          if (!second) O[n][e] += swap[((DELTA ? 16 : 0) + n * 4 + e) * 32];
        }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int tok = n * 8 + t2 + (e & 1);
          if (DELTA) U[n][e] = beta[tok] * (U[n][e] - P[n][e]);
          if (!mine(tok)) U[n][e] = 0.f;
        }
      split_left(U[0], U[1], uh, ul);
      if constexpr (DELTA) {
        load_matrices(bh, sb + R::kT + tok_cols_t);
        load_matrices(bl, sb + R::kT + R::kSmall + tok_cols_t);
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) U[n][e] = 0.f;
        mma_split(U, uh, ul, bh, bl);
      }
      if constexpr (DELTA) split_left(U[0], U[1], uh, ul);
      if (!second) {
        load_matrices(bh, sb + R::kQ + tok_cols_t);
        load_matrices(bl, sb + R::kQ + R::kSmall + tok_cols_t);
        mma_split(O, uh, ul, bh, bl);
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) {   // (where the value was, which both warps have read)
            const int tok = n * 8 + t2 + (e & 1);
            if (mine(tok)) sV[tok * vld + pair * 16 + g + (e >> 1) * 8] = O[n][e];
          }
      }
      const float* G = reinterpret_cast<const float*>(st + R::kG) + ((grp + 1) * (kTT / kB) / groups - 1) * DP + r0 + t2;
#pragma unroll
      for (int n = 0; n < kN; n += 2) {
        load_matrices_trans(bh, sb + R::kB + tok_rows + n * 16);
        load_matrices_trans(bl, sb + R::kB + R::kMat + tok_rows + n * 16);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          mma_bf16(Z[n + e], uh, bl[2 * e], bl[2 * e + 1]);
          mma_bf16(Z[n + e], ul, bh[2 * e], bh[2 * e + 1]);
          mma_bf16(Z[n + e], uh, bh[2 * e], bh[2 * e + 1]);
          const float2 f = *reinterpret_cast<const float2*>(G + 8 * (n + e));
          Z[n + e][0] *= f.x; Z[n + e][1] *= f.y;
          Z[n + e][2] *= f.x; Z[n + e][3] *= f.y;
        }
      }
      if (groups > 1) pair_sync(pair);   // (the sums are swapped once more)
    }
  }
  copies_wait<0>();
  __syncthreads();
  put_out(tiles - 1);
#pragma unroll
  for (int n = 0; n < kN; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = r0 + 8 * n + t2 + (e & 1), c = c0 + (e >> 1) * 8;
      if (r < p.dim && c < p.state_cols) state[(long long)r * p.state_cols + c] = Z[n][e];
    }
}

// Heads whose columns several blocks share: norm, weight and gate of the raw outputs. A warp per
// (token, head).
template <typename T, bool DELTA>
__global__ void __launch_bounds__(256) scan_output_kernel(const ScanArgs p, long long n) {
  pdl_wait();
  pdl_trigger();
  const long long k = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (k >= n) return;
  const float* o = p.raw + k * p.raw_cols;
  head_output<T, DELTA>(p, o, k / p.heads, (int)(k % p.heads), DELTA ? 0.f : o[p.vdim + 1]);
}

template <typename K>
static bool set_smem(K k, size_t bytes) {
  return bytes <= 40 * 1024 ||
         cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) == cudaSuccess;
}

template <typename T, int DP, bool DELTA>
static int launch_scan(const ScanArgs& a, int n_seq, int n_tiles, int max_rows, cudaStream_t stream) {
  // (one-token steps and 32-bit models; on tensor cores a warp has 16 columns)
  const int wc = a.warp_cols;
  if (a.nc % wc || a.nc / wc > max_warps(DELTA) || (long long)a.nc * (a.slices - 1) >= a.ncols ||
      (long long)a.nc * a.slices < a.ncols)
    return -2;
  const long long blocks = (long long)n_seq * a.heads * a.slices;
  const dim3 threads(a.nc / wc * 32);
  if (blocks > 0x7fffffffll || (long long)n_tiles * a.heads > 0x7fffffffll) return -6;
  if (max_rows == 1) {
    using Sh = StepShape<DP>;
    const size_t smem = (size_t)Sh::smem_floats(a.nc) * sizeof(float);
    const dim3 step_threads(a.nc / 4 * Sh::kGroups);
    if (step_threads.x > Sh::max_threads(DELTA)) return -2;
    if (!set_smem(step_kernel<T, DP, DELTA>, smem)) return -3;
    return launch_pdl(step_kernel<T, DP, DELTA>, dim3((unsigned)blocks), step_threads, smem, stream, a) ==
                   cudaSuccess
               ? 0
               : -5;
  }
  if (n_tiles < 1 || a.records == nullptr || a.tiles == nullptr || a.first_tile == nullptr ||
      a.record < (sizeof(T) == 2 ? MmaRecord<DP, DELTA>::bytes(a.nc * a.slices) / 4
                                 : stage_floats<DP, DELTA>(a.nc * a.slices)))
    return -2;
  if (!DELTA && launch_pdl(memory_gates_kernel<T>, dim3((unsigned)(n_seq * a.heads)),
                           dim3(max_rows <= 128 ? 128 : max_rows <= 512 ? 512 : 1024), 0, stream,
                           a) != cudaSuccess)
    return -5;
  const dim3 tile_grid((unsigned)(n_tiles * a.heads)), tile_threads(DP <= 128 ? 128 : 256);
  if constexpr (sizeof(T) == 2) {
    using R = MmaRecord<DP, DELTA>;
    const size_t tile_smem = (size_t)2 * kTT * DP * 4 + R::kV + kTT * (kTT + 4) * 4;
    if (!set_smem(tile_mma_kernel<DP, DELTA>, tile_smem)) return -3;
    if (launch_pdl(tile_mma_kernel<DP, DELTA>, tile_grid, tile_threads, tile_smem, stream, a) != cudaSuccess)
      return -5;
    const size_t stage = R::bytes(a.nc);
    const size_t swap = (size_t)a.nc / 16 * swap_floats(DELTA) * 32 * 4;
    const bool four = 4 * stage + swap <= 220 * 1024;
    auto k = four ? scan_mma_kernel<DP, DELTA, 4> : scan_mma_kernel<DP, DELTA, 3>;
    const size_t smem = (four ? 4 : 3) * stage + swap;
    if (smem > 220 * 1024) return -6;
    if (!set_smem(k, smem)) return -3;
    return launch_pdl(k, dim3((unsigned)blocks), dim3(a.nc / 16 * 64), smem, stream, a) == cudaSuccess ? 0 : -5;
  } else {
    const size_t tile_smem = (size_t)(DELTA ? 3 : 2) * kTT * DP * sizeof(float);
    if (!set_smem(tile_kernel<T, DP, DELTA>, tile_smem)) return -3;
    if (launch_pdl(tile_kernel<T, DP, DELTA>, tile_grid, tile_threads, tile_smem, stream, a) != cudaSuccess)
      return -5;
    const size_t stage = (size_t)stage_floats<DP, DELTA>(a.nc) * sizeof(float);
    const bool three = 3 * stage <= 220 * 1024;
    auto k = three ? scan_kernel<T, DP, DELTA, 3> : scan_kernel<T, DP, DELTA, 2>;
    const size_t smem = (three ? 3 : 2) * stage;
    if (smem > 220 * 1024) return -6;
    if (!set_smem(k, smem)) return -3;
    return launch_pdl(k, dim3((unsigned)blocks), threads, smem, stream, a) == cudaSuccess ? 0 : -5;
  }
}

template <typename T, bool DELTA>
static int run_scan(const ScanArgs& a, int n_seq, int n_tiles, int max_rows, long long rows,
                    cudaStream_t stream) {
  const int rc = a.dim <= 32    ? launch_scan<T, 32, DELTA>(a, n_seq, n_tiles, max_rows, stream)
                 : a.dim <= 64  ? launch_scan<T, 64, DELTA>(a, n_seq, n_tiles, max_rows, stream)
                 : a.dim <= 128 ? launch_scan<T, 128, DELTA>(a, n_seq, n_tiles, max_rows, stream)
                 : a.dim <= 256 ? launch_scan<T, 256, DELTA>(a, n_seq, n_tiles, max_rows, stream)
                                : -6;
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

// Columns of a warp: on tensor cores (16-bit models, portions of several tokens) always 16
static int warp_cols(int dim, int dtype, bool several) {
  return dim <= 128 || (several && dtype == 0) ? 16 : 8;
}

// The common part of both entry points
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
int ab200_scan_min_slices(int dim, int ncols, int delta, int dtype, int several) {
  if (dim < 1 || dim > 256) return 0;
  const int most = max_warps(delta != 0) * warp_cols(dim, dtype, several != 0);
  return (ncols + most - 1) / most;
}

// Floats of a tile's record of a head (portions of more than one token).
long long ab200_scan_record(int dim, int ncols, int slices, int delta, int dtype) {
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
  a.record = ab200_scan_record(dim, vdim, slices, 1, dtype);
  a.heads = heads; a.group = heads / kv_heads; a.dim = dim; a.vdim = vdim;
  a.taps = taps;
  a.channels = 2 * kv_heads * dim + heads * vdim;
  a.eps = eps;
  a.out = out; a.ldo = ldo;
  a.status = status;
  finish_args(a, slices, vdim, vdim, raw, dtype, max_rows > 1);
  return dtype == 0 ? run_scan<bf16, true>(a, n_seq, n_tiles, max_rows, T, stream)
                    : run_scan<float, true>(a, n_seq, n_tiles, max_rows, T, stream);
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
  a.record = ab200_scan_record(dim, vdim + 1, slices, 0, dtype);
  a.gates = reinterpret_cast<float*>(gates);
  a.heads = heads; a.group = 1; a.dim = dim; a.vdim = vdim;
  a.taps = 1;
  a.eps = eps;
  a.out = out; a.ldo = ldo;
  a.status = status;
  finish_args(a, slices, vdim + 1, vdim + 2, raw, dtype, max_rows > 1);
  return dtype == 0 ? run_scan<bf16, false>(a, n_seq, n_tiles, max_rows, T, stream)
                    : run_scan<float, false>(a, n_seq, n_tiles, max_rows, T, stream);
}

}  // extern "C"
