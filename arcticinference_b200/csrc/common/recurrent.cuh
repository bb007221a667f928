// What the kernels of recurrent layers share: arguments, inputs, outputs (recurrent.cu says what they
// compute).
#pragma once

#include "common/elem.cuh"
#include "common/pdl.cuh"

namespace ab200 {

// The recurrences (recurrent.cu)
enum Rule : int { kMemory = 0, kDelta = 1, kForget = 2 };

// warps of a block: 128 columns of wide states, and the normaliser's beside them
__host__ __device__ constexpr int max_warps(int rule) { return rule == kMemory ? 9 : 8; }

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
  const void* decay;         // delta: [T][ld_decay], head h's channels at column h * dim; forget: the
  long long ld_decay;        // gates' projection, likewise
  const void* gate;          // output gate [T][ld_gate], head h at column h * vdim (forget: none)
  long long ld_gate;
  const float* conv;         // delta: [taps][channels]: queries', keys', values' weights
  const float* a_exp;        // delta: [heads] exp(A_log)
  const float* dt_bias;      // delta, forget: [heads][dim]
  const float* lower;        // forget: [heads][dim], lower bound of the gates
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
// Forget gate f = lower + (1 - lower) sigmoid(z): 1 - f, which keeps its digits where f is near 1
__device__ __forceinline__ float forget_put(float z, float lower) { return (1.f - lower) * sigmoid_f(-z); }
__device__ __forceinline__ float forget_keep(float z, float lower) {
  return fmaf(1.f - lower, sigmoid_f(z), lower);
}
// log2 of f; log(1 - x)'s first terms in x = 1 - f where the fast logarithm would lose them
__device__ __forceinline__ float forget_log2(float keep, float put) {
  const float series = -put * fmaf(put, fmaf(put, fmaf(put, 0.25f, 0.33333333f), 0.5f), 1.f);
  return put < 0.03f ? series * kLog2e : log2_fast(keep);
}
// log gates of the matrix memory
__device__ __forceinline__ float2 memory_log_gates(float zi, float zf, float cap) {
  const float z = cap * tanhf(zf / cap);
  return make_float2(cap * tanhf(zi / cap), fminf(z, 0.f) - log1pf(expf(-fabsf(z))));
}

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

// Outputs of padding rows: finite, no state involved
template <typename T, int RULE>
__device__ __forceinline__ void put_zeros(const ScanArgs& p, const Seq& s, int h, int slice) {
  if (s.slot >= p.num_slots && threadIdx.x == 0) report_error(p.status, kErrBounds, 50, s.slot);
  for (int t = 0; t < s.n; ++t) {
    if (p.raw != nullptr) {
      float* dst = p.raw + ((s.first + t) * p.heads + h) * p.raw_cols;
      const int c1 = min((slice + 1) * p.nc, p.ncols);
      for (int c = slice * p.nc + threadIdx.x; c < c1; c += blockDim.x) dst[c] = 0.f;
      if (RULE == kMemory && slice == 0 && threadIdx.x == 0) dst[p.ncols] = 1.f;
    } else {
      T* dst = reinterpret_cast<T*>(p.out) + (s.first + t) * p.ldo + (long long)h * p.vdim;
      for (int c = threadIdx.x; c < p.vdim; c += blockDim.x) dst[c] = from_f32<T>(0.f);
    }
  }
}

// A warp's token: norm, weight and gate (none: forget) of a head's outputs o (memory: with the
// normaliser's product in column vdim and `floor` = exp(-m)).
template <typename T, int RULE>
__device__ __forceinline__ void head_output(const ScanArgs& p, const float* o, long long row, int h,
                                            float floor) {
  const int lane = threadIdx.x & 31;
  const T* g = reinterpret_cast<const T*>(p.gate) + row * p.ld_gate + (long long)h * p.vdim;
  const float* w = p.norm + (long long)h * p.norm_step;
  T* dst = reinterpret_cast<T*>(p.out) + row * p.ldo + (long long)h * p.vdim;
  float scale = RULE != kMemory ? 1.f : 1.f / (fmaxf(fabsf(o[p.vdim]), floor) + 1e-6f);
  float ss = 0.f;
  for (int c = lane; c < p.vdim; c += 32) {
    const float x = o[c] * scale;
    ss = fmaf(x, x, ss);
  }
  scale *= 1.f / sqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
  for (int c = lane; c < p.vdim; c += 32)
    dst[c] = from_f32<T>(o[c] * scale * w[c] * (RULE == kForget ? 1.f : sigmoid_f(to_f32<T>(g[c]))));
}

// A block's tile: eight columns a thread, the `lanes` lanes of a token side by side. g, wa, wb: gate
// and norm weights of the thread's first columns.
template <typename T, int RULE>
__device__ __forceinline__ void vector_outputs(const ScanArgs& p, const float* o_tile, int ld, const float* floors,
                                               int nt, int lanes, const T* gate, T* out, const float* w,
                                               Raw8<T> g, float4 wa, float4 wb) {
  // (whole warps: the lanes of a token lie in one)
  for (int x = threadIdx.x; x < (kTT * lanes + 31) / 32 * 32; x += blockDim.x) {
    const int t = x / lanes, c = (x - t * lanes) * 8;
    const bool ok = t < nt;
    const float* o = o_tile + (ok ? t : 0) * ld;
    if (x != threadIdx.x && ok) {
      if (RULE != kForget) g.load(gate + t * p.ld_gate + c);
      wa = load4(w + c);
      wb = load4(w + c + 4);
    }
    const float4 a = load4(o + c), b = load4(o + c + 4);
    float f = RULE != kMemory ? 1.f : 1.f / (fmaxf(fabsf(o[p.vdim]), floors[ok ? t : 0]) + 1e-6f);
    float ss = dot4(a, a, dot4(b, b, 0.f)) * f * f;
    for (int k = lanes / 2; k > 0; k >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, k);
    f *= 1.f / sqrtf(ss / (float)p.vdim + p.eps);
    if (!ok) continue;
    T* dst = out + t * p.ldo + c;
    if (RULE == kForget) {
      store4(dst, make_float4(a.x * f * wa.x, a.y * f * wa.y, a.z * f * wa.z, a.w * f * wa.w));
      store4(dst + 4, make_float4(b.x * f * wb.x, b.y * f * wb.y, b.z * f * wb.z, b.w * f * wb.w));
      continue;
    }
    const float4 g0 = g.lo(), g1 = g.hi();
    store4(dst, make_float4(a.x * f * wa.x * sigmoid_f(g0.x), a.y * f * wa.y * sigmoid_f(g0.y),
                            a.z * f * wa.z * sigmoid_f(g0.z), a.w * f * wa.w * sigmoid_f(g0.w)));
    store4(dst + 4, make_float4(b.x * f * wb.x * sigmoid_f(g1.x), b.y * f * wb.y * sigmoid_f(g1.y),
                                b.z * f * wb.z * sigmoid_f(g1.z), b.w * f * wb.w * sigmoid_f(g1.w)));
  }
}

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

template <typename K>
inline bool set_smem(K k, size_t bytes) {
  return bytes <= 40 * 1024 ||
         cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) == cudaSuccess;
}

// Portions of several tokens of 16-bit models (recurrent_mma.cu).
int launch_tiles_mma(const ScanArgs& a, int rule, int n_seq, int n_tiles, cudaStream_t stream);

}  // namespace ab200
