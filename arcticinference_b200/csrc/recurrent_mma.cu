// Portions of several tokens of recurrent layers on tensor cores, for 16-bit models (recurrent.cu has the
// formulas, one-token steps and 32-bit models). mma.sync: Z lives in the registers of the warps that own
// its columns, as the accumulator of the update and, converted in place, as the left operand of the
// read-outs; nothing but the small token-side operands passes through shared memory. Every operand is the
// sum of two bf16 numbers, so that products carry 16 significant bits, and sums and Z are fp32. A tile's 16
// tokens are one group, solved with the inverse of the unit triangular matrix that its a, b and beta form.

#include "api.h"
#include "common/recurrent.cuh"

namespace ab200 {

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
template <int DP, int RULE>
__global__ void __launch_bounds__(DP <= 128 ? 128 : 256, DP > 128 ? 2 : RULE == kMemory ? 6 : 4)
tile_mma_kernel(const ScanArgs p) {
  typedef __nv_bfloat16 T;
  constexpr bool DELTA = RULE == kDelta, MEMORY = RULE == kMemory, FORGET = RULE == kForget;
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
  float2 bias = make_float2(0.f, 0.f), lower = bias;
  float ae = 0.f;
  if (!MEMORY) {
    if (d0 < p.dim) {
      const T* src = reinterpret_cast<const T*>(p.decay) + (s.first + t0 + half * 8) * p.ld_decay + h * p.dim + d0;
      const bool two = d0 + 1 < p.dim;
      if (DELTA) ae = -kLog2e * p.a_exp[h];     // (logs are to base 2 from here on)
      if (FORGET) {
        lower.x = p.lower[h * p.dim + d0];
        if (two) lower.y = p.lower[h * p.dim + d0 + 1];
      }
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
    if (FORGET) {
      if (tid < kTT) beta[tid] = 1.f;
    } else if (tid < kTT)
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
  const bool halves = FORGET && p.vec;
  if (halves) {   // (the keys come with the decays: enough threads for half of the tokens each)
    const int quads = (DP + vcols) / 4;
    for (int x = tid; x < 2 * quads; x += kThreads) {
      const int late = x >= quads, d_all = (x - late * quads) * 4;
      const bool query = d_all < DP;
      const int d = query ? d_all : d_all - DP;
      const bool ok = d < (query ? p.dim : p.vdim);
      const T* src = in.proj + (long long)(t0 + late * 8) * p.ld + (query ? in.q_col : in.v_col) + (ok ? d : 0);
      float* dst = query ? sC + late * 8 * DP + d : rec_v + late * 8 * vld + d;
      const int dst_ld = query ? DP : vld;
      uint2 raw[8];
#pragma unroll
      for (int t = 0; t < 8; ++t, src += p.ld) {
        raw[t] = make_uint2(0u, 0u);
        if (ok && late * 8 + t < nt) raw[t] = *reinterpret_cast<const uint2*>(src);
      }
#pragma unroll
      for (int t = 0; t < 8; ++t, dst += dst_ld) {
        const float4 y = widen(raw[t].x, raw[t].y);
        store4(dst, query ? silu4(y) : y);
      }
    }
  }
  for (int x = halves ? 2 * DP + vcols : tid * 4; x < 2 * DP + vcols; x += kThreads * 4) {
    const int part = x < DP ? 0 : x < 2 * DP ? 1 : 2;
    if (FORGET && part == 1) continue;   // (keys: with the decays)
    const int d = x - part * DP, limit = part == 2 ? p.vdim : p.dim;
    float* dst = part == 2 ? rec_v + d : (part == 0 ? sC : sB) + d;
    const int dst_ld = part == 2 ? vld : DP;
    if (!FORGET && p.vec && (!DELTA || p.taps <= kTaps)) {
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
        const int one = MEMORY && part == 2 ? p.vdim - d : -1;   // the normaliser's column
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
            if (FORGET && part == 0) y[e] = silu_f(y[e]);
          }
        }
        if (MEMORY && part == 2 && d + e == p.vdim) y[e] = 1.f;
      }
      store4(dst + t * dst_ld, make_float4(y[0], y[1], y[2], y[3]));
    }
  }
  // cumulative log decays
  float2 cum = make_float2(0.f, 0.f);
  if (!MEMORY) {
#pragma unroll
    for (int t = 0; t < 8; ++t) {
      const float zx = __uint_as_float(zr[t] << 16), zy = __uint_as_float(zr[t] & 0xffff0000u);
      if (FORGET && tid < DP) {   // and the keys
        const bool x_in = d0 < p.dim && half * 8 + t < nt, y_in = d0 + 1 < p.dim && half * 8 + t < nt;
        const float kx = x_in ? forget_put(zx + bias.x, lower.x) : 0.f;
        const float ky = y_in ? forget_put(zy + bias.y, lower.y) : 0.f;
        *reinterpret_cast<float2*>(sB + (half * 8 + t) * DP + d0) = make_float2(kx, ky);
        if (x_in) cum.x += fmaxf(forget_log2(forget_keep(zx + bias.x, lower.x), kx), kMinLogDecay * kLog2e);
        if (y_in) cum.y += fmaxf(forget_log2(forget_keep(zy + bias.y, lower.y), ky), kMinLogDecay * kLog2e);
      } else if (DELTA && half * 8 + t < nt) {
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
  } else if (MEMORY) {
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
      const float put = MEMORY ? invK[tok] : 0.f;
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

template <int DP, int RULE, int STAGES>
__global__ void __launch_bounds__(max_warps(RULE) * 64, 1) scan_mma_kernel(const ScanArgs p) {
  typedef __nv_bfloat16 T;
  constexpr bool DELTA = RULE == kDelta;
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
    put_zeros<T, RULE>(p, s, h, slice);
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
        if (RULE == kMemory && slice == 0 && lane == 0) dst[p.ncols] = beta[t];
      }
    } else if (p.vec_out) {
      vector_outputs<T, RULE>(p, sV, vld, beta, nt, lanes, gate + (long long)t0 * p.ld_gate,
                               out + (long long)t0 * p.ldo, w, gates, wa, wb);
    } else {
      for (int t = warp; t < nt; t += threads / 32)
        head_output<T, RULE>(p, sV + t * vld, s.first + t0 + t, h, beta[t]);
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
    if (RULE != kForget && p.vec_out && o_t < nt)   // the first outputs' gates, ahead
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

template <int DP, int RULE>
static int launch_tiles(const ScanArgs& a, int n_seq, int n_tiles, cudaStream_t stream) {
  const dim3 tile_grid((unsigned)(n_tiles * a.heads)), tile_threads(DP <= 128 ? 128 : 256);
  const long long blocks = (long long)n_seq * a.heads * a.slices;
  constexpr bool DELTA = RULE == kDelta;
  using R = MmaRecord<DP, DELTA>;
  const size_t tile_smem = (size_t)2 * kTT * DP * 4 + R::kV + kTT * (kTT + 4) * 4;
  if (!set_smem(tile_mma_kernel<DP, RULE>, tile_smem)) return -3;
  if (launch_pdl(tile_mma_kernel<DP, RULE>, tile_grid, tile_threads, tile_smem, stream, a) != cudaSuccess)
    return -5;
  const size_t stage = R::bytes(a.nc);
  const size_t swap = (size_t)a.nc / 16 * swap_floats(DELTA) * 32 * 4;
  const bool four = 4 * stage + swap <= 220 * 1024;
  auto k = four ? scan_mma_kernel<DP, RULE, 4> : scan_mma_kernel<DP, RULE, 3>;
  const size_t smem = (four ? 4 : 3) * stage + swap;
  if (smem > 220 * 1024) return -6;
  if (!set_smem(k, smem)) return -3;
  return launch_pdl(k, dim3((unsigned)blocks), dim3(a.nc / 16 * 64), smem, stream, a) == cudaSuccess ? 0 : -5;
}

int launch_tiles_mma(const ScanArgs& a, int rule, int n_seq, int n_tiles, cudaStream_t stream) {
#define AB200_TILES(DP)                                                    \
  (rule == kDelta    ? launch_tiles<DP, kDelta>(a, n_seq, n_tiles, stream)  \
   : rule == kForget ? launch_tiles<DP, kForget>(a, n_seq, n_tiles, stream) \
                     : launch_tiles<DP, kMemory>(a, n_seq, n_tiles, stream))
  return a.dim <= 32    ? AB200_TILES(32)
         : a.dim <= 64  ? AB200_TILES(64)
         : a.dim <= 128 ? AB200_TILES(128)
         : a.dim <= 256 ? AB200_TILES(256)
                        : -6;
#undef AB200_TILES
}

}  // namespace ab200
