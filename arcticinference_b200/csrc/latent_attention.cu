// Attention in latent space for sm_100a: queries [T, H, R] against a paged cache of one latent
// vector of R = 128 .. 512 numbers per token, which is key and value of every head at once.
// Decode and short chunks; softmax over the keys up to the token itself that its mask shows.
//
// The keys are the tensor core's M side. Per tile of 128 keys
//     S^T [128 keys x n]   = C Q^T       (tcgen05.mma, A = the latents K-major as they lie)
//     O^T [R x n]         += C^T P^T     (A = the same shared-memory tile read MN-major)
// with n = 16 .. 64 query rows. A row is one (token, head) pair and rows of a sequence are simply
// consecutive rows of the query matrix, so any number of heads packs without padding and a
// decode tile of 16 heads is 16 columns wide instead of 16 of 128 padded rows. Every latent is
// fetched once per tile and used twice. O^T takes R/128 * n TMEM columns (n = 48, R = 512: 192),
// which is what lets one CTA own the whole latent width.
//
// Latents arrive as 128 x 64 pieces (one 128-byte swizzle atom wide) in a ring; a piece is free
// again when its share of O^T has been accumulated.
// S of tile j + 1 is issued before O of tile j where the ring holds two tiles (R <= 256).
//
// A cache row may carry 64 more columns that belong to the key only (a rotated part that the heads
// share, beside the latent): a piece outside the ring, in one or two buffers of its own, that is
// free as soon as its share of S is done.
//
// Softmax: four warps, a thread per key. A column's maximum over the keys is a butterfly over
// the warp's lanes (16 columns in 16 shuffles) and four words of shared memory; sums stay
// per-thread until the end. O is rescaled only in tiles where a maximum moved.
//
// A sink per head is one more term of a row's sum, added at the end; an output gate per head scales
// the row as it is written.
//
// With several pieces of the keys per sequence a CTA writes normalised fp32 partials and their
// log-sum-exp, folded by the merge kernel of attention.cu (which then adds the sink and applies the gate).

#include <math.h>
#include <string.h>

#include "api.h"
#include "common/elem.cuh"
#include "common/pdl.cuh"
#include "common/ptx.cuh"
#include "common/tensormap.h"

namespace ab200 {

constexpr int kLatThreads = 192;      // 4 softmax warps, the TMA warp, the MMA warp
constexpr int kLatKeys = 128;
constexpr uint32_t kPieceBytes = kLatKeys * 64 * 2;
constexpr int kLatMaxSlots = 12;

struct LatentArgs {
  const int* work;   // [num_work][8]: sequence, first row, rows (0 = no-op), position of row r's
                     // token minus r / H, first key, last key + 1, piece, pieces
  const int* block_tables;
  int max_blocks, block_size;
  int H, pieces;           // pieces: R / 64 per tile
  int slots, p_bufs, overlap;
  int x_bufs;              // buffers of the key-only piece (0: none)
  int mask_kind, mask_size;
  float scale, scale_log2;
  uint32_t tmem_cols;
  __nv_bfloat16* out;      // [T * H][R]
  float* o_part;           // [pieces of keys][T * H][R]
  float* lse_part;         // [pieces of keys][T * H]
  long long rows_total;    // T * H
  int* status;
};

// What acts on finished rows. (A parameter of its own: as part of LatentArgs it costs the 48-row kernel
// spilled registers.)
struct LatentExt {
  const float* sink;           // [H] or null
  const __nv_bfloat16* gate;   // [T][ldg], one per head, or null
  long long ldg;
};

__device__ __forceinline__ void bar_softmax() { asm volatile("bar.sync 1, 128;" ::: "memory"); }

__device__ __forceinline__ void tmem_ld_wait_dep16(uint32_t (&r)[16]) {
  asm volatile("tcgen05.wait::ld.sync.aligned;"
               : "+r"(r[0]), "+r"(r[1]), "+r"(r[2]), "+r"(r[3]), "+r"(r[4]), "+r"(r[5]), "+r"(r[6]),
                 "+r"(r[7]), "+r"(r[8]), "+r"(r[9]), "+r"(r[10]), "+r"(r[11]), "+r"(r[12]),
                 "+r"(r[13]), "+r"(r[14]), "+r"(r[15])
               :
               : "memory");
}
__device__ __forceinline__ void tmem_st_x16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]),
      "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]),
      "r"(r[15])
      : "memory");
}

// Reduces 16 values over the warp's lanes: lane l ends with the result of value
// ((l >> 4) & 1) * 8 + ((l >> 3) & 1) * 4 + ((l >> 2) & 1) * 2 + ((l >> 1) & 1).
template <bool MAX>
__device__ __forceinline__ float reduce16(float (&v)[16], int lane) {
#pragma unroll
  for (int w = 8, o = 16; w >= 1; w >>= 1, o >>= 1) {
    const bool hi = (lane & o) != 0;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      if (i < w) {
        const float mine = hi ? v[i + w] : v[i];
        const float send = hi ? v[i] : v[i + w];
        const float got = __shfl_xor_sync(0xffffffffu, send, o);
        v[i] = MAX ? fmaxf(mine, got) : mine + got;
      }
    }
  }
  const float other = __shfl_xor_sync(0xffffffffu, v[0], 1);
  return MAX ? fmaxf(v[0], other) : v[0] + other;
}
__device__ __forceinline__ int reduce16_index(int lane) {
  return ((lane >> 4) & 1) * 8 + ((lane >> 3) & 1) * 4 + ((lane >> 2) & 1) * 2 + ((lane >> 1) & 1);
}

template <int NR>
__global__ void __launch_bounds__(kLatThreads, 1)
latent_attention_kernel(const __grid_constant__ CUtensorMap tmap_q,
                        const __grid_constant__ CUtensorMap tmap_c, const LatentArgs p,
                        const LatentExt x) {
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~static_cast<uintptr_t>(1023));
  __shared__ __align__(16) float wred[NR * 4];   // per column: the four warps' values
  __shared__ __align__(16) float m_s[NR], neg_s[NR], alpha_s[NR], inv_s[NR];
  __shared__ int2 see_s[NR];                     // first and last visible key of each row
  __shared__ int rescale_s[2];
  __shared__ uint64_t bars[1 + 2 * kLatMaxSlots + 12];
  __shared__ uint32_t tmem_slot;
  __shared__ volatile int abort_s;

  const int NC = p.pieces;
  const int NX = p.x_bufs > 0 ? 1 : 0;
  const uint32_t sQ = smem_u32(smem);
  const uint32_t sC = sQ + (uint32_t)(NC + NX) * NR * 128u;
  const uint32_t sX = sC + (uint32_t)p.slots * kPieceBytes;
  const uint32_t sP = sX + (uint32_t)p.x_bufs * kPieceBytes;
  uint8_t* pC = smem + (size_t)(NC + NX) * NR * 128;
  uint8_t* pP = pC + (size_t)(p.slots + p.x_bufs) * kPieceBytes;
  const uint32_t bb = smem_u32(bars);
  const uint32_t q_full = bb;
  auto c_full = [&](int s) { return bb + 8u * (1 + s); };
  auto c_empty = [&](int s) { return bb + 8u * (1 + kLatMaxSlots + s); };
  auto s_full = [&](int s) { return bb + 8u * (1 + 2 * kLatMaxSlots + s); };
  auto s_empty = [&](int s) { return bb + 8u * (3 + 2 * kLatMaxSlots + s); };
  auto p_full = [&](int s) { return bb + 8u * (5 + 2 * kLatMaxSlots + s); };
  auto o_full = [&](int s) { return bb + 8u * (7 + 2 * kLatMaxSlots + s); };
  auto x_full = [&](int s) { return bb + 8u * (9 + 2 * kLatMaxSlots + s); };
  auto x_empty = [&](int s) { return bb + 8u * (11 + 2 * kLatMaxSlots + s); };
  const int warp = threadIdx.x >> 5;
  const int lane = threadIdx.x & 31;

  pdl_trigger();
  const int* wk = p.work + (long long)blockIdx.x * 8;
  const int n_rows = wk[2];
  if (n_rows <= 0) {   // padding entry of a fixed-size work list
    pdl_wait();
    return;
  }
  const int seq = wk[0], row0 = wk[1], pos0 = wk[3], kv_start = wk[4], piece = wk[6], n_pieces = wk[7];
  const int kv_end = min(wk[5], pos0 + (row0 + n_rows - 1) / p.H + 1);
  const int n_tiles = kv_end > kv_start ? (kv_end - kv_start + kLatKeys - 1) / kLatKeys : 0;
  const int bs = p.block_size;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < p.slots; ++s) {
      mbar_init(c_full(s), 1);
      mbar_init(c_empty(s), 1);
    }
    for (int s = 0; s < 2; ++s) {
      mbar_init(s_full(s), 1);
      mbar_init(s_empty(s), 4);
      mbar_init(p_full(s), 4);
      mbar_init(o_full(s), 1);
      mbar_init(x_full(s), 1);
      mbar_init(x_empty(s), 1);
      rescale_s[s] = 0;
    }
    abort_s = 0;
    fence_barrier_init();
    prefetch_tensormap(&tmap_q);
    prefetch_tensormap(&tmap_c);
  }
  for (int i = threadIdx.x; i < NR; i += kLatThreads) {
    m_s[i] = -INFINITY;
    const int pos = pos0 + (row0 + i) / p.H;
    see_s[i] = make_int2(first_visible(p.mask_kind, p.mask_size, pos), min(pos, kv_end - 1));
  }
  if (warp == 5) {
    tmem_alloc(smem_u32(&tmem_slot), p.tmem_cols);
    tmem_relinquish();
  }
  // Keys past the end of the last tile are never loaded and meet P = 0: what lies there must be
  // finite. A slot that an earlier tile has filled is; the others are cleared.
  if (n_tiles > 0) {
    const int nkeys = kv_end - kv_start - (n_tiles - 1) * kLatKeys;
    const int r_first = (nkeys + bs - 1) / bs * bs;
    if (r_first < kLatKeys) {
      const int vecs = (kLatKeys - r_first) * 8;
      for (int c = 0; c < NC; ++c) {
        const int idx = (n_tiles - 1) * NC + c;
        if (idx >= p.slots) break;
        uint4* z = reinterpret_cast<uint4*>(pC + (size_t)idx * kPieceBytes + (size_t)r_first * 128);
        for (int i = threadIdx.x; i < vecs; i += kLatThreads) z[i] = make_uint4(0, 0, 0, 0);
      }
    }
  }
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_wait();
  const uint32_t tS = tmem_slot;                 // S buffers at columns 0, NR
  const uint32_t tO = tmem_slot + 2 * NR;        // R / 128 blocks of NR columns

  if (warp == 4) {
    // ------------------------------ TMA producer ------------------------------
    if (n_tiles > 0) {
      if (lane == 0) {
        mbar_arrive_expect_tx(q_full, (uint32_t)(NC + NX) * NR * 128u);
        for (int c = 0; c < NC + NX; ++c)
          tma_load_2d(sQ + (uint32_t)c * NR * 128u, &tmap_q, q_full, c * 64, row0);
      }
      // A lane per (piece, cache block) box of the tile: it waits for the piece's slot itself and
      // issues its copy, so a tile's copies leave as fast as their slots come free.
      const int* bt = p.block_tables + (long long)seq * p.max_blocks;
      const int nb_max = kLatKeys / bs;
      const int boxes = (NC + NX) * nb_max;
      bool ok = true;
      int bid_next = 0;
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int key0 = kv_start + j * kLatKeys;
        const int nblk = (min(kLatKeys, kv_end - key0) + bs - 1) / bs;
        for (int i0 = 0; i0 < boxes && ok; i0 += 32) {
          const int i = i0 + lane;
          const int c = i / nb_max, blk = i % nb_max;
          const bool mine = i < boxes && blk < nblk;
          const int bid = (j == 0 || boxes > 32) ? (mine ? bt[key0 / bs + blk] : 0) : bid_next;
          // a piece of the latent has a slot of the ring, the key-only piece one of its buffers
          const bool kx = c >= NC;
          const int idx = kx ? j : j * NC + c;
          const int bufs = kx ? p.x_bufs : p.slots;
          const int slot = idx % bufs;
          const uint32_t ph = (uint32_t)(idx / bufs) & 1u;
          const uint32_t full = kx ? x_full(slot) : c_full(slot);
          const uint32_t empty = kx ? x_empty(slot) : c_empty(slot);
          const uint32_t dst = (kx ? sX : sC) + (uint32_t)slot * kPieceBytes;
          if (boxes <= 32 && j + 1 < n_tiles) {   // the next tile's table entry is on its way
            const int next0 = key0 + kLatKeys;
            const int nn = (min(kLatKeys, kv_end - next0) + bs - 1) / bs;
            bid_next = (i < boxes && blk < nn) ? bt[next0 / bs + blk] : 0;
          }
          bool done = !mine;
          unsigned long long t0 = 0;
          uint32_t spins = 0;
          while (!done) {
            if (mbar_try_wait(empty, ph ^ 1u)) {
              if (blk == 0) mbar_arrive_expect_tx(full, (uint32_t)(nblk * bs) * 128u);
              tma_load_2d(dst + (uint32_t)(blk * bs) * 128u, &tmap_c, full, c * 64, bid * bs);
              done = true;
            } else if ((++spins & 63u) == 0u) {
              if (abort_s) {
                ok = false;
                break;
              }
              if (t0 == 0) t0 = globaltimer_ns();
              else if (globaltimer_ns() - t0 > kWaitLimitNs) {
                abort_s = 1;
                report_error(p.status, kErrBarrierTimeout, 1500 + slot, j);
                ok = false;
                break;
              }
            }
          }
          ok = __all_sync(0xffffffffu, ok);
        }
      }
      if (!ok) {   // unwinding: give copies that were already issued a short time to land
        const unsigned long long t0 = globaltimer_ns();
        while (globaltimer_ns() - t0 < 5000000ull) {
        }
      }
    }
  } else if (warp == 5) {
    // ------------------------------- MMA issuer -------------------------------
    // The whole warp walks the loop with uniform values and one elected lane issues: descriptors
    // then live in uniform registers, and an instruction goes out as fast as the tensor core
    // takes it.
    if (n_tiles > 0) {
      const uint32_t idesc_s = make_idesc(128, NR, 1, 1, 0, 0);
      const uint32_t idesc_o = make_idesc(128, NR, 1, 1, 1, 0);
      const uint32_t tm = __shfl_sync(0xffffffffu, tmem_slot, 0);
      const uint32_t tS_u = tm, tO_u = tm + 2 * NR;
      const uint64_t c_k = make_desc_kmajor_sw128(sC);                   // + 1024 per slot
      const uint64_t c_mn = make_desc_mnmajor_sw128(sC, kPieceBytes);
      const uint64_t q_k = make_desc_kmajor_sw128(sQ);                   // + NR * 8 per piece
      const uint64_t p_k = make_desc_kmajor_sw128(sP);
      const uint64_t x_k = make_desc_kmajor_sw128(sX);
      int s_slot = 0, o_slot = 0;
      uint32_t s_ph = 0;
      auto wait = [&](uint32_t bar, uint32_t parity, int code, int j) -> bool {
        return __all_sync(0xffffffffu, mbar_wait(bar, parity, &abort_s, p.status, code, j));
      };
      bool ok = wait(q_full, 0, 1600, 0);
      auto issue_s = [&](int j) -> bool {
        const int st = j & 1;
        if (!wait(s_empty(st), ((uint32_t)(j >> 1) & 1u) ^ 1u, 1620 + st, j)) return false;
        for (int c = 0; c < NC; ++c) {
          if (!wait(c_full(s_slot), s_ph, 1610, j)) return false;
          tc_fence_after();
          const uint64_t cd = c_k + (uint64_t)(s_slot * (int)(kPieceBytes / 16));
          const uint64_t qd = q_k + (uint64_t)(c * (NR * 8));
          if (elect_one()) {
#pragma unroll
            for (int k = 0; k < 4; ++k)
              umma_f16_ss(tS_u + (uint32_t)st * NR, cd + (uint64_t)(2 * k), qd + (uint64_t)(2 * k),
                          idesc_s, (c > 0 || k > 0) ? 1u : 0u);
            if (c == NC - 1 && NX == 0) tc_commit(s_full(st));
          }
          __syncwarp();
          if (++s_slot == p.slots) {
            s_slot = 0;
            s_ph ^= 1u;
          }
        }
        if (NX) {
          const int xb = p.x_bufs == 2 ? (j & 1) : 0;
          const uint32_t xph = (uint32_t)(p.x_bufs == 2 ? (j >> 1) : j) & 1u;
          if (!wait(x_full(xb), xph, 1630 + xb, j)) return false;
          tc_fence_after();
          const uint64_t xd = x_k + (uint64_t)(xb * (int)(kPieceBytes / 16));
          const uint64_t qd = q_k + (uint64_t)(NC * (NR * 8));
          if (elect_one()) {
#pragma unroll
            for (int k = 0; k < 4; ++k)
              umma_f16_ss(tS_u + (uint32_t)st * NR, xd + (uint64_t)(2 * k), qd + (uint64_t)(2 * k),
                          idesc_s, 1u);
            tc_commit(x_empty(xb));
            tc_commit(s_full(st));
          }
          __syncwarp();
        }
        return true;
      };
      auto issue_o = [&](int j) -> bool {
        const int pb = p.p_bufs == 2 ? (j & 1) : 0;
        const uint32_t pph = (uint32_t)(p.p_bufs == 2 ? (j >> 1) : j) & 1u;
        if (!wait(p_full(pb), pph, 1640 + pb, j)) return false;
        tc_fence_after();
        const uint64_t pd = p_k + (uint64_t)(pb * (NR * 16));
        for (int rc = 0; rc < NC / 2; ++rc) {
          // two neighbouring pieces (128 latent columns); a pair never wraps: slots is even
          const uint64_t cd = c_mn + (uint64_t)(o_slot * (int)(kPieceBytes / 16));
          if (elect_one()) {
#pragma unroll
            for (int k = 0; k < kLatKeys / 16; ++k)
              umma_f16_ss(tO_u + (uint32_t)(rc * NR), cd + (uint64_t)(128 * k),
                          pd + (uint64_t)((k / 4) * (NR * 8) + 2 * (k % 4)), idesc_o,
                          (j > 0 || k > 0) ? 1u : 0u);
            tc_commit(c_empty(o_slot));
            tc_commit(c_empty(o_slot + 1));
            if (rc == NC / 2 - 1) tc_commit(o_full(j & 1));
          }
          __syncwarp();
          o_slot += 2;
          if (o_slot == p.slots) o_slot = 0;
        }
        return true;
      };
      if (ok) ok = issue_s(0);
      for (int j = 0; j < n_tiles && ok; ++j) {
        if (p.overlap && j + 1 < n_tiles) ok = issue_s(j + 1);
        if (ok) ok = issue_o(j);
        if (ok && !p.overlap && j + 1 < n_tiles) ok = issue_s(j + 1);
      }
    }
  } else {
    // ------------------------------ softmax warps ------------------------------
    // A wait that runs out leaves `ok` false; the warp then only keeps the barriers going (every
    // loop has the same trip count in all four warps), so that nobody waits for it.
    const int tid = threadIdx.x;     // key of the tile, TMEM lane
    const uint32_t lane_off = (uint32_t)(warp * 32) << 16;
    const float sc = p.scale_log2;
    const int my_col = reduce16_index(lane);
    float l[NR];
#pragma unroll
    for (int i = 0; i < NR; ++i) l[i] = 0.f;
    bool ok = true;
    const int min_lim = pos0 + row0 / p.H;
    const int max_low =
        first_visible(p.mask_kind, p.mask_size, pos0 + (row0 + n_rows - 1) / p.H);
    for (int j = 0; j < n_tiles; ++j) {
      const int st = j & 1;
      const int key0 = kv_start + j * kLatKeys;
      const int key = key0 + tid;
      const bool need_mask = key0 + kLatKeys - 1 > min(min_lim, kv_end - 1) || key0 < max_low;
      ok = __all_sync(0xffffffffu, ok && mbar_wait(s_full(st), (uint32_t)(j >> 1) & 1u, &abort_s,
                                                   p.status, 1700 + st, j));
      tc_fence_after();
      const uint32_t ts = tS + (uint32_t)st * NR + lane_off;
      uint32_t sr[NR / 16][16];   // this key's scores
      if (ok) {
#pragma unroll
        for (int g = 0; g < NR / 16; ++g) tmem_ld_x16(ts + 16u * g, sr[g]);
#pragma unroll
        for (int g = 0; g < NR / 16; ++g) tmem_ld_wait_dep16(sr[g]);
        if (need_mask) {
#pragma unroll
          for (int i = 0; i < NR; ++i) {
            const int2 seen = see_s[i];
            if (key < seen.x || key > seen.y) sr[i / 16][i % 16] = 0xff800000u;   // -inf
          }
        }
#pragma unroll
        for (int g = 0; g < NR / 16; ++g) {
          float v[16];
#pragma unroll
          for (int i = 0; i < 16; ++i) v[i] = __uint_as_float(sr[g][i]);
          const float mx = reduce16<true>(v, lane);
          if ((lane & 1) == 0) wred[(16 * g + my_col) * 4 + warp] = mx;
        }
      }
      bar_softmax();
      if (tid < NR) {
        const float4 q = *reinterpret_cast<const float4*>(&wred[tid * 4]);
        const float m_old = m_s[tid];
        // Any reference point near the maximum serves: it moves only when the maximum has grown by
        // more than 2^8, so that O is rarely rescaled (weights stay below 2^8 in fp32 and bf16)
        const float mx = fmaxf(fmaxf(q.x, q.y), fmaxf(q.z, q.w));
        const float m_new = (m_old == -INFINITY || (mx - m_old) * sc > 8.f) ? fmaxf(m_old, mx) : m_old;
        const float m_safe = m_new == -INFINITY ? 0.f : m_new;
        // a row that has seen no key yet holds O = 0 and l = 0: nothing to rescale
        const float alpha = m_old == -INFINITY ? 1.f : ex2_approx((m_old - m_safe) * sc);
        m_s[tid] = m_new;
        neg_s[tid] = -m_safe * sc;
        alpha_s[tid] = alpha;
        if (alpha != 1.f) rescale_s[st] = 1;
      }
      if (tid == 127) rescale_s[st ^ 1] = 0;
      bar_softmax();
      const bool rescale = j > 0 && *reinterpret_cast<volatile int*>(&rescale_s[st]) != 0;
      // A rescale must not race with O(j-1) accumulating, and P(j) overwrites the buffer that
      // O(j - p_bufs) reads
      const int jw = (rescale || p.p_bufs == 1) ? j - 1 : j - 2;
      if (jw >= 0)
        ok = __all_sync(0xffffffffu, ok && mbar_wait(o_full(jw & 1), (uint32_t)(jw >> 1) & 1u,
                                                     &abort_s, p.status, 1710, j));
      if (rescale && ok) {
        tc_fence_after();
#pragma unroll
        for (int i = 0; i < NR; i += 4) {
          const float4 a = *reinterpret_cast<const float4*>(&alpha_s[i]);
          l[i] *= a.x; l[i + 1] *= a.y; l[i + 2] *= a.z; l[i + 3] *= a.w;
        }
        for (int rc = 0; rc < NC / 2; ++rc) {
#pragma unroll
          for (int g = 0; g < NR / 16; ++g) {
            uint32_t r[16];
            const uint32_t to = tO + (uint32_t)(rc * NR + 16 * g) + lane_off;
            tmem_ld_x16(to, r);
            tmem_ld_wait_dep16(r);
#pragma unroll
            for (int i = 0; i < 16; ++i)
              r[i] = __float_as_uint(__uint_as_float(r[i]) * alpha_s[16 * g + i]);
            tmem_st_x16(to, r);
          }
        }
        tmem_st_wait();
      }
      if (ok) {
        const int pb = p.p_bufs == 2 ? st : 0;
        uint8_t* prow = pP + (size_t)pb * NR * 256 + (size_t)(tid >> 6) * NR * 128 + (tid & 7) * 2;
        const int chunk = (tid & 63) >> 3;
#pragma unroll
        for (int g = 0; g < NR / 16; ++g) {
          float e[16];
#pragma unroll
          for (int i = 0; i < 16; i += 4) {
            const float4 ng = *reinterpret_cast<const float4*>(&neg_s[16 * g + i]);
            e[i] = ex2_approx(fmaf(__uint_as_float(sr[g][i]), sc, ng.x));
            e[i + 1] = ex2_approx(fmaf(__uint_as_float(sr[g][i + 1]), sc, ng.y));
            e[i + 2] = ex2_approx(fmaf(__uint_as_float(sr[g][i + 2]), sc, ng.z));
            e[i + 3] = ex2_approx(fmaf(__uint_as_float(sr[g][i + 3]), sc, ng.w));
          }
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            const int n = 16 * g + i;
            l[n] += e[i];
            *reinterpret_cast<__nv_bfloat16*>(prow + n * 128 + ((chunk ^ (n & 7)) << 4)) =
                __float2bfloat16(e[i]);
          }
        }
      }
      tc_fence_before();
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) {
        mbar_arrive(s_empty(st));
        mbar_arrive(p_full(p.p_bufs == 2 ? st : 0));
      }
    }
    // row sums over the keys, normalisation factors, log-sum-exp
#pragma unroll
    for (int g = 0; g < NR / 16; ++g) {
      float v[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) v[i] = l[16 * g + i];
      const float s = reduce16<false>(v, lane);
      if ((lane & 1) == 0) wred[(16 * g + my_col) * 4 + warp] = s;
    }
    bar_softmax();
    if (tid < NR) {
      const float4 q = *reinterpret_cast<const float4*>(&wred[tid * 4]);
      float sum = (q.x + q.y) + (q.z + q.w);
      if (n_pieces > 1 && tid < n_rows)
        p.lse_part[(long long)piece * p.rows_total + row0 + tid] =
            sum > 0.f ? m_s[tid] * p.scale + logf(sum) : -INFINITY;
      float factor = 1.f;
      if (n_pieces <= 1 && tid < n_rows && sum > 0.f) {   // (else the merge does it)
        const int tok = (row0 + tid) / p.H, head = row0 + tid - tok * p.H;
        if (x.sink != nullptr) sum += ex2_approx(fmaf(x.sink[head], 1.4426950408889634f, neg_s[tid]));
        if (x.gate != nullptr)
          factor = __fdividef(1.f, 1.f + __expf(-__bfloat162float(x.gate[tok * x.ldg + head])));
      }
      inv_s[tid] = sum > 0.f ? factor / sum : 0.f;
    }
    bar_softmax();
    if (n_tiles > 0) {
      const int jl = n_tiles - 1;
      ok = __all_sync(0xffffffffu, ok && mbar_wait(o_full(jl & 1), (uint32_t)(jl >> 1) & 1u, &abort_s,
                                                   p.status, 1720, jl));
      tc_fence_after();
    }
    const int R = NC * 64;
    if (ok) {
      for (int rc = 0; rc < NC / 2; ++rc) {
        const int col = rc * 128 + tid;
#pragma unroll
        for (int g = 0; g < NR / 16; ++g) {
          uint32_t r[16];
          if (n_tiles > 0) {
            tmem_ld_x16(tO + (uint32_t)(rc * NR + 16 * g) + lane_off, r);
            tmem_ld_wait_dep16(r);
          } else {
#pragma unroll
            for (int i = 0; i < 16; ++i) r[i] = 0u;
          }
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            const int n = 16 * g + i;
            if (n < n_rows) {
              const float v = __uint_as_float(r[i]) * inv_s[n];
              if (n_pieces > 1)
                p.o_part[((long long)piece * p.rows_total + row0 + n) * R + col] = v;
              else
                p.out[(long long)(row0 + n) * R + col] = __float2bfloat16(v);
            }
          }
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 5) {
    tc_fence_after();
    tmem_dealloc(tmem_slot, p.tmem_cols);
  }
}

template <int NR>
static int launch_latent(const CUtensorMap& tq, const CUtensorMap& tc, LatentArgs a, const LatentExt& x,
                         int num_work, cudaStream_t stream) {
  const int NC = a.pieces;
  const size_t limit = 227 * 1024 - 4096;   // static shared memory and alignment aside
  const int NX = a.x_bufs;   // (wanted: 0 or 1)
  const size_t q_bytes = (size_t)(NC + NX) * NR * 128;
  const size_t room = limit - q_bytes;
  a.p_bufs = 2;
  auto fit = [&](int pb, int xb) {
    const size_t other = (size_t)pb * NR * 256 + (size_t)xb * kPieceBytes;
    if (other >= room) return 0;
    int s = (int)((room - other) / kPieceBytes) & ~1;
    return s > kLatMaxSlots ? kLatMaxSlots : s;
  };
  a.slots = fit(2, NX);
  if (a.slots < NC + 2 && fit(1, NX) > a.slots) {
    a.p_bufs = 1;
    a.slots = fit(1, NX);
  }
  if (a.slots < NC) return -6;
  // a second buffer of the key-only piece where it costs no slot that overlapping needs
  if (NX && (fit(a.p_bufs, 2) >= a.slots || fit(a.p_bufs, 2) >= 2 * NC)) {
    a.x_bufs = 2;
    a.slots = fit(a.p_bufs, 2);
  }
  a.overlap = a.slots >= 2 * NC;
  a.tmem_cols = 32;
  while (a.tmem_cols < (uint32_t)((2 + NC / 2) * NR)) a.tmem_cols <<= 1;
  const size_t smem = q_bytes + (size_t)(a.slots + a.x_bufs) * kPieceBytes +
                      (size_t)a.p_bufs * NR * 256 + 1024;
  static bool attr_set[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return -3;
  if (!attr_set[dev]) {
    if (cudaFuncSetAttribute(latent_attention_kernel<NR>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                             224 * 1024) != cudaSuccess)
      return -3;
    attr_set[dev] = true;
  }
  return launch_pdl(latent_attention_kernel<NR>, dim3((unsigned)num_work), dim3(kLatThreads), smem,
                    stream, tq, tc, a, x) == cudaSuccess
             ? 0
             : -5;
}

}  // namespace ab200

using namespace ab200;

extern "C" {

// q bf16 [T * H, R + key_extra], out [T * H, R], both contiguous; cache [num_blocks, block_size,
// R + key_extra]; R a multiple of 128 up to 512, key_extra 0 or 64 (columns of the key only);
// tile_rows 16, 32, 48 or 64, the rows per work item (at most 48 with R = 512 and key_extra). sink
// fp32 [H] and gate bf16 [T, ldg] (column h: head h's, of which the sigmoid is taken) may be null.
int ab200_latent_attention(const void* q, long long q_rows, const void* cache, int num_blocks,
                           int block_size, const void* block_tables, int max_blocks,
                           const void* work, int num_work, const void* tok_splits, int max_splits,
                           long long T, int H, int R, int key_extra, int mask_kind, int mask_size,
                           int tile_rows, float scale, const void* sink, const void* gate,
                           long long ldg, void* out, void* o_part, void* lse_part, int* status,
                           cudaStream_t stream) {
  if (num_work <= 0 || T <= 0) return 0;
  if (R % 128 || R < 128 || R > 512 || H <= 0 || q_rows != T * H) return -2;
  if (key_extra != 0 && key_extra != 64) return -2;
  if (mask_kind < kMaskCausal || mask_kind > kMaskChunk || (mask_kind != kMaskCausal && mask_size < 1))
    return -2;
  if (block_size < 8 || block_size > kLatKeys || kLatKeys % block_size) return -2;
  if (T * H > 0x7fffffffll || (long long)num_blocks * block_size > 0x7fffffffll) return -6;
  if (max_splits > 1 && (o_part == nullptr || lse_part == nullptr || tok_splits == nullptr)) return -2;
  const int W = R + key_extra;
  CUtensorMap tq, tc;
  if (make_tmap_2d(&tq, q, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, (uint64_t)q_rows, (uint64_t)W,
                   (uint64_t)W * 2, (uint32_t)tile_rows, 64) != 0)
    return -4;
  if (make_tmap_2d(&tc, cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, (uint64_t)num_blocks * block_size,
                   (uint64_t)W, (uint64_t)W * 2, (uint32_t)block_size, 64) != 0)
    return -4;
  const LatentExt x = {reinterpret_cast<const float*>(sink), reinterpret_cast<const __nv_bfloat16*>(gate), ldg};
  LatentArgs a;
  memset(&a, 0, sizeof(a));
  a.work = reinterpret_cast<const int*>(work);
  a.block_tables = reinterpret_cast<const int*>(block_tables);
  a.max_blocks = max_blocks;
  a.block_size = block_size;
  a.H = H;
  a.pieces = R / 64;
  a.x_bufs = key_extra / 64;
  a.mask_kind = mask_kind;
  a.mask_size = mask_size;
  a.scale = scale;
  a.scale_log2 = scale * 1.4426950408889634f;
  a.out = reinterpret_cast<__nv_bfloat16*>(out);
  a.o_part = reinterpret_cast<float*>(o_part);
  a.lse_part = reinterpret_cast<float*>(lse_part);
  a.rows_total = q_rows;
  a.status = status;
  int rc;
  switch (tile_rows) {
    case 16: rc = launch_latent<16>(tq, tc, a, x, num_work, stream); break;
    case 32: rc = launch_latent<32>(tq, tc, a, x, num_work, stream); break;
    case 48: rc = launch_latent<48>(tq, tc, a, x, num_work, stream); break;
    case 64: rc = launch_latent<64>(tq, tc, a, x, num_work, stream); break;
    default: return -2;
  }
  if (rc != 0 || max_splits <= 1) return rc;
  return ab200_attention_merge(o_part, lse_part, tok_splits, T, H, R, sink, gate, ldg, out,
                               (long long)H * R, stream);
}

}  // extern "C"
