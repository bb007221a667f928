// Grouped bf16 matrix products for sm_100a: out[rows of g] = x[rows of g] * w[g]^T, one launch for
// all groups. It serves
//   * the experts of a mixture (rows sorted by expert; the (expert, first row, rows) tiles are
//     made on the device by the router, so nothing waits for the host and a captured decode
//     step replays), gate and up together with the activation in the epilogue, or down;
//   * per-head maps (head h's columns of every token times head h's matrix);
//   * a dense gated feed-forward (one group) with the activation in the epilogue.
//
// The machine is the linear layer's (gemm_bf16.cu): a persistent warp-specialised kernel, one
// thread feeding a ring of 128B-swizzled stages by TMA, one thread issuing tcgen05.mma
// 128 x bn x 16 into double-buffered TMEM accumulators, four epilogue warps. Weight tiles (up to
// 256 features) sit on the N side, so a group of a few tokens streams its weights at full width;
// such a group fetches 32 activation rows per stage instead of 128.
//
// With an activation the rows of w alternate in blocks of 16 gate and 16 up rows: 32 accumulator
// columns hold both factors of 16 outputs and a thread multiplies them in registers.

#include <string.h>

#include "api.h"
#include "common/elem.cuh"
#include "common/pdl.cuh"
#include "common/tensormap.h"

namespace ab200 {

constexpr int kGgThreads = 192;
constexpr int kGgBlockK = 64;
constexpr int kGgMaxStages = 8;
constexpr uint32_t kGgABytes = 128 * kGgBlockK * 2;

struct GroupedArgs {
  int N, K, bn, stages, kblocks, n_tiles;
  int M, m_tiles, groups;   // without a tile list: rows and row tiles per group
  int x_by_group;           // the activations' map has a group dimension
  int m_fastest;            // work order: row tiles of one weight tile next to each other
  int act;
  GateParams gate;
  uint32_t tmem_cols;
  const int4* tiles;
  const int* num_tiles;
  __nv_bfloat16* out;
  long long ldo, out_gstride;
  int* status;
};

struct GgWork {
  int group, row0, nrows, nt;
};

__device__ __forceinline__ GgWork gg_work(const GroupedArgs& p, int w, int m_total) {
  int mt, nt;
  if (p.m_fastest) {
    mt = w % m_total;
    nt = w / m_total;
  } else {
    nt = w % p.n_tiles;
    mt = w / p.n_tiles;
  }
  GgWork r;
  r.nt = nt;
  if (p.tiles != nullptr) {
    const int4 t = p.tiles[mt];
    r.group = t.x;
    r.row0 = t.y;
    r.nrows = t.z;
  } else {
    r.group = mt / p.m_tiles;
    r.row0 = (mt % p.m_tiles) * 128;
    r.nrows = min(128, p.M - r.row0);
  }
  return r;
}

// The activations' rounding to bf16 is far coarser than the fast exponential and division.
__device__ __forceinline__ float gg_gated(int act, const GateParams& p, float g, float u) {
  float t;   // g * sigmoid(t)
  if (act == kActClampedSwish) {
    g = fminf(g, p.limit);
    u = fminf(fmaxf(u, -p.limit), p.limit) + 1.f;
    t = p.alpha * g;
  } else {   // gelu_tanh(z) = z * sigmoid(2 sqrt(2/pi) (...))
    t = act == kActSilu ? g : 1.5957691216057308f * (g + 0.044715f * g * g * g);
  }
  return __fdividef(g, 1.f + __expf(-t)) * u;
}

__global__ void __launch_bounds__(kGgThreads, 1)
grouped_gemm_kernel(const __grid_constant__ CUtensorMap tmap_x,
                    const __grid_constant__ CUtensorMap tmap_x32,
                    const __grid_constant__ CUtensorMap tmap_w, const GroupedArgs p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~static_cast<uintptr_t>(1023));
  const uint32_t b_bytes = (uint32_t)p.bn * kGgBlockK * 2;
  const uint32_t stage_bytes = kGgABytes + b_bytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + (size_t)p.stages * stage_bytes);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2 * kGgMaxStages + 4);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const uint32_t smem_base = smem_u32(smem);
  const uint32_t bars_base = smem_u32(bars);
  auto full_bar = [&](int s) { return bars_base + 8u * s; };
  auto empty_bar = [&](int s) { return bars_base + 8u * (kGgMaxStages + s); };
  auto tfull_bar = [&](int a) { return bars_base + 8u * (2 * kGgMaxStages + a); };
  auto tempty_bar = [&](int a) { return bars_base + 8u * (2 * kGgMaxStages + 2 + a); };
  const int warp = threadIdx.x >> 5;
  const int lane = threadIdx.x & 31;

  pdl_trigger();
  if (threadIdx.x == 0) {
    for (int s = 0; s < p.stages; ++s) {
      mbar_init(full_bar(s), 1);
      mbar_init(empty_bar(s), 1);
    }
    for (int a = 0; a < 2; ++a) {
      mbar_init(tfull_bar(a), 1);
      mbar_init(tempty_bar(a), 4);
    }
    *abort_flag = 0;
    fence_barrier_init();
    prefetch_tensormap(&tmap_x);
    prefetch_tensormap(&tmap_x32);
    prefetch_tensormap(&tmap_w);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), p.tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t acc_stride = p.tmem_cols / 2;
  pdl_wait();   // the tile list and the activations come from earlier kernels
  const int m_total = p.tiles != nullptr ? *p.num_tiles : p.groups * p.m_tiles;
  const int total_work = m_total * p.n_tiles;

  if (warp == 0) {
    // ------------------------------ TMA producer ------------------------------
    if (lane == 0) {
      int stage = 0;
      uint32_t phase = 0;
      long long issued = 0;
      bool ok = true;
      for (int w = blockIdx.x; w < total_work && ok; w += gridDim.x) {
        const GgWork t = gg_work(p, w, m_total);
        const bool few = t.nrows <= 32;
        const uint32_t bytes = b_bytes + (few ? 32u * kGgBlockK * 2u : kGgABytes);
        const int xg = p.x_by_group ? t.group : 0;
        for (int kb = 0; kb < p.kblocks; ++kb) {
          if (!mbar_wait(empty_bar(stage), phase ^ 1u, abort_flag, p.status, 1100 + stage, kb)) {
            ok = false;
            break;
          }
          mbar_arrive_expect_tx(full_bar(stage), bytes);
          const uint32_t dst = smem_base + (uint32_t)stage * stage_bytes;
          tma_load_3d(dst, few ? &tmap_x32 : &tmap_x, full_bar(stage), kb * kGgBlockK, t.row0, xg);
          tma_load_3d(dst + kGgABytes, &tmap_w, full_bar(stage), kb * kGgBlockK, t.nt * p.bn, t.group);
          ++issued;
          if (++stage == p.stages) {
            stage = 0;
            phase ^= 1u;
          }
        }
      }
      if (!ok) {   // unwinding: give copies that were already issued a short time to land
        const int pending = (int)min((long long)p.stages, issued);
        for (int i = 0; i < pending; ++i) {
          if (--stage < 0) {
            stage = p.stages - 1;
            phase ^= 1u;
          }
          mbar_drain(full_bar(stage), phase);
        }
      }
    }
  } else if (warp == 1) {
    // ------------------------------- MMA issuer -------------------------------
    // The warp walks the loop with uniform values and one elected lane issues, which keeps the
    // descriptors in uniform registers: an instruction then costs what the tensor core takes,
    // not what moving its operands there takes.
    const uint32_t idesc = make_idesc(128, (uint32_t)p.bn, 1, 1, 0, 0);
    const uint32_t tm = __shfl_sync(0xffffffffu, tmem_base, 0);
    const uint64_t a0 = make_desc_kmajor_sw128(smem_base);
    const uint64_t stage_step = stage_bytes / 16;
    int stage = 0, acc = 0;
    uint32_t phase = 0, acc_phase = 0;
    bool ok = true;
    for (int w = blockIdx.x; w < total_work && ok; w += gridDim.x) {
      if (!__all_sync(0xffffffffu, mbar_wait(tempty_bar(acc), acc_phase ^ 1u, abort_flag, p.status,
                                             1200 + acc, w)))
        break;
      tc_fence_after();
      const uint32_t d_tmem = tm + (uint32_t)acc * acc_stride;
      for (int kb = 0; kb < p.kblocks; ++kb) {
        if (!__all_sync(0xffffffffu, mbar_wait(full_bar(stage), phase, abort_flag, p.status,
                                               1300 + stage, kb))) {
          ok = false;
          break;
        }
        tc_fence_after();
        const uint64_t a_desc = a0 + (uint64_t)stage * stage_step;
        const uint64_t b_desc = a_desc + (uint64_t)(kGgABytes / 16);
        if (elect_one()) {
#pragma unroll
          for (int k = 0; k < kGgBlockK / 16; ++k)
            umma_f16_ss(d_tmem, a_desc + (uint64_t)(2 * k), b_desc + (uint64_t)(2 * k), idesc,
                        (kb > 0 || k > 0) ? 1u : 0u);
          tc_commit(empty_bar(stage));
          if (kb == p.kblocks - 1) tc_commit(tfull_bar(acc));
        }
        __syncwarp();
        if (++stage == p.stages) {
          stage = 0;
          phase ^= 1u;
        }
      }
      if (!ok) break;
      acc ^= 1;
      if (acc == 0) acc_phase ^= 1u;
    }
  } else {
    // --------------------------------- epilogue --------------------------------
    const int quad = warp & 3;   // TMEM lane quadrant this warp may read
    const int row = quad * 32 + lane;
    int acc = 0;
    uint32_t acc_phase = 0;
    for (int w = blockIdx.x; w < total_work; w += gridDim.x) {
      const GgWork t = gg_work(p, w, m_total);
      const bool row_ok = row < t.nrows;
      const int n0 = t.nt * p.bn;
      if (!__all_sync(0xffffffffu, mbar_wait(tfull_bar(acc), acc_phase, abort_flag, p.status,
                                             1400 + acc, w)))
        break;
      tc_fence_after();
      const uint32_t t_addr = tmem_base + (uint32_t)acc * acc_stride + ((uint32_t)(quad * 32) << 16);
      __nv_bfloat16* dst = p.out + (long long)(t.row0 + row) * p.ldo + (long long)t.group * p.out_gstride;
      if (quad * 32 < t.nrows) {   // a warp whose rows are all beyond the group has nothing to store
        for (int c0 = 0; c0 < p.bn && n0 + c0 < p.N; c0 += 32) {
          uint32_t r[32];
          __syncwarp();
          tmem_ld_x32(t_addr + (uint32_t)c0, r);
          tmem_ld_wait_dep(r);
          if (!row_ok) continue;
          if (p.act != 0) {
            uint32_t o[8];
#pragma unroll
            for (int i = 0; i < 8; ++i)
              o[i] = pack_bf16x2(gg_gated(p.act, p.gate, __uint_as_float(r[2 * i]),
                                          __uint_as_float(r[16 + 2 * i])),
                                 gg_gated(p.act, p.gate, __uint_as_float(r[2 * i + 1]),
                                          __uint_as_float(r[17 + 2 * i])));
            uint4* q = reinterpret_cast<uint4*>(dst + (n0 + c0) / 2);
            q[0] = make_uint4(o[0], o[1], o[2], o[3]);
            q[1] = make_uint4(o[4], o[5], o[6], o[7]);
          } else {
#pragma unroll
            for (int i = 0; i < 4; ++i)
              if (n0 + c0 + 8 * i + 8 <= p.N)
                *reinterpret_cast<uint4*>(dst + n0 + c0 + 8 * i) = make_uint4(
                    pack_bf16x2(__uint_as_float(r[8 * i]), __uint_as_float(r[8 * i + 1])),
                    pack_bf16x2(__uint_as_float(r[8 * i + 2]), __uint_as_float(r[8 * i + 3])),
                    pack_bf16x2(__uint_as_float(r[8 * i + 4]), __uint_as_float(r[8 * i + 5])),
                    pack_bf16x2(__uint_as_float(r[8 * i + 6]), __uint_as_float(r[8 * i + 7])));
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(tempty_bar(acc));
      acc ^= 1;
      if (acc == 0) acc_phase ^= 1u;
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, p.tmem_cols);
  }
}

}  // namespace ab200

using namespace ab200;

extern "C" {

// Strides in elements, multiples of 8; K and N multiples of 8 (N of 32 with an activation).
// x [x_rows, K] with row stride ldx; x_gstride > 0: group g's activations start g * x_gstride
// further. w[g] at w + g * w_gstride, rows ldw apart. With `tiles` (int32 x 4: group, first row,
// rows; `num_tiles` of them, at most max_tiles) x and out hold the rows of all groups one after
// the other; without, every group has M rows. act: 0, 1 (silu), 2 (gelu_tanh) or 3 (clamped swish
// with act_limit and act_alpha): gated product, out has N / 2 columns.
int ab200_grouped_gemm(const void* x, long long ldx, long long x_gstride, long long x_rows,
                       const void* w, long long ldw, long long w_gstride, void* out, long long ldo,
                       long long out_gstride, int M, int N, int K, int groups, const void* tiles,
                       const void* num_tiles, int max_tiles, int act, float act_limit,
                       float act_alpha, int* status, cudaStream_t stream) {
  if (N <= 0 || K <= 0 || groups <= 0 || x_rows <= 0 || (tiles == nullptr ? M : max_tiles) <= 0)
    return 0;
  if ((K % 8) || (N % 8) || (ldx % 8) || (x_gstride % 8) || (ldw % 8) || (w_gstride % 8) ||
      (ldo % 8) || (out_gstride % 8) || (act != 0 && N % 32) || act < 0 || act > 3 ||
      ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w) |
        reinterpret_cast<uintptr_t>(out)) & 15))
    return -2;
  if (tiles != nullptr && (num_tiles == nullptr || x_gstride != 0)) return -2;
  static bool attr_set[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) return -3;
  if (!attr_set[dev]) {
    if (cudaFuncSetAttribute(grouped_gemm_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                             227 * 1024) != cudaSuccess)
      return -3;
    attr_set[dev] = true;
  }
  static int sms = 0;
  if (sms == 0) {
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    if (sms <= 0) sms = 148;
  }
  GroupedArgs a;
  memset(&a, 0, sizeof(a));
  a.N = N;
  a.K = K;
  a.kblocks = (K + kGgBlockK - 1) / kGgBlockK;
  a.M = M;
  a.m_tiles = (M + 127) / 128;
  a.groups = groups;
  a.x_by_group = x_gstride > 0;
  a.act = act;
  a.gate.limit = act_limit;
  a.gate.alpha = act_alpha;
  a.tiles = reinterpret_cast<const int4*>(tiles);
  a.num_tiles = reinterpret_cast<const int*>(num_tiles);
  a.out = reinterpret_cast<__nv_bfloat16*>(out);
  a.ldo = ldo;
  a.out_gstride = out_gstride;
  a.status = status;
  // widest weight tile that still gives every SM one (the number of row tiles of a list is only
  // known on the device; about one per 128 rows, at least one per group in use)
  const long long m_est = tiles ? (max_tiles < groups ? max_tiles : groups) + x_rows / 128
                                : (long long)groups * a.m_tiles;
  a.bn = 256;
  while (a.bn > 64 && m_est * ((N + a.bn - 1) / a.bn) < sms) a.bn /= 2;
  while (a.bn > 32 && a.bn / 2 >= N) a.bn /= 2;
  a.n_tiles = (N + a.bn - 1) / a.bn;
  a.m_fastest = tiles == nullptr && groups == 1;
  a.tmem_cols = 32;
  while (a.tmem_cols < 2u * (uint32_t)a.bn) a.tmem_cols <<= 1;
  const size_t stage = kGgABytes + (size_t)a.bn * kGgBlockK * 2;
  a.stages = (int)((227 * 1024 - 2048) / stage);
  if (a.stages > kGgMaxStages) a.stages = kGgMaxStages;

  CUtensorMap tx, tx32, tw;
  {
    const uint64_t dims[3] = {(uint64_t)K, (uint64_t)x_rows, (uint64_t)(a.x_by_group ? groups : 1)};
    const uint64_t strides[2] = {(uint64_t)ldx * 2, (uint64_t)(a.x_by_group ? x_gstride : ldx) * 2};
    const uint32_t box[3] = {64, 128, 1}, box32[3] = {64, 32, 1};
    if (make_tmap_nd(&tx, x, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, dims, strides, box) != 0) return -4;
    if (make_tmap_nd(&tx32, x, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, dims, strides, box32) != 0)
      return -4;
  }
  {
    const uint64_t dims[3] = {(uint64_t)K, (uint64_t)N, (uint64_t)groups};
    const uint64_t strides[2] = {(uint64_t)ldw * 2, (uint64_t)(w_gstride > 0 ? w_gstride : ldw) * 2};
    const uint32_t box[3] = {64, (uint32_t)a.bn, 1};
    if (make_tmap_nd(&tw, w, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, dims, strides, box) != 0) return -4;
  }
  const long long total = (tiles ? (long long)max_tiles : (long long)groups * a.m_tiles) * a.n_tiles;
  if (total > 0x7fffffff) return -6;
  const int grid = total < sms ? (int)total : sms;
  const size_t smem = (size_t)a.stages * stage + 1024 + 512;
  return launch_pdl(grouped_gemm_kernel, dim3(grid), dim3(kGgThreads), smem, stream, tx, tx32, tw,
                    a) == cudaSuccess
             ? 0
             : -5;
}

}  // extern "C"
