// Scores and values of talking_attention.cu for prompt portions on the fifth-generation tensor cores (head_dim 64 or 128, bfloat16).
//
// Both kernels work on tiles of 128 rows: row m stands for (token m / per, head hk * per + m % per) of one request, per = H / G query
// heads of a kv head. A tile never crosses the border of two blocks of positions, so all of its rows share the scratch buffer's
// column 0. Operands arrive by TMA (128-byte swizzle): queries as a 4-d box, pages of the caches as 4-d boxes named by the block
// table, mixed weights as a 4-d box of the scratch buffer. One thread issues tcgen05.mma into tensor memory.
//
//   scores  S = Q K^T, 128 x 64 a step, two buffers of tensor memory; grid also over runs of keys, since the tiles of one row
//           tile are independent. Eight warps turn a buffer into exponentials, a thread a row: tcgen05.ld, scale, cap, mask on the
//           diagonal, exp2, row sums per tile of 64 keys; through shared memory into the scratch rows, 16 bytes a lane.
//   values  O += W V, 128 x D x 64 a step; O stays in tensor memory. Four warps store it; before, they clear the rows of the first and
//           last value tile that belong to no visible key (what lies there may be no number, and zero times that is none).
//
// Every wait is bounded; a wait that runs out raises *error, and the CTA still frees its tensor memory.
#include <cuda.h>

#include "talking_attention.cuh"

using namespace sb;

#if SB_HEAD_DIM == 64 || SB_HEAD_DIM == 128

typedef __nv_bfloat16 bf16;

namespace talk {
namespace {

constexpr int D = SB_HEAD_DIM;
constexpr int KA = D / 64;            // 128-byte swizzle atoms (64 elements) per operand row
constexpr int BM = 128;               // rows per CTA
constexpr int RUN = 16, RUN_FEW = 8;  // score steps (of 64 keys) a CTA takes; the shorter run where there would be few CTAs (4 to 24
                                      // measured: a CTA's start costs about three steps)
constexpr int NS_S = 2, NS_V = 3;     // stages (two CTAs of either kernel share an SM)
constexpr int BT_CACHE = 512;         // block-table entries kept in shared memory
constexpr unsigned WAIT_LIMIT = 1u << 26;
constexpr int LDE = 36;               // staging row stride (floats): 32 and 16 bytes of padding
constexpr int Q_BYTES = BM * D * 2, K_BYTES = BN * D * 2, W_BYTES = BM * BN * 2, V_BYTES = BN * D * 2;
constexpr int EPI = 8;                // epilogue warps of the scores
constexpr int S_TILES = Q_BYTES + NS_S * K_BYTES, S_STAGE = EPI * 32 * LDE * 4;
constexpr int S_SMEM = S_TILES + S_STAGE + 256 + BT_CACHE * 4;
constexpr int V_TILES = NS_V * (W_BYTES + V_BYTES);
constexpr int V_SMEM = V_TILES + 256 + BT_CACHE * 4;
constexpr uint32_t S_COLS = 2 * BN, V_COLS = D;
static_assert(S_SMEM <= 113 * 1024 && V_SMEM <= 113 * 1024, "two CTAs an SM");

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void mbar_init(uint64_t* bar, unsigned count) {
  asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_u32(bar)), "r"(count));
}
__device__ __forceinline__ void mbar_expect_tx(uint64_t* bar, unsigned bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(smem_u32(bar)), "r"(bytes) : "memory");
}
__device__ __forceinline__ void mbar_arrive(uint64_t* bar) {
  asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ bool mbar_wait(uint64_t* bar, unsigned parity) {
  const uint32_t addr = smem_u32(bar);
  for (unsigned i = 0; i < WAIT_LIMIT; ++i) {
    uint32_t done;
    asm volatile("{\n .reg .pred p;\n mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n selp.u32 %0, 1, 0, p;\n}\n"
                 : "=r"(done) : "r"(addr), "r"(parity) : "memory");
    if (done) return true;
  }
  return false;
}
__device__ __forceinline__ void tma_load_4d(void* dst, const CUtensorMap* map, uint64_t* bar, int c0, int c1, int c2, int c3) {
  asm volatile("cp.async.bulk.tensor.4d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5, %6}], [%2];"
               ::"r"(smem_u32(dst)), "l"(map), "r"(smem_u32(bar)), "r"(c0), "r"(c1), "r"(c2), "r"(c3) : "memory");
}
__device__ __forceinline__ void tc_fence_before() { asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void tc_fence_after() { asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void tc_commit(uint64_t* bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void tc_mma(uint32_t tmem_d, uint64_t desc_a, uint64_t desc_b, uint32_t idesc, uint32_t accumulate) {
  asm volatile("{\n .reg .pred p;\n setp.ne.b32 p, %4, 0;\n tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n}\n"
               ::"r"(tmem_d), "l"(desc_a), "l"(desc_b), "r"(idesc), "r"(accumulate) : "memory");
}
__device__ __forceinline__ void tc_wait_ld() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void tc_load32(uint32_t taddr, float* r) {
  uint32_t* u = reinterpret_cast<uint32_t*>(r);
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, "
      "%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31}, [%32];"
      : "=r"(u[0]), "=r"(u[1]), "=r"(u[2]), "=r"(u[3]), "=r"(u[4]), "=r"(u[5]), "=r"(u[6]), "=r"(u[7]), "=r"(u[8]), "=r"(u[9]),
        "=r"(u[10]), "=r"(u[11]), "=r"(u[12]), "=r"(u[13]), "=r"(u[14]), "=r"(u[15]), "=r"(u[16]), "=r"(u[17]), "=r"(u[18]),
        "=r"(u[19]), "=r"(u[20]), "=r"(u[21]), "=r"(u[22]), "=r"(u[23]), "=r"(u[24]), "=r"(u[25]), "=r"(u[26]), "=r"(u[27]),
        "=r"(u[28]), "=r"(u[29]), "=r"(u[30]), "=r"(u[31])
      : "r"(taddr));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}
// Shared-memory matrix descriptor, 128-byte swizzle, 8-row groups 1024 bytes apart; ``lbo`` is the distance between 64-element
// swizzle atoms along the non-k dimension of an MN-major operand (not used by K-major operands).
__device__ __forceinline__ uint64_t make_desc(uint32_t smem_addr, uint32_t lbo_bytes) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr & 0x3FFFF) >> 4);
  d |= (uint64_t)((lbo_bytes >> 4) & 0x3FFF) << 16;
  d |= (uint64_t)(1024 >> 4) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}
__host__ __device__ constexpr uint32_t make_idesc(int m, int n, bool b_mn_major) {
  return (1u << 4) | (1u << 7) | (1u << 10) | ((b_mn_major ? 1u : 0u) << 16) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(m >> 4) << 24);
}

// tanh by its Taylor series, for |z| <= SERIES_LIMIT (the first term left out is below 2^-24 of z): no special-function unit, whose
// two calls per score (three with the exponential) bound the scores otherwise.
constexpr float SERIES_LIMIT = 0.3f;
__device__ __forceinline__ float tanh_series(float z) {
  const float y = z * z;
  return z * fmaf(y, fmaf(y, fmaf(y, fmaf(y, 62.f / 2835.f, -17.f / 315.f), 2.f / 15.f), -1.f / 3.f), 1.f);
}

// The index-th row tile of a request, counted from its last (those see most keys): tokens [tok0, tok1) of the request, keys
// [lo, hi), scratch column 0 at key kt0.
struct Tile {
  int r, hk, q0, p0, tok0, tok1, lo, hi, kt0;
  const int* bt;
};
__device__ __forceinline__ bool find_tile(const Params& p, int index, Tile& w) {
  w.r = p.wide_rows ? p.wide_rows[blockIdx.z] : (int)blockIdx.z;
  w.hk = blockIdx.x;
  w.q0 = p.cu_q[w.r];
  const int qn = p.cu_q[w.r + 1] - w.q0;
  if (qn <= 0 || (p.deep_on && qn * p.per <= 16)) return false;
  w.p0 = p.kv_len[w.r] - qn;
  const int tpt = BM / p.per;
  // tokens of the request up to the first border of two blocks of positions, then whole blocks
  const int first = p.chunk > 0 ? min(qn, p.chunk - w.p0 % p.chunk) : qn;
  const int n_first = (first + tpt - 1) / tpt, rest = qn - first;
  const int per_block = p.chunk > 0 ? (p.chunk + tpt - 1) / tpt : 1;
  const int n = n_first + (rest > 0 ? rest / p.chunk * per_block + (rest % p.chunk + tpt - 1) / tpt : 0);
  if (index >= n) return false;
  const int i = n - 1 - index;
  if (i < n_first) {
    w.tok0 = i * tpt;
    w.tok1 = min(w.tok0 + tpt, first);
  } else {
    const int k = (i - n_first) / per_block, j = (i - n_first) - k * per_block, block0 = first + k * p.chunk;
    w.tok0 = block0 + j * tpt;
    w.tok1 = min(w.tok0 + tpt, min(block0 + p.chunk, qn));
  }
  w.tok0 = max(w.tok0, p.t_lo - w.q0);
  w.tok1 = min(w.tok1, p.t_hi - w.q0);
  if (w.tok0 >= w.tok1) return false;                         // another launch covers these tokens
  w.lo = first_key(p, w.p0 + w.tok0);
  w.hi = w.p0 + w.tok1;
  w.kt0 = w.lo & ~(BN - 1);
  w.bt = p.block_table + (size_t)w.r * p.bt_width;
  return true;
}

// The table entries of keys [from, to), fetched once by a warp; entry of block blk at bt[blk - first].
__device__ __forceinline__ const int* table_of(const Params& p, const Tile& w, int from, int to, int* bt_s, int lane, int& first) {
  first = from / p.ps;
  const int n = min((to - 1) / p.ps, p.bt_width - 1) - first + 1;
  if (n > BT_CACHE) { first = 0; return w.bt; }
  for (int i = lane; i < n; i += 32) bt_s[i] = w.bt[first + i];
  __syncwarp();
  return bt_s;
}

// One thread: 64 keys from kt on (a multiple of 64) of kv head hk, the pages that hold keys of [lo, hi), into rows 0..63 of atoms
// ``atom`` bytes apart. Returns the number of boxes issued (call with bar null to count only).
__device__ __forceinline__ int load_keys(const Params& p, const CUtensorMap* map, const int* bt, int bt_first, int hk, int kt, int lo, int hi,
                                         unsigned char* dst, int atom, uint64_t* bar) {
  const int step = p.ps < BN ? p.ps : BN;                     // keys of a box
  int n = 0;
  for (int k = kt; k < kt + BN; k += step) {
    if (k >= hi || k + step <= lo) continue;
    const int blk = p.ps_shift >= 0 ? k >> p.ps_shift : k / p.ps;
    if (blk >= p.bt_width) continue;
    if (bar) {
      const int page = bt[blk - bt_first];
#pragma unroll
      for (int a = 0; a < KA; ++a) tma_load_4d(dst + (size_t)a * atom + (size_t)(k - kt) * 128, map, bar, a * 64, k - blk * p.ps, hk, page);
    }
    ++n;
  }
  return n;
}

// ------------------------------------------------------------------------------------------------------------ scores
__global__ void __launch_bounds__(64 + EPI * 32, 2) scores_tc_kernel(const __grid_constant__ CUtensorMap map_q,
                                                                     const __grid_constant__ CUtensorMap map_k, const Params p, int n_runs,
                                                                     int run_steps, int* error) {
  extern __shared__ __align__(1024) unsigned char smem[];
  unsigned char *Qs = smem, *Ks = smem + Q_BYTES;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + S_TILES + S_STAGE);
  uint64_t &q_full = bars[0], *k_full = bars + 1, *k_empty = bars + 1 + NS_S, *s_full = bars + 1 + 2 * NS_S, *s_empty = bars + 3 + 2 * NS_S;
  uint32_t& tmem_base_s = *reinterpret_cast<uint32_t*>(bars + 5 + 2 * NS_S);
  int* bt_s = reinterpret_cast<int*>(smem + S_TILES + S_STAGE + 256);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait();
  Tile w;
  if (!find_tile(p, blockIdx.y / n_runs, w)) return;
  const int run = blockIdx.y % n_runs;
  const int n_steps_all = (w.hi - w.kt0 + BN - 1) / BN, step0 = run * run_steps, n_steps = min(n_steps_all - step0, run_steps);
  if (n_steps <= 0) return;
  if ((smem_u32(smem) & 1023u) != 0) {                        // never seen; refuse rather than compute with a wrong swizzle
    if (threadIdx.x == 0) atomicExch(error, 1);
    return;
  }
  const int kt_first = w.kt0 + step0 * BN;
  if (threadIdx.x == 0) {
    mbar_init(&q_full, 1);
#pragma unroll
    for (int s = 0; s < NS_S; ++s) { mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1); }
#pragma unroll
    for (int b = 0; b < 2; ++b) { mbar_init(&s_full[b], 1); mbar_init(&s_empty[b], EPI / 2); }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base_s)), "r"(S_COLS) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = tmem_base_s;
  const int tpt = BM / p.per;
  bool failed = false;

  if (warp == 0) {
    int bt_first;
    const int* bt = table_of(p, w, max(kt_first, w.lo), min(kt_first + n_steps * BN, w.hi), bt_s, lane, bt_first);
    if (lane == 0) {
      mbar_expect_tx(&q_full, (unsigned)(tpt * p.per * D * 2));
#pragma unroll
      for (int a = 0; a < KA; ++a) tma_load_4d(Qs + (size_t)a * BM * 128, &map_q, &q_full, a * 64, 0, w.hk, w.q0 + w.tok0);
      const unsigned box = (unsigned)((p.ps < BN ? p.ps : BN) * D * 2);
      for (int j = 0; j < n_steps; ++j) {
        const int s = j % NS_S, kt = kt_first + j * BN;
        if (!mbar_wait(&k_empty[s], ((j / NS_S) & 1) ^ 1)) { failed = true; break; }
        mbar_expect_tx(&k_full[s], load_keys(p, &map_k, bt, bt_first, w.hk, kt, w.lo, w.hi, nullptr, 0, nullptr) * box);
        load_keys(p, &map_k, bt, bt_first, w.hk, kt, w.lo, w.hi, Ks + (size_t)s * K_BYTES, BN * 128, &k_full[s]);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = make_idesc(BM, BN, false);
      const uint64_t dq = make_desc(smem_u32(Qs), 0);
      failed = !mbar_wait(&q_full, 0);
      for (int j = 0; j < n_steps && !failed; ++j) {
        if (!mbar_wait(&k_full[j % NS_S], (j / NS_S) & 1) || !mbar_wait(&s_empty[j & 1], ((j >> 1) & 1) ^ 1)) { failed = true; break; }
        tc_fence_after();
        const uint64_t dk = make_desc(smem_u32(Ks + (size_t)(j % NS_S) * K_BYTES), 0);
        const uint32_t acc = tmem_base + (uint32_t)((j & 1) * BN);
#pragma unroll
        for (int kk = 0; kk < D / 16; ++kk) {
          // 16 k-values further: 32 bytes within an atom (4 steps), then the next atom of Q (128 rows) and K (64 rows)
          const uint64_t qo = (uint64_t)((kk >> 2) * (BM * 128 >> 4) + (kk & 3) * 2), ko = (uint64_t)((kk >> 2) * (BN * 128 >> 4) + (kk & 3) * 2);
          tc_mma(acc, dq + qo, dk + ko, idesc, kk != 0 ? 1u : 0u);
        }
        tc_commit(&s_full[j & 1]);
        tc_commit(&k_empty[j % NS_S]);
      }
    }
  } else {
    const int q = warp & 3, set = (warp - 2) >> 2;            // the 32 tensor-memory lanes of this warp; the buffer it reads
    const int row = q * 32 + lane, tok = row / p.per;
    const bool row_ok = row < tpt * p.per && w.tok0 + tok < w.tok1;
    const int pos = row_ok ? w.p0 + w.tok0 + tok : -1;
    const size_t srow = row_ok ? (size_t)(w.q0 + w.tok0 + tok - p.t_lo) * p.H + w.hk * p.per + (row - tok * p.per) : 0;
    float* stage = reinterpret_cast<float*>(smem + S_TILES) + (warp - 2) * 32 * LDE;
    const uint32_t lane_addr = tmem_base + ((uint32_t)(q * 32) << 16) + (uint32_t)(set * BN);
    const int first_pos = w.p0 + w.tok0;                      // smallest position of the tile's rows
    const float two_in = p.cap_in * (2.f * LOG2E), cap_log2 = p.cap * LOG2E, scale_log2 = p.scale * LOG2E;
    const int tiles_pitch = p.pitch / BN;
    for (int j = set; j < n_steps && !failed; j += 2) {
      if (!mbar_wait(&s_full[set], (j >> 1) & 1)) { failed = true; break; }
      tc_fence_after();
      const int kt = kt_first + j * BN;
      float v[BN];
      tc_load32(lane_addr, v);
      tc_load32(lane_addr + 32u, v + 32);
      tc_wait_ld();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&s_empty[set]);              // the scores are in registers: the buffer may be used again
      const bool live = kt <= pos;                            // the row reads keys of this tile (its first key is never behind it)
      if (!__any_sync(0xffffffffu, live)) continue;
      if (p.cap > 0.f) {
        float big = 0.f;
#pragma unroll
        for (int i = 0; i < BN; ++i) big = fmaxf(big, fabsf(v[i]));
        if (__all_sync(0xffffffffu, big * p.cap_in <= SERIES_LIMIT)) {
#pragma unroll
          for (int i = 0; i < BN; ++i) v[i] = cap_log2 * tanh_series(v[i] * p.cap_in);
        } else {
#pragma unroll
          for (int i = 0; i < BN; ++i) v[i] = capped_log2(v[i], two_in, cap_log2);
        }
      } else {
#pragma unroll
        for (int i = 0; i < BN; ++i) v[i] *= scale_log2;
      }
      if (kt + BN - 1 > first_pos || kt < w.lo) {
#pragma unroll
        for (int i = 0; i < BN; ++i) v[i] = (kt + i <= pos && kt + i >= w.lo) ? v[i] : -INFINITY;
      }
      float m = 0.f;
      if (!p.fixed) {
        m = -INFINITY;
#pragma unroll
        for (int i = 0; i < BN; ++i) m = fmaxf(m, v[i]);
        const float ref = (m == -INFINITY) ? 0.f : m;
#pragma unroll
        for (int i = 0; i < BN; ++i) v[i] -= ref;
      }
      float s0 = 0.f, s1 = 0.f;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
#pragma unroll
        for (int i = 0; i < 32; i += 4) {
          float4 e;
          e.x = ex2(v[half * 32 + i]); e.y = ex2(v[half * 32 + i + 1]); e.z = ex2(v[half * 32 + i + 2]); e.w = ex2(v[half * 32 + i + 3]);
          s0 += e.x + e.y;
          s1 += e.z + e.w;
          *reinterpret_cast<float4*>(stage + lane * LDE + i) = e;
        }
        __syncwarp();
        // four rows an instruction: eight lanes a row, 16 bytes each
        float* dst0 = p.e + (kt - w.kt0) + half * 32 + (lane & 7) * 4;
#pragma unroll
        for (int i = 0; i < 32; i += 4) {
          const int rr = i + (lane >> 3);
          const unsigned at = __shfl_sync(0xffffffffu, live ? (unsigned)srow : 0xffffffffu, rr);
          if (at != 0xffffffffu)
            *reinterpret_cast<float4*>(dst0 + (size_t)at * p.pitch) = *reinterpret_cast<const float4*>(stage + rr * LDE + (lane & 7) * 4);
        }
        __syncwarp();
      }
      if (live) p.stats[srow * tiles_pitch + (kt - w.kt0) / BN] = make_float2(m, s0 + s1);
    }
  }
  if (failed) atomicExch(error, 1);
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(S_COLS) : "memory");
  }
}

// ------------------------------------------------------------------------------------------------------------ values
__global__ void __launch_bounds__(192, 2) values_tc_kernel(const __grid_constant__ CUtensorMap map_w,
                                                           const __grid_constant__ CUtensorMap map_v, const Params p, int* error) {
  extern __shared__ __align__(1024) unsigned char smem[];
  unsigned char *Ws = smem, *Vs = smem + NS_V * W_BYTES;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + V_TILES);
  uint64_t *full = bars, *empty = bars + NS_V, &landed = bars[2 * NS_V], &cleared = bars[2 * NS_V + 1], &o_full = bars[2 * NS_V + 2];
  uint32_t& tmem_base_s = *reinterpret_cast<uint32_t*>(bars + 2 * NS_V + 3);
  int* bt_s = reinterpret_cast<int*>(smem + V_TILES + 256);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait();
  Tile w;
  if (!find_tile(p, blockIdx.y, w)) return;
  if ((smem_u32(smem) & 1023u) != 0) {
    if (threadIdx.x == 0) atomicExch(error, 1);
    return;
  }
  const int n_tiles = (w.hi - w.kt0 + BN - 1) / BN;
  if (threadIdx.x == 0) {
#pragma unroll
    for (int s = 0; s < NS_V; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
    mbar_init(&landed, 1);
    mbar_init(&cleared, 4);
    mbar_init(&o_full, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base_s)), "r"(V_COLS) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = tmem_base_s;
  const int tpt = BM / p.per;
  bool failed = false;
  // the value rows of tile j that hold no key the tile's rows can see: [0, head) and [tail, 64)
  auto edges = [&](int j, int& head, int& tail) {
    head = j == 0 ? w.lo - w.kt0 : 0;
    tail = min(BN, w.hi - (w.kt0 + j * BN));
    return head > 0 || tail < BN;
  };

  if (warp == 0) {
    int bt_first;
    const int* bt = table_of(p, w, w.lo, w.hi, bt_s, lane, bt_first);
    if (lane == 0) {
      const unsigned box = (unsigned)((p.ps < BN ? p.ps : BN) * D * 2);
      for (int j = 0; j < n_tiles; ++j) {
        const int s = j % NS_V, kt = w.kt0 + j * BN;
        if (!mbar_wait(&empty[s], ((j / NS_V) & 1) ^ 1)) { failed = true; break; }
        const int n = load_keys(p, &map_v, bt, bt_first, w.hk, kt, w.lo, w.hi, nullptr, 0, nullptr);
        mbar_expect_tx(&full[s], n * box + (unsigned)(tpt * p.per * BN * 2));
        tma_load_4d(Ws + (size_t)s * W_BYTES, &map_w, &full[s], j * BN, 0, w.hk, w.q0 + w.tok0 - p.t_lo);
        load_keys(p, &map_v, bt, bt_first, w.hk, kt, w.lo, w.hi, Vs + (size_t)s * V_BYTES, BN * 128, &full[s]);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = make_idesc(BM, D, true);
      unsigned clears = 0;
      for (int j = 0; j < n_tiles; ++j) {
        const int s = j % NS_V;
        if (!mbar_wait(&full[s], (j / NS_V) & 1)) { failed = true; break; }
        int head, tail;
        if (edges(j, head, tail)) {
          mbar_arrive(&landed);
          if (!mbar_wait(&cleared, clears & 1)) { failed = true; break; }
          ++clears;
        }
        tc_fence_after();
        const uint32_t wa = smem_u32(Ws + (size_t)s * W_BYTES), va = smem_u32(Vs + (size_t)s * V_BYTES);
#pragma unroll
        for (int kk = 0; kk < BN / 16; ++kk)
          tc_mma(tmem_base, make_desc(wa + (uint32_t)(kk * 32), 0), make_desc(va + (uint32_t)(kk * 2048), BN * 128), idesc, (j | kk) != 0 ? 1u : 0u);
        tc_commit(&empty[s]);
      }
      tc_commit(&o_full);
    }
  } else {
    unsigned clears = 0;
    for (int j = 0; j < n_tiles && !failed; j = (j == 0 && n_tiles > 1) ? n_tiles - 1 : n_tiles) {
      int head, tail;
      if (!edges(j, head, tail)) continue;
      if (!mbar_wait(&landed, clears & 1)) { failed = true; break; }
      ++clears;
      unsigned char* vt = Vs + (size_t)(j % NS_V) * V_BYTES;
      const int gone = head + (BN - tail);
      for (int idx = (warp - 2) * 32 + lane; idx < gone * 8 * KA; idx += 128) {
        const int a = idx / (gone * 8), rest = idx - a * gone * 8, at = rest >> 3, vrow = at < head ? at : tail + (at - head);
        *reinterpret_cast<uint4*>(vt + (size_t)a * BN * 128 + (size_t)vrow * 128 + ((rest & 7) << 4)) = make_uint4(0u, 0u, 0u, 0u);
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");   // these writes are read by the tensor core
      __syncwarp();
      if (lane == 0) mbar_arrive(&cleared);
    }
    if (!failed && !mbar_wait(&o_full, 0)) failed = true;
    tc_fence_after();
    if (!failed) {
      const int q = warp & 3, row = q * 32 + lane, tok = row / p.per;
      float o[D];
#pragma unroll
      for (int c = 0; c < D / 32; ++c) tc_load32(tmem_base + ((uint32_t)(q * 32) << 16) + (uint32_t)(c * 32), o + c * 32);
      tc_wait_ld();
      if (row < tpt * p.per && w.tok0 + tok < w.tok1) {
        bf16* dst = (bf16*)p.out + ((size_t)(w.q0 + w.tok0 + tok) * p.H + w.hk * p.per + (row - tok * p.per)) * D;
#pragma unroll
        for (int i = 0; i < D / 8; ++i)
          *reinterpret_cast<uint4*>(dst + i * 8) = make_uint4(pack_bf16(o[8 * i], o[8 * i + 1]), pack_bf16(o[8 * i + 2], o[8 * i + 3]),
                                                              pack_bf16(o[8 * i + 4], o[8 * i + 5]), pack_bf16(o[8 * i + 6], o[8 * i + 7]));
      }
    }
  }
  if (failed) atomicExch(error, 1);
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(V_COLS) : "memory");
  }
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                  const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                  CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
EncodeTiledFn g_encode = nullptr;

int encode4(CUtensorMap* map, const void* basep, const cuuint64_t (&dims)[4], const cuuint64_t (&strides)[3], const cuuint32_t (&box)[4]) {
  if (!g_encode) {
    void* fn = nullptr;
    cudaDriverEntryPointQueryResult qres;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &qres) != cudaSuccess || !fn) return -300;
    g_encode = (EncodeTiledFn)fn;
  }
  const cuuint32_t estr[4] = {1, 1, 1, 1};
  const CUresult rc = g_encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, const_cast<void*>(basep), dims, strides, box, estr,
                               CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
                               CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return rc == CUDA_SUCCESS ? 0 : -301 - (int)rc;
}

// a [tokens, G, per, row of ``cols`` elements] tensor whose tokens are ``stride`` elements apart, in boxes of 64 elements of a tile's rows
int encode_rows(CUtensorMap* map, const void* basep, const Params& p, int n_tokens, int cols, size_t stride) {
  const cuuint64_t dims[4] = {(cuuint64_t)cols, (cuuint64_t)p.per, (cuuint64_t)p.G, (cuuint64_t)n_tokens};
  const cuuint64_t strides[3] = {(cuuint64_t)cols * 2, (cuuint64_t)p.per * cols * 2, (cuuint64_t)stride * 2};
  const cuuint32_t box[4] = {64, (cuuint32_t)p.per, 1, (cuuint32_t)(BM / p.per)};
  return encode4(map, basep, dims, strides, box);
}
int encode_cache(CUtensorMap* map, const void* basep, const Params& p) {
  const cuuint64_t dims[4] = {(cuuint64_t)D, (cuuint64_t)p.ps, (cuuint64_t)p.G, (cuuint64_t)p.num_pages};
  const cuuint64_t strides[3] = {(cuuint64_t)D * 2, (cuuint64_t)p.ps * D * 2, (cuuint64_t)p.G * p.ps * D * 2};
  const cuuint32_t box[4] = {64, (cuuint32_t)(p.ps < BN ? p.ps : BN), 1, 1};
  return encode4(map, basep, dims, strides, box);
}
int row_tiles(const Params& p, int max_q) {
  const int tpt = BM / p.per;
  return (max_q + tpt - 1) / tpt + (p.chunk > 0 ? max_q / p.chunk + 2 : 0);      // (a tile more at every border inside the portion)
}

}  // namespace

bool tc_takes(int H, int G, int ps, int q_stride, int chunk) {
  const int per = H / G;
  if (per > BM || ps < 8 || q_stride % 8 || (chunk > 0 && chunk < BN)) return false;      // (short blocks would leave tiles mostly empty)
  return ps <= BN ? BN % ps == 0 : (ps % BN == 0 && ps <= 256);
}
int tc_tokens_per_tile(int H, int G) { return BM / (H / G); }

int tc_scores(const Params& p, int n_tokens, int max_keys, int max_q, int n_requests, int* error, cudaStream_t stream) {
  CUtensorMap map_q, map_k;
  if (int rc = encode_rows(&map_q, p.q, p, n_tokens, D, p.q_stride)) return rc;
  if (int rc = encode_cache(&map_k, p.kc, p)) return rc;
  const int steps = (max_keys + BN - 1) / BN, tiles = row_tiles(p, max_q);
  const int run_steps = (long long)tiles * p.G * n_requests * ((steps + RUN - 1) / RUN) >= 3 * sm_count() ? RUN : RUN_FEW;
  const int n_runs = (steps + run_steps - 1) / run_steps;
  const long long y = (long long)tiles * n_runs;
  if (y > 65535) return SB_ERR_LIMIT;
  cudaFuncSetAttribute(scores_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, S_SMEM);
  SB_PDL_CHECK(launch_pdl(scores_tc_kernel, dim3(p.G, (unsigned)y, n_requests), dim3(64 + EPI * 32), (size_t)S_SMEM, stream, map_q, map_k, p,
                          n_runs, run_steps, error));
  return 0;
}

int tc_values(const Params& p, int max_q, int n_requests, int* error, cudaStream_t stream) {
  CUtensorMap map_w, map_v;
  if (int rc = encode_rows(&map_w, p.w, p, p.t_hi - p.t_lo, p.pitch, (size_t)p.H * p.pitch)) return rc;
  if (int rc = encode_cache(&map_v, p.vc, p)) return rc;
  cudaFuncSetAttribute(values_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, V_SMEM);
  SB_PDL_CHECK(launch_pdl(values_tc_kernel, dim3(p.G, (unsigned)row_tiles(p, max_q), n_requests), dim3(192), (size_t)V_SMEM, stream, map_w, map_v,
                          p, error));
  return 0;
}

}  // namespace talk

#else

namespace talk {
bool tc_takes(int, int, int, int, int) { return false; }
int tc_tokens_per_tile(int, int) { return 1; }
int tc_scores(const Params&, int, int, int, int, int*, cudaStream_t) { return SB_ERR_SHAPE; }
int tc_values(const Params&, int, int, int*, cudaStream_t) { return SB_ERR_SHAPE; }
}  // namespace talk

#endif
