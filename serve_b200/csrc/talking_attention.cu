// Attention whose heads' weights are mixed by an H x H matrix between the softmax and the values ("talking heads"):
//
//   s_h(i, j) = cap * tanh((q_h(i) . k(j)) * scale / cap)           (or without a cap)
//   p_h(i, j) = exp(s_h(i, j)) / (exp(sink_h) + sum_j exp(s_h(i, j)))   over the visible keys (the sink is optional)
//   w_h(i, j) = sum_g talk[h, g] p_g(i, j),    out_h(i) = sum_j w_h(i, j) v(j)
//
// A weight that meets a value needs the finished softmax of every head, so the work is three passes over a scratch buffer:
//
//   scores  per (request, kv head, rows, keys): e = exp(s - m), m the maximum of the row's tile of 64 keys, and per tile (m, sum)
//   mix     per token: the tiles' (m, sum) give every head's maximum and denominator; p = e * exp(m - M) / den, mixed over the heads
//   values  per (request, kv head, rows): the product of mixed weights and values
//
// (a step of few rows mixes inside the values' kernel: two passes)
//
// Scratch rows: token t (counted from the first token of the launch), head h, ``pitch`` keys, column 0 standing for the key
// base(t) = the first key the token may read, rounded down to a tile of 64. Tiles never depend on how a prompt was cut or on
// what else is in the batch. A query sees the keys j <= i, with ``chunk`` > 0 only those of its own block of chunk positions.
//
// In bfloat16 scores and values run on mma.sync m16n8k16 with float accumulation, and so does the mix: p is split into two
// bfloat16 numbers (p = hi + lo to 2^-17), so the mixed weights keep float's sums and are rounded once, for the product with the
// values. In float32 everything is plain fused multiply-adds. Two shapes, as in the other attention kernels: requests with at most
// 16 rows (tokens x heads of a kv head) are "deep", the others "wide". Compile with -DSB_HEAD_DIM=<multiple of 16, 16..256>.
#include "talking_attention.cuh"

#ifndef SB_HEAD_DIM
#error "define SB_HEAD_DIM"
#endif

using namespace sb;
using namespace talk;
typedef __nv_bfloat16 bf16;

namespace {

constexpr int D = SB_HEAD_DIM;
constexpr int LDS = D + 8;           // row stride of a key or value tile in shared memory (elements)
constexpr int LDW = BN + 8;          // row stride of a weight tile in shared memory
constexpr int CHUNKS = D / 8;        // 16-byte pieces per row
// shared memory of the deep values: four warps' 32 value rows, over which their sums [4][16][D + 2] lie afterwards
constexpr size_t DEEP_TILES = (size_t)4 * 32 * LDS * 2, DEEP_SUMS = (size_t)4 * 16 * (D + 2) * 4;
constexpr size_t DEEP_BYTES = ((DEEP_TILES > DEEP_SUMS ? DEEP_TILES : DEEP_SUMS) + 15) / 16 * 16;
static_assert(D % 16 == 0 && D >= 16 && D <= 256, "head_dim must be a multiple of 16 in 16..256");

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool valid) {
  const int n = valid ? 16 : 0;   // 0: nothing is read, the 16 bytes are filled with zeros
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(smem_u32(dst)), "l"(src), "r"(n));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N)); }
__device__ __forceinline__ void ldmatrix_x4(uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}

// Where key ``key`` of kv head hk lies in a cache tensor (elements), or -1 where there is no page.
__device__ __forceinline__ long long cache_row(const Params& p, const int* bt, int hk, int key) {
  const int blk = p.ps_shift >= 0 ? (key >> p.ps_shift) : key / p.ps;
  const int page = blk < p.bt_width ? bt[blk] : -1;
  if (page < 0 || page >= p.num_pages) return -1;
  return (((long long)page * p.G + hk) * p.ps + (key - blk * p.ps)) * D;
}

// keys [kt, kt + 64) of kv head hk into shared memory; keys outside [lo, hi) become zeros. BY_COLUMN: in the order of the scores'
// product columns (row 8 nt + n holds key column_key(nt, n)), so that the rows of a matrix fragment are neighbours.
template <bool BY_COLUMN>
__device__ __forceinline__ void load_tile(const Params& p, const bf16* cache, const int* bt, int hk, int kt, int lo, int hi, bf16* dst,
                                          int tid, int nthreads) {
  for (int idx = tid; idx < BN * CHUNKS; idx += nthreads) {
    const int row = idx / CHUNKS, ch = idx - row * CHUNKS, key = kt + row;
    const long long off = (key >= lo && key < hi) ? cache_row(p, bt, hk, key) : -1;
    const int at = BY_COLUMN ? (row & ~15) + ((row & 2) << 2) + ((row >> 1) & 6) + (row & 1) : row;
    cp_async16(dst + at * LDS + ch * 8, cache + (off >= 0 ? off + ch * 8 : 0), off >= 0);
  }
}

// A row's scores of one tile (16 a lane over a quad of lanes, keys kt + 16 i + 4 tq + 0..3) -> e and the tile's (m, sum).
// raw[i][0..3]: the products; the row stores its tile if it reads any of its keys.
__device__ __forceinline__ void finish_row(const Params& p, float (&raw)[4][4], int kt, int first, int pos, size_t row, int tq) {
  float m = p.fixed ? 0.f : -INFINITY;
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const int key = kt + 16 * i + 4 * tq + c;
      const float s = (key >= first && key <= pos) ? score_log2(p, raw[i][c]) : -INFINITY;
      raw[i][c] = s;
      if (!p.fixed) m = fmaxf(m, s);
    }
  if (!p.fixed) {
    m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 1));
    m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 2));
  }
  const int base = first & ~(BN - 1);
  const bool live = pos >= 0 && kt >= base && kt <= pos;      // (then at least one key of the tile is visible and m is finite)
  float sum = 0.f;
  float* dst = p.e + row * p.pitch + (kt - base) + 4 * tq;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    float4 v;
    v.x = ex2(raw[i][0] - m); v.y = ex2(raw[i][1] - m); v.z = ex2(raw[i][2] - m); v.w = ex2(raw[i][3] - m);
    sum += (v.x + v.y) + (v.z + v.w);
    if (live) *reinterpret_cast<float4*>(dst + 16 * i) = v;
  }
  sum += __shfl_xor_sync(0xffffffffu, sum, 1);
  sum += __shfl_xor_sync(0xffffffffu, sum, 2);
  if (live && tq == 0) p.stats[row * (p.pitch / BN) + (kt - base) / BN] = make_float2(m, sum);
}

// The key of column n of product tile nt: a lane's two columns of tiles 2i and 2i+1 are then four neighbouring keys.
__device__ __forceinline__ int column_key(int nt, int n) { return 16 * (nt >> 1) + ((n >> 1) << 2) + (n & 1) + ((nt & 1) << 1); }

// What a wide block works on: rows [m0, m0 + BM) of (request, kv head), row m = (token m / per, head hk * per + m % per).
struct WideTile {
  int r, hk, q0, M, m0, p0, lo, hi;
  const int* bt;
};
template <int BM> __device__ __forceinline__ bool wide_tile(const Params& p, WideTile& w) {
  w.r = p.wide_rows ? p.wide_rows[blockIdx.z] : (int)blockIdx.z;
  w.hk = blockIdx.x;
  w.q0 = p.cu_q[w.r];
  const int qn = p.cu_q[w.r + 1] - w.q0;
  w.M = qn * p.per;
  if (p.deep_on && w.M <= 16) return false;
  const int n_tiles = (w.M + BM - 1) / BM;
  if ((int)blockIdx.y >= n_tiles) return false;
  w.m0 = (n_tiles - 1 - (int)blockIdx.y) * BM;                // later rows see more keys: they go first
  int tok_a = w.m0 / p.per, tok_b = (min(w.m0 + BM, w.M) - 1) / p.per;
  tok_a = max(tok_a, p.t_lo - w.q0);
  tok_b = min(tok_b, p.t_hi - 1 - w.q0);
  if (tok_a > tok_b) return false;                            // another launch covers these tokens
  w.p0 = p.kv_len[w.r] - qn;
  w.lo = first_key(p, w.p0 + tok_a);
  w.hi = w.p0 + tok_b + 1;
  w.bt = p.block_table + (size_t)w.r * p.bt_width;
  return true;
}
// Row m of the tile: scratch row and position (-1: the launch does not cover it).
__device__ __forceinline__ void row_of(const Params& p, const WideTile& w, int m, size_t& row, int& pos) {
  const int tok = m / p.per, t = w.q0 + tok;
  const bool ok = m < w.M && t >= p.t_lo && t < p.t_hi;
  pos = ok ? w.p0 + tok : -1;
  row = ok ? (size_t)(t - p.t_lo) * p.H + w.hk * p.per + (m - tok * p.per) : 0;
}

// ------------------------------------------------------------------------------------------------- scores, bfloat16
template <int NW>
__global__ void __launch_bounds__(NW * 32) scores_wide_kernel(const Params p) {
  constexpr int BM = 16 * NW, THREADS = 32 * NW;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  bf16* Qs = reinterpret_cast<bf16*>(smem_raw);               // [BM][LDS]
  bf16* Ks = Qs + BM * LDS;                                   // 2 stages x [BN][LDS]
  pdl_wait();
  WideTile w;
  if (!wide_tile<BM>(p, w)) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3;
  const bf16* q = (const bf16*)p.q;
  for (int idx = tid; idx < BM * CHUNKS; idx += THREADS) {
    const int row = idx / CHUNKS, ch = idx - row * CHUNKS, m = w.m0 + row;
    const bool ok = m < w.M;
    const int tok = ok ? m / p.per : 0, hd = ok ? w.hk * p.per + (m - tok * p.per) : 0;
    cp_async16(Qs + row * LDS + ch * 8, q + (size_t)(w.q0 + tok) * p.q_stride + (size_t)hd * D + ch * 8, ok);
  }
  const int kt0 = w.lo & ~(BN - 1), n_tiles = (w.hi - kt0 + BN - 1) / BN;
  load_tile<true>(p, (const bf16*)p.kc, w.bt, w.hk, kt0, w.lo, w.hi, Ks, tid, THREADS);
  cp_async_commit();
  size_t row_a, row_b;
  int pos_a, pos_b;
  row_of(p, w, w.m0 + warp * 16 + g, row_a, pos_a);
  row_of(p, w, w.m0 + warp * 16 + g + 8, row_b, pos_b);
  const int first_a = pos_a >= 0 ? first_key(p, pos_a) : 0, first_b = pos_b >= 0 ? first_key(p, pos_b) : 0;
  constexpr bool Q_REGS = D <= 128;
  uint32_t qf[Q_REGS ? D / 16 : 1][4];
  for (int it = 0; it < n_tiles; ++it) {
    const int kt = kt0 + it * BN;
    const bf16* K = Ks + (it & 1) * BN * LDS;
    if (it + 1 < n_tiles) {
      load_tile<true>(p, (const bf16*)p.kc, w.bt, w.hk, kt + BN, w.lo, w.hi, Ks + ((it + 1) & 1) * BN * LDS, tid, THREADS);
      cp_async_commit();
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    if (Q_REGS && it == 0) {
#pragma unroll
      for (int kk = 0; kk < D / 16; ++kk)
        ldmatrix_x4(qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3], Qs + (warp * 16 + (lane & 15)) * LDS + kk * 16 + (lane >> 4) * 8);
    }
    float acc[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < D / 16; ++kk) {
      uint32_t a0, a1, a2, a3;
      if (Q_REGS) { a0 = qf[kk][0]; a1 = qf[kk][1]; a2 = qf[kk][2]; a3 = qf[kk][3]; }
      else ldmatrix_x4(a0, a1, a2, a3, Qs + (warp * 16 + (lane & 15)) * LDS + kk * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        // matrices: (tile 2i, k 0-7), (tile 2i, k 8-15), (tile 2i+1, k 0-7), (tile 2i+1, k 8-15)
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4(b0, b1, b2, b3, K + (16 * i + (lane & 7) + ((lane >> 4) << 3)) * LDS + kk * 16 + ((lane >> 3) & 1) * 8);
        mma_bf16(acc[2 * i], a0, a1, a2, a3, b0, b1);
        mma_bf16(acc[2 * i + 1], a0, a1, a2, a3, b2, b3);
      }
    }
    float ra[4][4], rb[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      ra[i][0] = acc[2 * i][0]; ra[i][1] = acc[2 * i][1]; ra[i][2] = acc[2 * i + 1][0]; ra[i][3] = acc[2 * i + 1][1];
      rb[i][0] = acc[2 * i][2]; rb[i][1] = acc[2 * i][3]; rb[i][2] = acc[2 * i + 1][2]; rb[i][3] = acc[2 * i + 1][3];
    }
    finish_row(p, ra, kt, first_a, pos_a, row_a, tq);
    finish_row(p, rb, kt, first_b, pos_b, row_b, tq);
    __syncthreads();
  }
  pdl_launch_dependents();
}

// Requests of at most 16 rows: a warp per (request, kv head, tile of 64 keys), keys straight from memory into the product's
// registers. A lane fetches 16 bytes of a key at a time; the order of the head's elements inside a product step is the
// lanes', the same for queries and keys.
__global__ void __launch_bounds__(128) scores_deep_kernel(const Params p) {
  constexpr int NB = D / 32;                 // whole blocks of 32 elements; a last one of 16 if D is an odd multiple of 16
  constexpr bool TAIL = (D % 32) != 0;
  constexpr int AT_ONCE = D <= 64 ? 8 : (D <= 128 ? 4 : 2);
  pdl_wait();
  const int r = blockIdx.z, hk = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, tq = lane & 3;
  const int q0 = p.cu_q[r], qn = p.cu_q[r + 1] - q0, M = qn * p.per;
  if (M <= 0 || M > 16) return;
  const int p0 = p.kv_len[r] - qn;
  const int lo = first_key(p, p0), hi = p0 + qn, kt0 = lo & ~(BN - 1), n_tiles = (hi - kt0 + BN - 1) / BN;
  const int first_tile = blockIdx.y * 4 + warp;
  if (first_tile >= n_tiles) return;
  const int* bt = p.block_table + (size_t)r * p.bt_width;
  const bf16 *q = (const bf16*)p.q, *kc = (const bf16*)p.kc;
  uint4 qa[NB > 0 ? NB : 1], qb[NB > 0 ? NB : 1];
  uint2 ta = make_uint2(0, 0), tb = make_uint2(0, 0);
  size_t row_a = 0, row_b = 0;
  int pos_a = -1, pos_b = -1;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int m = g + 8 * half;
    const int tok = m / p.per, t = q0 + tok, hd = hk * p.per + (m - tok * p.per);
    const bool ok = m < M && t >= p.t_lo && t < p.t_hi;
    const bf16* src = q + (size_t)(ok ? t : q0) * p.q_stride + (size_t)(ok ? hd : 0) * D;
    if (half == 0) { pos_a = ok ? p0 + tok : -1; row_a = ok ? (size_t)(t - p.t_lo) * p.H + hd : 0; }
    else { pos_b = ok ? p0 + tok : -1; row_b = ok ? (size_t)(t - p.t_lo) * p.H + hd : 0; }
#pragma unroll
    for (int b = 0; b < NB; ++b) {
      const uint4 v = ok ? *reinterpret_cast<const uint4*>(src + b * 32 + tq * 8) : make_uint4(0, 0, 0, 0);
      if (half == 0) qa[b] = v; else qb[b] = v;
    }
    if (TAIL) {
      const uint2 v = ok ? *reinterpret_cast<const uint2*>(src + NB * 32 + tq * 4) : make_uint2(0, 0);
      if (half == 0) ta = v; else tb = v;
    }
  }
  const int first_a = pos_a >= 0 ? first_key(p, pos_a) : 0, first_b = pos_b >= 0 ? first_key(p, pos_b) : 0;
  for (int tile = first_tile; tile < n_tiles; tile += gridDim.y * 4) {
    const int kt = kt0 + tile * BN;
    float acc[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
#pragma unroll
    for (int n0 = 0; n0 < 8; n0 += AT_ONCE) {
      uint4 kf[AT_ONCE][NB > 0 ? NB : 1];
      uint2 kt2[AT_ONCE];
#pragma unroll
      for (int n = 0; n < AT_ONCE; ++n) {
        const int key = kt + column_key(n0 + n, g);
        const long long off = (key >= lo && key < hi) ? cache_row(p, bt, hk, key) : -1;
#pragma unroll
        for (int b = 0; b < NB; ++b)
          kf[n][b] = off >= 0 ? *reinterpret_cast<const uint4*>(kc + off + b * 32 + tq * 8) : make_uint4(0, 0, 0, 0);
        if (TAIL) kt2[n] = off >= 0 ? *reinterpret_cast<const uint2*>(kc + off + NB * 32 + tq * 4) : make_uint2(0, 0);
      }
#pragma unroll
      for (int n = 0; n < AT_ONCE; ++n) {
#pragma unroll
        for (int b = 0; b < NB; ++b) {
          mma_bf16(acc[n0 + n], qa[b].x, qb[b].x, qa[b].y, qb[b].y, kf[n][b].x, kf[n][b].y);
          mma_bf16(acc[n0 + n], qa[b].z, qb[b].z, qa[b].w, qb[b].w, kf[n][b].z, kf[n][b].w);
        }
        if (TAIL) mma_bf16(acc[n0 + n], ta.x, tb.x, ta.y, tb.y, kt2[n].x, kt2[n].y);
      }
    }
    float ra[4][4], rb[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      ra[i][0] = acc[2 * i][0]; ra[i][1] = acc[2 * i][1]; ra[i][2] = acc[2 * i + 1][0]; ra[i][3] = acc[2 * i + 1][1];
      rb[i][0] = acc[2 * i][2]; rb[i][1] = acc[2 * i][3]; rb[i][2] = acc[2 * i + 1][2]; rb[i][3] = acc[2 * i + 1][3];
    }
    finish_row(p, ra, kt, first_a, pos_a, row_a, tq);
    if (M > 8) finish_row(p, rb, kt, first_b, pos_b, row_b, tq);
  }
  pdl_launch_dependents();
}

// ---------------------------------------------------------------------------------------------------------- mix
// Every head's maximum (log2) and 1 / denominator of token row t (scratch), from the tiles' statistics: ``team`` neighbouring
// threads a head (a power of two up to 32).
__device__ __forceinline__ void token_softmax(const Params& p, int t, int n_tiles, float* M_s, float* inv_s) {
  const int tiles_pitch = p.pitch / BN;
  int team = 32;
  while (team > 1 && team * p.H > (int)blockDim.x) team >>= 1;
  const int at = threadIdx.x & (team - 1), per_round = blockDim.x / team;
  const int rounds = (p.H + per_round - 1) / per_round;
  for (int k = 0; k < rounds; ++k) {
    const int h = k * per_round + threadIdx.x / team;
    const bool ok = h < p.H;
    const float2* st = p.stats + ((size_t)t * p.H + (ok ? h : 0)) * tiles_pitch;
    const float sink = (p.sinks && ok) ? p.sinks[h] * LOG2E : -INFINITY;
    float m = p.fixed ? 0.f : sink, l = 0.f;
    if (p.fixed) {
      for (int i = at; i < n_tiles; i += team) l += st[i].y;
    } else {
      for (int i = at; i < n_tiles; i += team) m = fmaxf(m, st[i].x);
      for (int o = team >> 1; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
      for (int i = at; i < n_tiles; i += team) l += st[i].y * exp2f(st[i].x - m);
    }
    for (int o = team >> 1; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
    if (ok && at == 0) { M_s[h] = m; inv_s[h] = 1.f / (l + exp2f(sink - m)); }
  }
  __syncthreads();
}

// grid (tokens, tile blocks), 4 warps; a warp takes tiles of 64 keys, a strip of 32 at a time. The product is talk [16 MT x Hp] times
// p [Hp x 32 keys], 16 heads g a step; column n of the q-th of a strip's four product tiles stands for key 4 n + q, so a lane reads 16
// bytes of a head's row and writes 16. A step's rows are fetched while the step before it is computed.
template <int MT>
__global__ void __launch_bounds__(128) mix_kernel(const Params p) {
  extern __shared__ float mix_s[];
  float *M_s = mix_s, *inv_s = mix_s + p.H;
  pdl_wait();
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, tq = lane & 3;
  const int pos = p.positions[p.t_lo + t];
  const int base = first_key(p, pos) & ~(BN - 1), n_tiles = (pos - base) / BN + 1;
  const int n_all = p.zero_ahead ? min((pos + p.zero_ahead - base) / BN + 1, p.pitch / BN) : n_tiles;
  if ((int)blockIdx.y * 4 >= n_all) return;
  const int tiles_pitch = p.pitch / BN, tile_step = gridDim.y * 4;
  const int kt_n = (p.H + 15) / 16, hp = kt_n * 16;
  const uint32_t* talk = reinterpret_cast<const uint32_t*>(p.talk);     // pairs of neighbouring columns
  const size_t row0 = (size_t)t * p.H;
  // heads kk * 16 + 2 tq + {0, 1, 8, 9}: e of four keys each
  auto head_of = [&](int kk, int i) { return kk * 16 + 2 * tq + (i & 1) + ((i >> 1) << 3); };
  auto fetch = [&](int tile, int strip, int kk, float4 (&ev)[4]) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int h = head_of(kk, i);
      ev[i] = h < p.H ? __ldcs(reinterpret_cast<const float4*>(p.e + (row0 + h) * p.pitch + tile * BN + strip * 32 + g * 4))
                      : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  int tile = blockIdx.y * 4 + warp, strip = 0, mg = 0, kk = 0;
  float4 next[4];
  if (tile < n_tiles) fetch(tile, 0, 0, next);
  token_softmax(p, t, n_tiles, M_s, inv_s);
  float acc[MT][4][4];
  while (tile < n_tiles) {
    float4 ev[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) ev[i] = next[i];
    const int at_tile = tile, at_strip = strip, at_mg = mg, at_kk = kk;
    if (++kk == kt_n) {
      kk = 0;
      mg += MT;
      if (mg >= kt_n) {
        mg = 0;
        strip ^= 1;
        if (strip == 0) tile += tile_step;
      }
    }
    if (tile < n_tiles) fetch(tile, strip, kk, next);
    if (at_kk == 0) {
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < 4; ++n) acc[m][n][0] = acc[m][n][1] = acc[m][n][2] = acc[m][n][3] = 0.f;
    }
    uint32_t hi[4][2], lo[4][2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      float f[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int h = head_of(at_kk, 2 * j + i);
        f[i] = h < p.H ? inv_s[h] : 0.f;
        if (!p.fixed && h < p.H) f[i] *= ex2(p.stats[(row0 + h) * tiles_pitch + at_tile].x - M_s[h]);
      }
      const float4 a = ev[2 * j], b = ev[2 * j + 1];
      const float xs[4] = {a.x * f[0], a.y * f[0], a.z * f[0], a.w * f[0]}, ys[4] = {b.x * f[1], b.y * f[1], b.z * f[1], b.w * f[1]};
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const __nv_bfloat162 h2 = __floats2bfloat162_rn(xs[n], ys[n]);
        hi[n][j] = *reinterpret_cast<const uint32_t*>(&h2);
        lo[n][j] = pack_bf16(xs[n] - __low2float(h2), ys[n] - __high2float(h2));
      }
    }
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      if (at_mg + m < kt_n) {
        const uint32_t* a = talk + ((size_t)((at_mg + m) * 16 + g) * hp + at_kk * 16) / 2 + tq;
        const uint32_t a0 = __ldg(a), a1 = __ldg(a + 4 * hp), a2 = __ldg(a + 4), a3 = __ldg(a + 4 * hp + 4);
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          mma_bf16(acc[m][n], a0, a1, a2, a3, lo[n][0], lo[n][1]);
          mma_bf16(acc[m][n], a0, a1, a2, a3, hi[n][0], hi[n][1]);
        }
      }
    }
    if (at_kk != kt_n - 1) continue;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int h = (at_mg + m) * 16 + g + 8 * half;
        if (h < p.H) {
          uint4 v;
          v.x = pack_bf16(acc[m][0][2 * half], acc[m][1][2 * half]);
          v.y = pack_bf16(acc[m][2][2 * half], acc[m][3][2 * half]);
          v.z = pack_bf16(acc[m][0][2 * half + 1], acc[m][1][2 * half + 1]);
          v.w = pack_bf16(acc[m][2][2 * half + 1], acc[m][3][2 * half + 1]);
          *reinterpret_cast<uint4*>((bf16*)p.w + (row0 + h) * p.pitch + at_tile * BN + at_strip * 32 + tq * 8) = v;
        }
      }
  }
  for (; tile < n_all; tile += tile_step)
    for (int h = g; h < p.H; h += 8) {
      uint4* dst = reinterpret_cast<uint4*>((bf16*)p.w + (row0 + h) * p.pitch + tile * BN + tq * 16);
      dst[0] = dst[1] = make_uint4(0, 0, 0, 0);
    }
}

// float32: a block per (token, tile of 64 keys); the tile's weights of all heads in shared memory (in parts of 128 heads).
__global__ void __launch_bounds__(256) mix_f32_kernel(const Params p) {
  constexpr int HB = 128;
  __shared__ float p_s[HB][BN];
  extern __shared__ float mix_s[];
  float *M_s = mix_s, *inv_s = mix_s + p.H;
  const int t = blockIdx.x;
  const int pos = p.positions[p.t_lo + t];
  const int base = first_key(p, pos) & ~(BN - 1), n_tiles = (pos - base) / BN + 1;
  if ((int)blockIdx.y >= n_tiles) return;
  token_softmax(p, t, n_tiles, M_s, inv_s);
  const size_t row0 = (size_t)t * p.H;
  const int key = threadIdx.x & 63, hq = threadIdx.x >> 6;
  float* w = (float*)p.w;
  const float* talk = (const float*)p.talk;
  for (int tile = blockIdx.y; tile < n_tiles; tile += gridDim.y) {
    for (int g0 = 0; g0 < p.H; g0 += HB) {
      const int gn = min(HB, p.H - g0);
      __syncthreads();
      for (int i = hq; i < gn; i += 4) {
        const int h = g0 + i;
        p_s[i][key] = p.e[(row0 + h) * p.pitch + tile * BN + key] * (exp2f(p.stats[(row0 + h) * (p.pitch / BN) + tile].x - M_s[h]) * inv_s[h]);
      }
      __syncthreads();
      for (int h = hq; h < p.H; h += 4) {
        float* dst = w + (row0 + h) * p.pitch + tile * BN + key;
        float a = g0 ? *dst : 0.f;                         // (this thread wrote it in the part before)
        for (int i = 0; i < gn; ++i) a = fmaf(talk[(size_t)h * p.H + g0 + i], p_s[i][key], a);
        *dst = a;
      }
    }
  }
}

// ------------------------------------------------------------------------------------------------- values, bfloat16
template <int NW>
__global__ void __launch_bounds__(NW * 32) values_wide_kernel(const Params p) {
  constexpr int BM = 16 * NW, THREADS = 32 * NW;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  bf16* Ws = reinterpret_cast<bf16*>(smem_raw);               // 2 stages x [BM][LDW]
  bf16* Vs = Ws + 2 * BM * LDW;                               // 2 stages x [BN][LDS]
  pdl_wait();
  WideTile w;
  if (!wide_tile<BM>(p, w)) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3;
  const int kt0 = w.lo & ~(BN - 1), n_tiles = (w.hi - kt0 + BN - 1) / BN;
  const bf16* ws = (const bf16*)p.w;
  auto load = [&](int it) {
    const int kt = kt0 + it * BN;
    bf16* W = Ws + (it & 1) * BM * LDW;
    for (int idx = tid; idx < BM * 8; idx += THREADS) {
      size_t row;
      int pos;
      row_of(p, w, w.m0 + (idx >> 3), row, pos);
      const int base = pos >= 0 ? first_key(p, pos) & ~(BN - 1) : 0;
      const bool ok = pos >= 0 && kt >= base && kt <= pos;    // (the tile's keys the row does not see carry zeros)
      cp_async16(W + (idx >> 3) * LDW + (idx & 7) * 8, ws + (ok ? row * p.pitch + (kt - base) + (idx & 7) * 8 : 0), ok);
    }
    load_tile<false>(p, (const bf16*)p.vc, w.bt, w.hk, kt, w.lo, w.hi, Vs + (it & 1) * BN * LDS, tid, THREADS);
    cp_async_commit();
  };
  load(0);
  float o[D / 8][4];
#pragma unroll
  for (int i = 0; i < D / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  for (int it = 0; it < n_tiles; ++it) {
    if (it + 1 < n_tiles) { load(it + 1); cp_async_wait<1>(); }
    else cp_async_wait<0>();
    __syncthreads();
    const bf16 *W = Ws + (it & 1) * BM * LDW, *V = Vs + (it & 1) * BN * LDS;
#pragma unroll
    for (int kk = 0; kk < BN / 16; ++kk) {
      uint32_t a0, a1, a2, a3;
      ldmatrix_x4(a0, a1, a2, a3, W + (warp * 16 + (lane & 15)) * LDW + kk * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int d = 0; d < D / 16; ++d) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(b0, b1, b2, b3, V + (kk * 16 + (lane & 15)) * LDS + d * 16 + (lane >> 4) * 8);
        mma_bf16(o[2 * d], a0, a1, a2, a3, b0, b1);
        mma_bf16(o[2 * d + 1], a0, a1, a2, a3, b2, b3);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int m = w.m0 + warp * 16 + g + 8 * half;
    size_t row;
    int pos;
    row_of(p, w, m, row, pos);
    if (pos < 0) continue;
    bf16* dst = (bf16*)p.out + ((size_t)p.t_lo * p.H + row) * D + tq * 2;
#pragma unroll
    for (int i = 0; i < D / 8; ++i) *reinterpret_cast<uint32_t*>(dst + i * 8) = pack_bf16(o[i][2 * half], o[i][2 * half + 1]);
  }
  pdl_launch_dependents();
}

// Requests of at most 16 rows: grid (kv heads, key splits, requests), 4 warps. A block takes 128 keys at a time, a warp 32 of them: a
// lane looks up where one key lies, and all of the warp's rows are on their way before the first is waited for. The warps' sums meet
// in shared memory, the splits' in the block that arrives last. FUSED: the step has few rows and no wide request, and the block mixes the weights
// itself, for the heads of its kv head only (every kv head's blocks read all heads' exponentials; a step of few rows has few of
// them), so no mixed weights are written and read.
template <bool FUSED>
__global__ void __launch_bounds__(128) values_deep_kernel(const Params p) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __shared__ int s_last;
  constexpr int WK = 32;
  pdl_wait();
  const int r = blockIdx.z, hk = blockIdx.x, split = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3;
  const int q0 = p.cu_q[r], qn = p.cu_q[r + 1] - q0, M = qn * p.per;
  if (M <= 0 || M > 16 || q0 + qn <= p.t_lo || q0 >= p.t_hi) return;
  const int p0 = p.kv_len[r] - qn;
  const int lo = first_key(p, p0), hi = p0 + qn, kt0 = lo & ~(BN - 1);
  const int* bt = p.block_table + (size_t)r * p.bt_width;
  bf16* V = reinterpret_cast<bf16*>(smem_raw) + warp * WK * LDS;
  const bf16 *ws = (const bf16*)p.w, *vc = (const bf16*)p.vc;
  size_t row[2];
  int pos[2], base[2];
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int m = g + 8 * half, tok = m / p.per, t = q0 + tok;
    const bool ok = m < M && t >= p.t_lo && t < p.t_hi;
    pos[half] = ok ? p0 + tok : -1;
    row[half] = ok ? (size_t)(t - p.t_lo) * p.H + hk * p.per + (m - tok * p.per) : 0;
    base[half] = ok ? first_key(p, pos[half]) & ~(BN - 1) : 0;
  }
  // FUSED: a strip's keys come out of the mix in the order 4 n + q (product tile q, column n): the value rows are laid out likewise
  auto fetch = [&](int kt) {
    const int key = kt + lane;
    const long long mine = (key >= lo && key < hi) ? cache_row(p, bt, hk, key) : -1;
#pragma unroll
    for (int idx0 = 0; idx0 < WK * CHUNKS; idx0 += 32) {
      const int idx = idx0 + lane, vrow = idx / CHUNKS, ch = idx - vrow * CHUNKS;
      const long long off = __shfl_sync(0xffffffffu, mine, vrow);
      const int at = FUSED ? ((vrow & 3) << 3) + (vrow >> 2) : vrow;
      cp_async16(V + at * LDS + ch * 8, vc + (off >= 0 ? off + ch * 8 : 0), off >= 0);
    }
    cp_async_commit();
  };
  const int step = p.n_splits * 4 * WK;
  int kt = kt0 + (split * 4 + warp) * WK;
  if (kt < hi) fetch(kt);
  float *M_s = reinterpret_cast<float*>(smem_raw + DEEP_BYTES), *inv_s = M_s + 16 * p.G;      // [token][H]
  if (FUSED) {
    for (int i = 0; i < qn; ++i) {
      const int t = q0 + i;
      if (t < p.t_lo || t >= p.t_hi) continue;
      token_softmax(p, t - p.t_lo, (p0 + i - (first_key(p, p0 + i) & ~(BN - 1))) / BN + 1, M_s + i * p.H, inv_s + i * p.H);
    }
  }
  float o[D / 8][4];
#pragma unroll
  for (int i = 0; i < D / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  for (bool fetched = true; kt < hi; kt += step, fetched = false) {
    if (!fetched) fetch(kt);
    uint32_t wf[WK / 16][4];
    if (FUSED) {
      float acc[4][4];
#pragma unroll
      for (int n = 0; n < 4; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
      const int kt_n = (p.H + 15) / 16, hp = kt_n * 16;
      const uint32_t* talk = reinterpret_cast<const uint32_t*>(p.talk);
      const int m_a = g, m_b = g + 8, tok_a = m_a / p.per, tok_b = m_b / p.per;
      for (int i = 0; i < qn; ++i) {
        // this token's rows of the product's first operand, the others' are zero: the sum over the tokens holds every row
        const int t = q0 + i, at_pos = p0 + i, at_base = first_key(p, at_pos) & ~(BN - 1);
        if (t < p.t_lo || t >= p.t_hi || kt < at_base || (kt & ~(BN - 1)) > at_pos) continue;
        const size_t row0 = (size_t)(t - p.t_lo) * p.H;
        const bool use_a = m_a < M && tok_a == i, use_b = m_b < M && tok_b == i;
        const uint32_t* ta = talk + (size_t)(use_a ? hk * p.per + (m_a - tok_a * p.per) : 0) * (hp / 2) + tq;
        const uint32_t* tb = talk + (size_t)(use_b ? hk * p.per + (m_b - tok_b * p.per) : 0) * (hp / 2) + tq;
        for (int kk = 0; kk < kt_n; ++kk) {
          float4 ev[4];
          float f[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const int h = kk * 16 + 2 * tq + (j & 1) + ((j >> 1) << 3);
            ev[j] = h < p.H ? *reinterpret_cast<const float4*>(p.e + (row0 + h) * p.pitch + (kt - at_base) + g * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
            f[j] = h < p.H ? inv_s[i * p.H + h] : 0.f;
            if (!p.fixed && h < p.H) f[j] *= ex2(p.stats[(row0 + h) * (p.pitch / BN) + (kt - at_base) / BN].x - M_s[i * p.H + h]);
          }
          const uint32_t a0 = use_a ? __ldg(ta + kk * 8) : 0u, a2 = use_a ? __ldg(ta + kk * 8 + 4) : 0u;
          const uint32_t a1 = use_b ? __ldg(tb + kk * 8) : 0u, a3 = use_b ? __ldg(tb + kk * 8 + 4) : 0u;
          uint32_t hi2[4][2], lo2[4][2];
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const float4 a = ev[2 * j], b = ev[2 * j + 1];
            const float xs[4] = {a.x * f[2 * j], a.y * f[2 * j], a.z * f[2 * j], a.w * f[2 * j]};
            const float ys[4] = {b.x * f[2 * j + 1], b.y * f[2 * j + 1], b.z * f[2 * j + 1], b.w * f[2 * j + 1]};
#pragma unroll
            for (int n = 0; n < 4; ++n) {
              const __nv_bfloat162 h2 = __floats2bfloat162_rn(xs[n], ys[n]);
              hi2[n][j] = *reinterpret_cast<const uint32_t*>(&h2);
              lo2[n][j] = pack_bf16(xs[n] - __low2float(h2), ys[n] - __high2float(h2));
            }
          }
#pragma unroll
          for (int n = 0; n < 4; ++n) {
            mma_bf16(acc[n], a0, a1, a2, a3, lo2[n][0], lo2[n][1]);
            mma_bf16(acc[n], a0, a1, a2, a3, hi2[n][0], hi2[n][1]);
          }
        }
      }
#pragma unroll
      for (int kk = 0; kk < WK / 16; ++kk) {
        wf[kk][0] = pack_bf16(acc[2 * kk][0], acc[2 * kk][1]);
        wf[kk][1] = pack_bf16(acc[2 * kk][2], acc[2 * kk][3]);
        wf[kk][2] = pack_bf16(acc[2 * kk + 1][0], acc[2 * kk + 1][1]);
        wf[kk][3] = pack_bf16(acc[2 * kk + 1][2], acc[2 * kk + 1][3]);
      }
    } else {
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const bool ok = pos[half] >= 0 && kt >= base[half] && (kt & ~(BN - 1)) <= pos[half];
        const bf16* src = ws + row[half] * p.pitch + (kt - base[half]) + tq * 2;
#pragma unroll
        for (int kk = 0; kk < WK / 16; ++kk) {
          wf[kk][half] = ok ? *reinterpret_cast<const uint32_t*>(src + kk * 16) : 0u;
          wf[kk][2 + half] = ok ? *reinterpret_cast<const uint32_t*>(src + kk * 16 + 8) : 0u;
        }
      }
    }
    cp_async_wait<0>();
    __syncwarp();
#pragma unroll
    for (int kk = 0; kk < WK / 16; ++kk)
#pragma unroll
      for (int d = 0; d < D / 16; ++d) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(b0, b1, b2, b3, V + (kk * 16 + (lane & 15)) * LDS + d * 16 + (lane >> 4) * 8);
        mma_bf16(o[2 * d], wf[kk][0], wf[kk][1], wf[kk][2], wf[kk][3], b0, b1);
        mma_bf16(o[2 * d + 1], wf[kk][0], wf[kk][1], wf[kk][2], wf[kk][3], b2, b3);
      }
    __syncwarp();
  }
  __syncthreads();
  float* sums = reinterpret_cast<float*>(smem_raw);           // [4][16][D + 2] over the value tiles
  constexpr int LDO = D + 2;
#pragma unroll
  for (int half = 0; half < 2; ++half)
#pragma unroll
    for (int i = 0; i < D / 8; ++i) {
      float* dst = sums + (warp * 16 + g + 8 * half) * LDO + i * 8 + tq * 2;
      dst[0] = o[i][2 * half];
      dst[1] = o[i][2 * half + 1];
    }
  __syncthreads();
  float* part = p.n_splits > 1 ? p.part + (((size_t)r * p.G + hk) * p.n_splits + split) * 16 * D : nullptr;
  auto store = [&](int m, int d, float v) {
    const int tok = m / p.per, t = q0 + tok;
    if (t >= p.t_lo && t < p.t_hi) ((bf16*)p.out)[((size_t)t * p.H + hk * p.per + (m - tok * p.per)) * D + d] = __float2bfloat16_rn(v);
  };
  for (int idx = tid; idx < M * D; idx += 128) {
    const int m = idx / D, d = idx - m * D;
    const float v = (sums[m * LDO + d] + sums[(16 + m) * LDO + d]) + (sums[(32 + m) * LDO + d] + sums[(48 + m) * LDO + d]);
    if (part) part[idx] = v;
    else store(m, d, v);
  }
  pdl_launch_dependents();
  if (!part) return;
  __threadfence();
  __syncthreads();
  if (tid == 0) s_last = atomicAdd(p.tickets + (size_t)r * p.G + hk, 1) == p.n_splits - 1;
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  const float* all = p.part + ((size_t)r * p.G + hk) * p.n_splits * 16 * D;
  for (int idx = tid; idx < M * D; idx += 128) {
    float v = 0.f;
    for (int s = 0; s < p.n_splits; ++s) v += __ldcg(all + (size_t)s * 16 * D + idx);
    store(idx / D, idx % D, v);
  }
  if (tid == 0) p.tickets[(size_t)r * p.G + hk] = 0;
}

// ------------------------------------------------------------------------------------------------------- float32
// One shape for all requests: tiles of 16 rows, 256 threads (row = tid / 16), all products plain fused multiply-adds.
constexpr int LDF = D + 4;
struct RowTile32 {
  WideTile w;
  size_t row;
  int pos, first, base;
};
__device__ __forceinline__ bool row_tile32(const Params& p, RowTile32& x) {
  if (!wide_tile<16>(p, x.w)) return false;
  row_of(p, x.w, x.w.m0 + (threadIdx.x >> 4), x.row, x.pos);
  x.first = x.pos >= 0 ? first_key(p, x.pos) : 0;
  x.base = x.first & ~(BN - 1);
  return true;
}
__device__ __forceinline__ void load_tile32(const Params& p, const float* cache, const WideTile& w, int kt, float* dst) {
  for (int idx = threadIdx.x; idx < BN * (D / 4); idx += 256) {
    const int row = idx / (D / 4), c = (idx - row * (D / 4)) * 4, key = kt + row;
    const long long off = (key >= w.lo && key < w.hi) ? cache_row(p, w.bt, w.hk, key) : -1;
    *reinterpret_cast<float4*>(dst + row * LDF + c) = off >= 0 ? *reinterpret_cast<const float4*>(cache + off + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
}

__global__ void __launch_bounds__(256) scores_f32_kernel(const Params p) {
  extern __shared__ __align__(16) float sm[];
  float *Qs = sm, *Ks = sm + 16 * LDF;
  RowTile32 x;
  if (!row_tile32(p, x)) return;
  const int tid = threadIdx.x, rr = tid >> 4, c = tid & 15;
  for (int idx = tid; idx < 16 * (D / 4); idx += 256) {
    const int row = idx / (D / 4), k = (idx - row * (D / 4)) * 4, m = x.w.m0 + row, tok = m / p.per;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (m < x.w.M) v = *reinterpret_cast<const float4*>((const float*)p.q + (size_t)(x.w.q0 + tok) * p.q_stride + (size_t)(x.w.hk * p.per + m - tok * p.per) * D + k);
    *reinterpret_cast<float4*>(Qs + row * LDF + k) = v;
  }
  for (int kt = x.w.lo & ~(BN - 1); kt < x.w.hi; kt += BN) {
    __syncthreads();
    load_tile32(p, (const float*)p.kc, x.w, kt, Ks);
    __syncthreads();
    float s[4] = {0.f, 0.f, 0.f, 0.f};
    for (int k = 0; k < D; k += 4) {
      const float4 a = *reinterpret_cast<const float4*>(Qs + rr * LDF + k);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float4 b = *reinterpret_cast<const float4*>(Ks + (c + 16 * i) * LDF + k);
        s[i] = fmaf(a.x, b.x, s[i]); s[i] = fmaf(a.y, b.y, s[i]); s[i] = fmaf(a.z, b.z, s[i]); s[i] = fmaf(a.w, b.w, s[i]);
      }
    }
    float m = -INFINITY;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int key = kt + c + 16 * i;
      float v = p.cap > 0.f ? p.cap * tanhf(s[i] * p.cap_in) : s[i] * p.scale;
      s[i] = (key >= x.first && key <= x.pos) ? v * LOG2E : -INFINITY;
      m = fmaxf(m, s[i]);
    }
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
    const bool live = x.pos >= 0 && kt >= x.base && kt <= x.pos;
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float v = live ? exp2f(s[i] - m) : 0.f;
      sum += v;
      if (live) p.e[x.row * p.pitch + (kt - x.base) + c + 16 * i] = v;
    }
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    if (live && c == 0) p.stats[x.row * (p.pitch / BN) + (kt - x.base) / BN] = make_float2(m, sum);
  }
}

__global__ void __launch_bounds__(256) values_f32_kernel(const Params p) {
  extern __shared__ __align__(16) float sm[];
  float *Ws = sm, *Vs = sm + 16 * LDW;
  RowTile32 x;
  if (!row_tile32(p, x)) return;
  const int tid = threadIdx.x, rr = tid >> 4, c = tid & 15;
  float o[D / 16];
#pragma unroll
  for (int i = 0; i < D / 16; ++i) o[i] = 0.f;
  const float* w = (const float*)p.w;
  for (int kt = x.w.lo & ~(BN - 1); kt < x.w.hi; kt += BN) {
    __syncthreads();
    load_tile32(p, (const float*)p.vc, x.w, kt, Vs);
    const bool live = x.pos >= 0 && kt >= x.base && kt <= x.pos;
#pragma unroll
    for (int i = 0; i < 4; ++i) Ws[rr * LDW + c + 16 * i] = live ? w[x.row * p.pitch + (kt - x.base) + c + 16 * i] : 0.f;
    __syncthreads();
    for (int j = 0; j < BN; ++j) {
      const float a = Ws[rr * LDW + j];
#pragma unroll
      for (int i = 0; i < D / 16; ++i) o[i] = fmaf(a, Vs[j * LDF + c + 16 * i], o[i]);
    }
  }
  if (x.pos < 0) return;
  float* dst = (float*)p.out + ((size_t)p.t_lo * p.H + x.row) * D + c;
#pragma unroll
  for (int i = 0; i < D / 16; ++i) dst[16 * i] = o[i];
}

template <typename K> int allow_smem(K k, size_t bytes) {
  if (bytes > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
    if (e != cudaSuccess) return (int)e;
  }
  return 0;
}

}  // namespace

// Attention with mixed heads for tokens [t_lo, t_hi) of a step. q [T, >= H * D] (row stride given), cache tensors
// [pages, G, ps, D], block_table [R, bt_width], cu_q [R + 1], kv_len [R], positions [T]; talk as in Params; e, stats, w the scratch
// buffers for t_hi - t_lo tokens of ``pitch`` keys (a multiple of 64 no shorter than what any of them reads, counted from its base);
// out [T, H * D]. which: bit 0 wide requests, bit 1 deep ones (float32 has one shape). wide_rows [n_wide] or null (all R).
// n_splits > 1: part [R, G, n_splits, 16, D] floats and tickets [R, G], zero before and after. max_keys: the most keys (from its
// base) a token of the launch reads, max_q the most tokens a request brings: they size grids only. use_tc: wide requests may run on
// tcgen05 (q has n_tokens rows; *error is raised if a bounded wait runs out).
SB_EXPORT int sb_talking_attention(const void* q, int q_stride, const void* kc, const void* vc, const int* block_table, int bt_width,
                                   const int* cu_q, const int* kv_len, const int* positions, int H, int G, int ps, int num_pages, float scale,
                                   float softcap, int chunk, const float* sinks, const void* talk, float* e, void* stats, void* w, int pitch,
                                   int t_lo, int t_hi, void* out, int R, int max_q, int max_keys, int which, const int* wide_rows, int n_wide,
                                   int n_splits, float* part, int* tickets, int n_tokens, int* error, int use_tc, int dtype,
                                   cudaStream_t stream) {
  const int n_tok = t_hi - t_lo;
  if (n_tok <= 0 || R <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || ps <= 0 || bt_width <= 0 || pitch <= 0 || pitch % BN || max_keys > pitch || q_stride < H * D || !talk || !e ||
      !stats || !w || n_splits < 1 || chunk < 0)
    return SB_ERR_SHAPE;
  if (!aligned16(q) || !aligned16(kc) || !aligned16(vc) || !aligned16(e) || !aligned16(w) || !aligned16(out) || q_stride % 8) return SB_ERR_ALIGN;
  if (n_splits > 1 && (!part || !tickets)) return SB_ERR_SHAPE;
  Params p;
  p.q = q; p.q_stride = q_stride; p.kc = kc; p.vc = vc; p.block_table = block_table; p.bt_width = bt_width;
  p.cu_q = cu_q; p.kv_len = kv_len; p.positions = positions;
  p.H = H; p.G = G; p.per = H / G; p.ps = ps; p.num_pages = num_pages;
  p.ps_shift = -1;
  for (int s = 0; s < 30; ++s) if ((1 << s) == ps) p.ps_shift = s;
  p.scale = scale; p.cap = softcap > 0.f ? softcap : 0.f; p.cap_in = softcap > 0.f ? scale / softcap : 0.f;
  p.fixed = softcap > 0.f && softcap <= FIXED_CAP && dtype == SB_DTYPE_BF16;
  p.zero_ahead = 0;
  p.chunk = chunk; p.sinks = sinks; p.talk = talk; p.e = e; p.stats = (float2*)stats; p.w = w; p.pitch = pitch; p.t_lo = t_lo; p.t_hi = t_hi;
  p.out = out; p.wide_rows = wide_rows; p.deep_on = (which & 2) != 0; p.n_splits = n_splits; p.part = part; p.tickets = tickets;
  const int max_tiles = (max_keys + BN - 1) / BN;
  const int mix_smem = 2 * H * (int)sizeof(float);
  if (H > 1024 || G > 65535 || R > 65535) return SB_ERR_LIMIT;
  if (dtype == SB_DTYPE_F32) {
    p.deep_on = 0;
    p.wide_rows = nullptr;
    const dim3 grid(G, (unsigned)((max_q * p.per + 15) / 16), R);
    const size_t smem_s = (size_t)(16 + BN) * LDF * sizeof(float), smem_v = ((size_t)16 * LDW + (size_t)BN * LDF) * sizeof(float);
    if (int rc = allow_smem(scores_f32_kernel, smem_s)) return rc;
    if (int rc = allow_smem(values_f32_kernel, smem_v)) return rc;
    scores_f32_kernel<<<grid, 256, smem_s, stream>>>(p);
    SB_LAUNCH_CHECK();
    mix_f32_kernel<<<dim3(n_tok, (unsigned)min(max_tiles, 1024)), 256, mix_smem, stream>>>(p);
    SB_LAUNCH_CHECK();
    values_f32_kernel<<<grid, 256, smem_v, stream>>>(p);
    SB_LAUNCH_CHECK();
    return 0;
  }
  if (dtype != SB_DTYPE_BF16) return SB_ERR_DTYPE;
  constexpr int NW = 4;
  const int nz = wide_rows ? n_wide : R;
  const bool wide = (which & 1) && nz > 0, deep = (which & 2) != 0;
  const dim3 wgrid(G, (unsigned)((max_q * p.per + 16 * NW - 1) / (16 * NW)), (unsigned)max(nz, 1));
  const bool tc = wide && use_tc && error && tc_takes(H, G, ps, q_stride, chunk);
  if (tc) {
    p.zero_ahead = tc_tokens_per_tile(H, G) - 1;
    if (int rc = tc_scores(p, n_tokens, max_keys, max_q, nz, error, stream)) return rc;
  } else if (wide) {
    const size_t smem = (size_t)(16 * NW + 2 * BN) * LDS * sizeof(bf16);
    if (int rc = allow_smem(scores_wide_kernel<NW>, smem)) return rc;
    SB_PDL_CHECK(launch_pdl(scores_wide_kernel<NW>, wgrid, dim3(NW * 32), smem, stream, p));
  }
  if (deep) SB_PDL_CHECK(launch_pdl(scores_deep_kernel, dim3(G, (unsigned)((max_tiles + 3) / 4), R), dim3(128), 0, stream, p));
  // (with more (request, kv head) pairs than SMs, every pair mixing for itself costs more than the launch it saves)
  const bool fused = !wide && R * G <= sm_count();
  if (!fused) {
    // few tokens: tiles go to blocks of their own; many: a block walks its token's tiles
    const int want = (4 * sm_count() + n_tok - 1) / n_tok, have = (max_tiles + 3) / 4;
    const dim3 grid(n_tok, (unsigned)max(1, min(want, have)));
    if (H <= 16) SB_PDL_CHECK(launch_pdl(mix_kernel<1>, grid, dim3(128), mix_smem, stream, p));
    else if (H <= 32) SB_PDL_CHECK(launch_pdl(mix_kernel<2>, grid, dim3(128), mix_smem, stream, p));
    else SB_PDL_CHECK(launch_pdl(mix_kernel<4>, grid, dim3(128), mix_smem, stream, p));
  }
  if (tc) {
    if (int rc = tc_values(p, max_q, nz, error, stream)) return rc;
  } else if (wide) {
    const size_t smem = (size_t)2 * (16 * NW * LDW + BN * LDS) * sizeof(bf16);
    if (int rc = allow_smem(values_wide_kernel<NW>, smem)) return rc;
    SB_PDL_CHECK(launch_pdl(values_wide_kernel<NW>, wgrid, dim3(NW * 32), smem, stream, p));
  }
  if (deep) {
    const size_t smem = DEEP_BYTES + (!fused ? 0 : (size_t)2 * 16 * G * sizeof(float));      // (a request's tokens times H: at most 16 G)
    if (smem > 200 * 1024) return SB_ERR_LIMIT;
    const dim3 grid(G, (unsigned)n_splits, R);
    if (!fused) {
      if (int rc = allow_smem(values_deep_kernel<false>, smem)) return rc;
      SB_PDL_CHECK(launch_pdl(values_deep_kernel<false>, grid, dim3(128), smem, stream, p));
    } else {
      if (int rc = allow_smem(values_deep_kernel<true>, smem)) return rc;
      SB_PDL_CHECK(launch_pdl(values_deep_kernel<true>, grid, dim3(128), smem, stream, p));
    }
  }
  return 0;
}
