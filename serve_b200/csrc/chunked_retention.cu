// The linear recurrence with one fixed decay d per head, S_t = d S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, for prompt portions in
// bfloat16: chunk by chunk on the tensor cores instead of token by token. With c the chunk's tokens 0 .. n-1 and S the state
// before it,
//   o_i = d^(i+1) S^T q_i + sum_{j <= i} d^(i-j) (q_i . k_j) v_j,        S' = d^n S + sum_j d^(n-1-j) k_j v_j^T.
// Three kernels: (1) the chunks' own sums of k v^T, all chunks at once; (2) a walk over a request's chunks that replaces every
// chunk's sum by the state before it and leaves the last state in the request's slot (element by element, so it is a stream of
// loads and stores); (3) the outputs, all chunks at once. q and k are rotated and k scaled on the way into shared memory.
// What enters the recurrence counts as 32-bit: every float operand x of a product is split into two bfloat16 numbers hi + lo
// (x to 2^-17), products run hi hi + lo hi + hi lo into float sums; v is a projection and bfloat16 as it is.
// Rows (requests) with at most ``min_tokens`` tokens are left to the walking kernel (sequence_ops.cu). Chunks count from a
// portion's first token.
#include "common.cuh"

using namespace sb;
typedef __nv_bfloat16 bf16;

namespace {

constexpr int CH = 64;             // tokens of a chunk
constexpr int VT = 64;             // value columns a group of four warps takes

struct ChunkArgs {
  const bf16 *q, *k, *v;           // [T, *], head h at h * dk (h * dv)
  int qs, ks, vs;                  // row strides
  const float2* angles; int half;  // [T, half] cosine and sine of a token's angles; pairs (i, i + half), i < half
  float k_scale;
  const float* decay;              // [H]
  float* state; long long state_stride;
  const int *slots, *cu_q, *rows;  // rows: the requests by falling number of tokens, or null: all of them in order
  float* out; int out_stride;      // [T, H * dv]
  float* sums;                     // [chunks, H, dk, dv]: first the chunks' sums, then the states before them
  int H, dk, dv, min_tokens;
};

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((unsigned)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((unsigned)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// x, y -> their two bfloat16 halves, packed (x in the low half)
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float4 load4(const bf16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&u.x), b = *reinterpret_cast<const __nv_bfloat162*>(&u.y);
  return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
}
__device__ __forceinline__ void split4(float4 x, bf16* hi, bf16* lo) {
  uint2 h, l;
  split2(x.x, x.y, h.x, l.x);
  split2(x.z, x.w, h.y, l.y);
  *reinterpret_cast<uint2*>(hi) = h;
  *reinterpret_cast<uint2*>(lo) = l;
}

// Where a block's chunk lies: false if there is none. The chunks of the rows before this one in the list are counted by the block.
struct Place { int row, t0, n, chunk, n_chunks; long long slot; };
__device__ __forceinline__ bool find_chunk(const ChunkArgs& a, int i, int c, Place& p, int* red) {
  const int r = a.rows ? a.rows[i] : i;
  const int q0 = a.cu_q[r], n = a.cu_q[r + 1] - q0;
  if (n <= a.min_tokens || c * CH >= n) return false;          // (the whole block)
  int before = 0;
  for (int u = threadIdx.x; u < i; u += blockDim.x) {
    const int ru = a.rows ? a.rows[u] : u;
    const int nu = a.cu_q[ru + 1] - a.cu_q[ru];
    if (nu > a.min_tokens) before += (nu + CH - 1) / CH;
  }
  if (i > 0) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) before += __shfl_xor_sync(0xffffffffu, before, o);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = before;
    __syncthreads();
    before = 0;
    for (int u = 0; u < (int)(blockDim.x >> 5); ++u) before += red[u];
  }
  p.row = r;
  p.t0 = q0 + c * CH;
  p.n = min(CH, n - c * CH);
  p.chunk = c;
  p.n_chunks = (n + CH - 1) / CH;
  p.slot = before;
  return true;
}

// The chunk's rows of q or k of one head, rotated and times ``factor[token]`` * scale, into hi and lo [CH][PITCH] (rows beyond n and
// columns beyond dk are zero). factor null: 1.
template <int DKT, int PITCH>
__device__ __forceinline__ void load_rotated(const bf16* src, int stride, const ChunkArgs& a, const Place& p, float scale, const float* factor,
                                             bf16* hi, bf16* lo) {
  const int hg = a.half >> 2;                      // groups of four pairs
  const int plain0 = a.half >> 1;                  // the first group of four that is not rotated (2 half / 4)
  const int per_row = hg + (DKT / 4 - plain0);
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
  for (int w = threadIdx.x; w < CH * per_row; w += blockDim.x) {
    const int t = w / per_row, g = w - t * per_row;
    const bool live = t < p.n;
    const bf16* row = src + (size_t)(p.t0 + t) * stride;
    const float f = live ? scale * (factor ? factor[t] : 1.f) : 0.f;
    if (g < hg) {
      float4 u = zero, v = zero, x, y;
      float4 cs0 = zero, cs1 = zero;               // c0 s0 c1 s1, c2 s2 c3 s3
      if (live) {
        u = load4(row + g * 4);
        v = load4(row + a.half + g * 4);
        const float4* an = reinterpret_cast<const float4*>(a.angles + (size_t)(p.t0 + t) * a.half + g * 4);
        cs0 = an[0];
        cs1 = an[1];
      }
      x = make_float4((u.x * cs0.x - v.x * cs0.y) * f, (u.y * cs0.z - v.y * cs0.w) * f, (u.z * cs1.x - v.z * cs1.y) * f, (u.w * cs1.z - v.w * cs1.w) * f);
      y = make_float4((v.x * cs0.x + u.x * cs0.y) * f, (v.y * cs0.z + u.y * cs0.w) * f, (v.z * cs1.x + u.z * cs1.y) * f, (v.w * cs1.z + u.w * cs1.w) * f);
      split4(x, hi + t * PITCH + g * 4, lo + t * PITCH + g * 4);
      split4(y, hi + t * PITCH + a.half + g * 4, lo + t * PITCH + a.half + g * 4);
    } else {
      const int c = (plain0 + g - hg) * 4;
      float4 x = zero;
      if (live && c < a.dk) x = load4(row + c);
      split4(make_float4(x.x * f, x.y * f, x.z * f, x.w * f), hi + t * PITCH + c, lo + t * PITCH + c);
    }
  }
}

// The chunk's rows of v of one head, columns j0 .. j0 + COLS - 1, into [CH][PITCH] (zero beyond n and dv).
template <int COLS, int PITCH>
__device__ __forceinline__ void load_values(const bf16* src, const ChunkArgs& a, const Place& p, int j0, bf16* dst) {
#pragma unroll 4
  for (int w = threadIdx.x; w < CH * (COLS / 4); w += blockDim.x) {
    const int t = w / (COLS / 4), c = (w - t * (COLS / 4)) * 4;
    uint2 x = make_uint2(0, 0);
    if (t < p.n && j0 + c < a.dv) x = *reinterpret_cast<const uint2*>(src + (size_t)(p.t0 + t) * a.vs + j0 + c);
    *reinterpret_cast<uint2*>(dst + t * PITCH + c) = x;
  }
}

// ---------------------------------------------------------------------------------------------- (1) a chunk's sum of k v^T
// grid (chunk, value tile, head + H * list entry); 256 threads. Eight warps over DKT / 16 row tiles and 8 / (DKT / 16) column groups.
template <int DKT>
__global__ void __launch_bounds__(256) chunk_sums_kernel(const ChunkArgs a) {
  constexpr int KP = DKT + 8, VP = VT + 8, MT = DKT / 16, NG = 8 / MT, NC = VT / NG;      // NC columns a warp
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ int red[8];
  __shared__ float factor[CH];
  bf16 *kh = reinterpret_cast<bf16*>(raw), *kl = kh + CH * KP, *vv = kl + CH * KP;
  const int i = blockIdx.z / a.H, h = blockIdx.z - i * a.H, j0 = blockIdx.y * VT;
  Place p;
  if (!find_chunk(a, i, blockIdx.x, p, red)) return;
  if (threadIdx.x < CH) factor[threadIdx.x] = (int)threadIdx.x < p.n ? powf(a.decay[h], (float)(p.n - 1 - (int)threadIdx.x)) : 0.f;
  __syncthreads();
  load_rotated<DKT, KP>(a.k + (size_t)h * a.dk, a.ks, a, p, a.k_scale, factor, kh, kl);
  load_values<VT, VP>(a.v + (size_t)h * a.dv, a, p, j0, vv);
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int m0 = (warp % MT) * 16, n0 = (warp / MT) * NC;
  float acc[NC / 8][4] = {};
#pragma unroll
  for (int kk = 0; kk < CH; kk += 16) {
    // k is stored token by token, so the product's left operand (rows = elements of k) is read transposed
    uint32_t ah[4], al[4];
    const int ar = (kk + (lane >> 4) * 8 + (lane & 7)) * KP + m0 + ((lane >> 3) & 1) * 8;
    ldsm4_t(ah, kh + ar);
    ldsm4_t(al, kl + ar);
#pragma unroll
    for (int nt = 0; nt < NC; nt += 16) {
      uint32_t b[4];
      ldsm4_t(b, vv + (kk + ((lane >> 3) & 1) * 8 + (lane & 7)) * VP + n0 + nt + (lane >> 4) * 8);
      mma(acc[nt / 8], ah, b[0], b[1]);
      mma(acc[nt / 8 + 1], ah, b[2], b[3]);
      mma(acc[nt / 8], al, b[0], b[1]);
      mma(acc[nt / 8 + 1], al, b[2], b[3]);
    }
  }
  float* dst = a.sums + ((p.slot + p.chunk) * a.H + h) * a.dk * a.dv;
  const int g = lane >> 2, c2 = (lane & 3) * 2;
#pragma unroll
  for (int nt = 0; nt < NC / 8; ++nt) {
    const int j = j0 + n0 + nt * 8 + c2, m = m0 + g;
    if (j < a.dv) {                                  // (dv is a multiple of four)
      if (m < a.dk) *reinterpret_cast<float2*>(dst + (size_t)m * a.dv + j) = make_float2(acc[nt][0], acc[nt][1]);
      if (m + 8 < a.dk) *reinterpret_cast<float2*>(dst + (size_t)(m + 8) * a.dv + j) = make_float2(acc[nt][2], acc[nt][3]);
    }
  }
}

// ---------------------------------------------------------------------------------------------- (2) the states before the chunks
// grid (ceil(dk dv / 2 / 256), H, list entries). A thread takes two neighbouring elements of the state through all chunks.
__global__ void __launch_bounds__(256) chunk_states_kernel(const ChunkArgs a) {
  __shared__ int red[8];
  Place p;
  if (!find_chunk(a, blockIdx.z, 0, p, red)) return;
  const int h = blockIdx.y, e = (blockIdx.x * 256 + threadIdx.x) * 2, per = a.dk * a.dv;
  if (e >= per) return;
  const int n = a.cu_q[p.row + 1] - a.cu_q[p.row];
  const float full = powf(a.decay[h], (float)CH), last = powf(a.decay[h], (float)(n - (p.n_chunks - 1) * CH));
  float2* st = reinterpret_cast<float2*>(a.state + (size_t)a.slots[p.row] * a.state_stride + (size_t)h * per + e);
  float* at = a.sums + (p.slot * a.H + h) * per + e;
  const size_t step = (size_t)a.H * per;
  float2 s = *st;
  constexpr int AHEAD = 16;
  for (int c0 = 0; c0 < p.n_chunks; c0 += AHEAD) {
    float2 x[AHEAD];
#pragma unroll
    for (int u = 0; u < AHEAD; ++u)
      if (c0 + u < p.n_chunks) x[u] = *reinterpret_cast<const float2*>(at + (size_t)(c0 + u) * step);
#pragma unroll
    for (int u = 0; u < AHEAD; ++u)
      if (c0 + u < p.n_chunks) {
        *reinterpret_cast<float2*>(at + (size_t)(c0 + u) * step) = s;
        const float d = c0 + u + 1 < p.n_chunks ? full : last;
        s.x = s.x * d + x[u].x; s.y = s.y * d + x[u].y;
      }
  }
  *st = s;
}

// ---------------------------------------------------------------------------------------------- (3) the outputs
// Elements of shared memory the keys and, after them, a part of the state take (both halves; vp: pitch of the state's rows).
__host__ __device__ constexpr int out_shared(int dkt, int vp) {
  return 2 * CH * (dkt + 8) > 2 * (dkt < 64 ? dkt : 64) * vp ? 2 * CH * (dkt + 8) : 2 * (dkt < 64 ? dkt : 64) * vp;
}
// grid (chunk, value tile of CG * 64, head + H * list entry); CG groups of four warps, a group 64 value columns, a warp 16 tokens.
// The state before the chunk comes in parts of at most 64 rows, into the place the keys have left: two blocks fit an SM.
template <int DKT, int CG>
__global__ void __launch_bounds__(128 * CG, 2) chunk_out_kernel(const ChunkArgs a) {
  constexpr int KP = DKT + 8, VC = CG * VT, VP = VC + 8, SR = DKT < 64 ? DKT : 64;
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ int red[8];
  __shared__ float pw[CH + 1];                       // powers of the decay
  bf16 *qh = reinterpret_cast<bf16*>(raw), *ql = qh + CH * KP, *kh = ql + CH * KP, *kl = kh + CH * KP, *vv = qh + 2 * CH * KP + out_shared(DKT, VP);
  bf16 *sh = kh, *sl = sh + SR * VP;
  const int i = blockIdx.z / a.H, h = blockIdx.z - i * a.H, j0 = blockIdx.y * VC;
  Place p;
  if (!find_chunk(a, i, blockIdx.x, p, red)) return;
  if (threadIdx.x <= CH) pw[threadIdx.x] = powf(a.decay[h], (float)threadIdx.x);
  load_rotated<DKT, KP>(a.q + (size_t)h * a.dk, a.qs, a, p, 1.f, nullptr, qh, ql);
  load_rotated<DKT, KP>(a.k + (size_t)h * a.dk, a.ks, a, p, a.k_scale, nullptr, kh, kl);
  load_values<VC, VP>(a.v + (size_t)h * a.dv, a, p, j0, vv);
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int i0 = (warp & 3) * 16, n0 = (warp >> 2) * VT;
  const bool live = i0 < p.n && j0 + n0 < a.dv;      // (a whole warp)
  const int g = lane >> 2, c2 = (lane & 3) * 2;
  const int a_off = (i0 + (lane & 15)) * KP + (lane >> 4) * 8;                                   // left operand, row-major
  const int bt_row = ((lane >> 3) & 1) * 8 + (lane & 7), bt_col = (lane >> 4) * 8;               // right operand stored k by n
  float s[CH / 8][4] = {}, o[VT / 8][4] = {};
  if (live) {
#pragma unroll
    for (int kk = 0; kk < DKT; kk += 16) {
      uint32_t ah[4], al[4];
      ldsm4(ah, qh + a_off + kk);
      ldsm4(al, ql + a_off + kk);
#pragma unroll
      for (int nt = 0; nt < CH; nt += 16) {
        if (nt <= i0) {                              // (a whole warp: keys of the same or earlier sixteens)
          uint32_t bh[4], bl[4];
          const int b_off = (nt + (lane >> 4) * 8 + (lane & 7)) * KP + kk + ((lane >> 3) & 1) * 8;
          ldsm4(bh, kh + b_off);
          ldsm4(bl, kl + b_off);
          mma(s[nt / 8], ah, bh[0], bh[1]);
          mma(s[nt / 8 + 1], ah, bh[2], bh[3]);
          mma(s[nt / 8], al, bh[0], bh[1]);
          mma(s[nt / 8 + 1], al, bh[2], bh[3]);
          mma(s[nt / 8], ah, bl[0], bl[1]);
          mma(s[nt / 8 + 1], ah, bl[2], bl[3]);
        }
      }
    }
  }
  const float* src = a.sums + ((p.slot + p.chunk) * a.H + h) * a.dk * a.dv;
#pragma unroll 1
  for (int m0 = 0; m0 < DKT; m0 += SR) {
    __syncthreads();                                 // the keys, or the part before, are read
#pragma unroll 4
    for (int w = threadIdx.x; w < SR * (VC / 4); w += blockDim.x) {
      const int m = w / (VC / 4), c = (w - m * (VC / 4)) * 4;
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (m0 + m < a.dk && j0 + c < a.dv) x = *reinterpret_cast<const float4*>(src + (size_t)(m0 + m) * a.dv + j0 + c);
      split4(x, sh + m * VP + c, sl + m * VP + c);
    }
    __syncthreads();
    if (!live) continue;
#pragma unroll
    for (int kk = 0; kk < SR; kk += 16) {
      uint32_t ah[4], al[4];
      ldsm4(ah, qh + a_off + m0 + kk);
      ldsm4(al, ql + a_off + m0 + kk);
#pragma unroll
      for (int nt = 0; nt < VT; nt += 16) {
        uint32_t bh[4], bl[4];
        const int b_off = (kk + bt_row) * VP + n0 + nt + bt_col;
        ldsm4_t(bh, sh + b_off);
        ldsm4_t(bl, sl + b_off);
        mma(o[nt / 8], ah, bh[0], bh[1]);
        mma(o[nt / 8 + 1], ah, bh[2], bh[3]);
        mma(o[nt / 8], al, bh[0], bh[1]);
        mma(o[nt / 8 + 1], al, bh[2], bh[3]);
        mma(o[nt / 8], ah, bl[0], bl[1]);
        mma(o[nt / 8 + 1], ah, bl[2], bl[3]);
      }
    }
  }
  if (!live) return;                                 // (nothing below waits for the block)
  const float d0 = pw[i0 + g + 1], d1 = pw[i0 + g + 9];
#pragma unroll
  for (int nt = 0; nt < VT / 8; ++nt) { o[nt][0] *= d0; o[nt][1] *= d0; o[nt][2] *= d1; o[nt][3] *= d1; }
#pragma unroll
  for (int kt = 0; kt < CH; kt += 16) {
    if (kt <= i0) {
      uint32_t ph[4], pl[4];
#pragma unroll
      for (int u = 0; u < 2; ++u) {                  // keys kt + 8 u + c2, + 1; tokens i0 + g, + 8
        float (&f)[4] = s[kt / 8 + u];
        const int j = kt + 8 * u + c2, ia = i0 + g, ib = ia + 8;
        const float x0 = j <= ia ? f[0] * pw[ia - j] : 0.f, x1 = j + 1 <= ia ? f[1] * pw[ia - j - 1] : 0.f;
        const float y0 = j <= ib ? f[2] * pw[ib - j] : 0.f, y1 = j + 1 <= ib ? f[3] * pw[ib - j - 1] : 0.f;
        split2(x0, x1, ph[2 * u], pl[2 * u]);
        split2(y0, y1, ph[2 * u + 1], pl[2 * u + 1]);
      }
#pragma unroll
      for (int nt = 0; nt < VT; nt += 16) {
        uint32_t b[4];
        ldsm4_t(b, vv + (kt + bt_row) * VP + n0 + nt + bt_col);
        mma(o[nt / 8], ph, b[0], b[1]);
        mma(o[nt / 8 + 1], ph, b[2], b[3]);
        mma(o[nt / 8], pl, b[0], b[1]);
        mma(o[nt / 8 + 1], pl, b[2], b[3]);
      }
    }
  }
  float* orow = a.out + (size_t)(p.t0 + i0 + g) * a.out_stride + (size_t)h * a.dv + j0 + n0;
#pragma unroll
  for (int nt = 0; nt < VT / 8; ++nt) {
    const int j = nt * 8 + c2;
    if (j0 + n0 + j < a.dv) {
      if (i0 + g < p.n) *reinterpret_cast<float2*>(orow + j) = make_float2(o[nt][0], o[nt][1]);
      if (i0 + g + 8 < p.n) *reinterpret_cast<float2*>(orow + (size_t)8 * a.out_stride + j) = make_float2(o[nt][2], o[nt][3]);
    }
  }
}

// angles[t][i] = cosine and sine of positions[t] * inv_freq[i]
__global__ void __launch_bounds__(256) angle_table_kernel(const int* __restrict__ positions, const float* __restrict__ inv_freq, int half, int n,
                                                          float2* __restrict__ angles) {
  const int w = blockIdx.x * blockDim.x + threadIdx.x;
  if (w >= n * half) return;
  const int t = w / half;
  float s, c;
  sincosf((float)positions[t] * inv_freq[w - t * half], &s, &c);
  angles[w] = make_float2(c, s);
}

template <int DKT>
int launch_chunked(const ChunkArgs& a, int n_list, int max_q, cudaStream_t stream) {
  const int chunks = (max_q + CH - 1) / CH;
  if ((long long)n_list * a.H > 65535 || (a.dv + VT - 1) / VT > 65535) return SB_ERR_LIMIT;
  {
    constexpr int smem = (2 * CH * (DKT + 8) + CH * (VT + 8)) * (int)sizeof(bf16);
    auto k = chunk_sums_kernel<DKT>;
    if (smem > 40 * 1024) cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    k<<<dim3(chunks, (a.dv + VT - 1) / VT, n_list * a.H), 256, smem, stream>>>(a);
    SB_LAUNCH_CHECK();
  }
  chunk_states_kernel<<<dim3((a.dk * a.dv / 2 + 255) / 256, a.H, n_list), 256, 0, stream>>>(a);
  SB_LAUNCH_CHECK();
  auto out = [&](auto kernel, int cg) {
    const int vc = cg * VT, smem = (2 * CH * (DKT + 8) + out_shared(DKT, vc + 8) + CH * (vc + 8)) * (int)sizeof(bf16);
    if (smem > 40 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    kernel<<<dim3(chunks, (a.dv + vc - 1) / vc, n_list * a.H), 128 * cg, smem, stream>>>(a);
  };
  if (a.dv > VT) out(chunk_out_kernel<DKT, 2>, 2);
  else out(chunk_out_kernel<DKT, 1>, 1);
  SB_LAUNCH_CHECK();
  return 0;
}

}  // namespace

// 1: the chunked kernels take this layout (bfloat16 operands; strides in elements, the three bases 8-byte aligned).
SB_EXPORT int sb_chunked_retention_supports(int dk, int dv, int rot_dims, int q_stride, int k_stride, int v_stride) {
  return dk > 0 && dv > 0 && dk <= 128 && dk % 4 == 0 && dv % 4 == 0 && rot_dims >= 0 && rot_dims % 8 == 0 && rot_dims <= dk && q_stride % 4 == 0 &&
         k_stride % 4 == 0 && v_stride % 4 == 0;
}

// angles float [n, half, 2]: cosine and sine of positions[t] * inv_freq[i].
SB_EXPORT int sb_angle_table(const int* positions, const float* inv_freq, int half, int n, float* angles, cudaStream_t stream) {
  if (n <= 0 || half <= 0) return 0;
  if ((long long)n * half > 0x7fffff00LL) return SB_ERR_LIMIT;
  if (!positions || !inv_freq || !aligned16(angles)) return SB_ERR_ALIGN;
  angle_table_kernel<<<(unsigned)(((long long)n * half + 255) / 256), 256, 0, stream>>>(positions, inv_freq, half, n, (float2*)angles);
  SB_LAUNCH_CHECK();
  return 0;
}

// S = d_h S + k v^T, o = S^T q over the tokens of every listed row that brings more than min_tokens, in bfloat16 (q, k and v as
// projected; q and k rotated by ``angles`` [T, rot_dims / 2, 2], k times k_scale). rows: the first n_list entries of the requests by
// falling token count, or null: n_list requests in order. sums: float work space, 16-byte aligned, [chunks, H, dk, dv] with room
// for every listed row's ceil(tokens / 64) chunks. out float [T, H * dv].
SB_EXPORT int sb_chunked_retention(const void* q, int q_stride, const void* k, int k_stride, const void* v, int v_stride, const float* angles,
                                   int rot_dims, float k_scale, const float* decay, float* state, long long state_stride, const int* slots,
                                   const int* cu_q, const int* rows, int n_list, int max_q, int min_tokens, float* out, int out_stride, int H,
                                   int dk, int dv, float* sums, cudaStream_t stream) {
  if (n_list <= 0 || max_q <= min_tokens) return 0;
  if (H <= 0 || !decay || !state || !sums || !out || !cu_q || !slots || (rot_dims && !angles) || min_tokens < 0) return SB_ERR_SHAPE;
  if (!sb_chunked_retention_supports(dk, dv, rot_dims, q_stride, k_stride, v_stride)) return SB_ERR_SHAPE;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) & 7) return SB_ERR_ALIGN;
  if (!aligned16(state) || state_stride % 4 || !aligned16(sums) || (reinterpret_cast<uintptr_t>(out) & 7) || (out_stride & 1) || (angles && !aligned16(angles)))
    return SB_ERR_ALIGN;
  if (H > 65535 || n_list > 65535) return SB_ERR_LIMIT;
  const ChunkArgs a = {(const bf16*)q, (const bf16*)k, (const bf16*)v, q_stride, k_stride, v_stride, (const float2*)angles, rot_dims / 2, k_scale, decay,
                       state, state_stride, slots, cu_q, rows, out, out_stride, sums, H, dk, dv, min_tokens};
  if (dk <= 32) return launch_chunked<32>(a, n_list, max_q, stream);
  if (dk <= 64) return launch_chunked<64>(a, n_list, max_q, stream);
  return launch_chunked<128>(a, n_list, max_q, stream);
}
