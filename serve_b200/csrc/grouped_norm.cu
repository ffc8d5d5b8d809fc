// Norms over parts of a row, and an activation made of normalised powers:
//
//   sb_add_grouped_rmsnorm  the row is cut into ``groups`` equal parts, each divided by its own sqrt(mean(part^2) + eps), times a
//                           weight; fused with the residual addition before it and, if asked, with the same kind of norm on the
//                           sub-layer's output that is added: x += rms_g(a) * w'; out = rms_g(x) * w. Without a weight out is x
//                           itself (sub-layers that read the residual stream as it is)
//   sb_poly_norm            a N(z) + b N(z^2) + c N(z^3) + e, N dividing a row by its root mean square
//
// All arithmetic is float; every part of a row is independent of the others, so a block takes one (row, part). Reductions run in a
// fixed order that depends on sizes only.
#include "common.cuh"

using namespace sb;
typedef __nv_bfloat16 bf16;

namespace {

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const bf16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&u.x), b = *reinterpret_cast<const __nv_bfloat162*>(&u.y);
  return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, float4 v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<uint32_t*>(&a);
  u.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = u;
}
__device__ __forceinline__ float dot4(float4 v) { return (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w); }
__device__ __forceinline__ float4 mul4(float4 v, float f, float4 w) { return make_float4(v.x * f * w.x, v.y * f * w.y, v.z * f * w.z, v.w * f * w.w); }

struct NormArgs {
  float* x; const void* delta; const float* through; const int* rows; const float* weight; void* out;      // weight null: out = x
  int dim, part; float eps;        // row length, length of a part
};

// The part stays in registers: VPT float4 a thread of its team, a block (grid: row, part), or, WARP, a warp (short parts: the
// blocks deal the parts of all rows out to their warps). x null: out = the norm of delta.
template <typename TD, typename TO, int VPT, bool WARP>
__global__ void __launch_bounds__(512) grouped_norm_vec_kernel(const NormArgs a, int n_parts, int groups) {
  __shared__ float red[WARP ? 1 : 32];
  const int team = WARP ? blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5) : (int)blockIdx.x;
  if (team >= n_parts) { pdl_wait(); return; }                // (a whole team; a block's only team never leaves)
  const int at = WARP ? threadIdx.x & 31 : threadIdx.x, step = WARP ? 32 : blockDim.x;
  const int r = team / groups, off = (team - r * groups) * a.part, nvec = a.part >> 2;
  auto sum = [&](float v) { return WARP ? warp_sum(v) : block_sum(v, red); };
  float4 d[VPT], v[VPT], w[VPT], wd[VPT];
#pragma unroll
  for (int k = 0; k < VPT; ++k) {        // weights: no kernel of a step writes them
    const int i = at + k * step;
    w[k] = make_float4(1.f, 1.f, 1.f, 1.f);
    wd[k] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < nvec) {
      if (a.weight) w[k] = load4(a.weight + off + i * 4);
      if (a.through) wd[k] = load4(a.through + off + i * 4);
    }
  }
  pdl_launch_dependents();
  pdl_wait();
  const int src = a.rows ? a.rows[r] : r;
  const TD* dr = a.delta ? (const TD*)a.delta + (size_t)src * a.dim + off : nullptr;
  float* xr = a.x ? a.x + (size_t)src * a.dim + off : nullptr;
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = at + k * step;
    d[k] = v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < nvec) {
      if (dr) d[k] = load4(dr + i * 4);
      if (xr) v[k] = load4(xr + i * 4);
    }
    ss += dot4(d[k]);
  }
  if (a.through) {
    const float inv = 1.0f / sqrtf(sum(ss) / (float)a.part + a.eps);
#pragma unroll
    for (int k = 0; k < VPT; ++k) d[k] = mul4(d[k], inv, wd[k]);
  }
  ss = 0.f;
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    v[k].x += d[k].x; v[k].y += d[k].y; v[k].z += d[k].z; v[k].w += d[k].w;
    ss += dot4(v[k]);
  }
  const float inv = a.weight ? 1.0f / sqrtf(sum(ss) / (float)a.part + a.eps) : 1.0f;
  TO* orow = (TO*)a.out + (size_t)r * a.dim + off;
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = at + k * step;
    if (i < nvec) {
      if (xr && dr && !a.rows) store4(xr + i * 4, v[k]);
      store4(orow + i * 4, mul4(v[k], inv, w[k]));
    }
  }
}

// Any part length: the part is kept in shared memory.
template <typename TD, typename TO>
__global__ void __launch_bounds__(256) grouped_norm_kernel(const NormArgs a) {
  __shared__ float red[32];
  extern __shared__ float buf[];
  const int src = a.rows ? a.rows[blockIdx.x] : (int)blockIdx.x;
  const int off = blockIdx.y * a.part;
  const TD* dr = a.delta ? (const TD*)a.delta + (size_t)src * a.dim + off : nullptr;
  float* xr = a.x ? a.x + (size_t)src * a.dim + off : nullptr;
  float inv_d = 1.f;
  if (a.through) {
    float ss = 0.f;
    for (int i = threadIdx.x; i < a.part; i += blockDim.x) { const float v = to_float(dr[i]); ss += v * v; }
    inv_d = 1.0f / sqrtf(block_sum(ss, red) / (float)a.part + a.eps);
  }
  float ss = 0.f;
  for (int i = threadIdx.x; i < a.part; i += blockDim.x) {
    float v = xr ? xr[i] : 0.f;
    if (dr) {
      float d = to_float(dr[i]);
      if (a.through) d = d * inv_d * a.through[off + i];
      v += d;
    }
    buf[i] = v;
    ss += v * v;
  }
  const float inv = a.weight ? 1.0f / sqrtf(block_sum(ss, red) / (float)a.part + a.eps) : 1.0f;
  TO* orow = (TO*)a.out + (size_t)blockIdx.x * a.dim + off;
  for (int i = threadIdx.x; i < a.part; i += blockDim.x) {
    const float v = buf[i];
    if (xr && dr && !a.rows) xr[i] = v;
    orow[i] = from_float<TO>(a.weight ? v * inv * a.weight[off + i] : v);
  }
}

template <typename TD, typename TO>
int launch_grouped_norm(const NormArgs& a, int n_rows, int groups, cudaStream_t stream) {
  const int nvec = a.part / 4;
  if (a.part % 4 == 0 && nvec <= 512 * 4 && (!a.x || aligned16(a.x)) && (!a.delta || aligned16(a.delta)) && (!a.through || aligned16(a.through)) &&
      aligned16(a.weight) && aligned16(a.out)) {
    const int n_parts = n_rows * groups;
#define SB_GROUPED(VPT, WARP, BLOCKS, THREADS)                                                                                         \
  SB_PDL_CHECK(launch_pdl(grouped_norm_vec_kernel<TD, TO, VPT, WARP>, dim3(BLOCKS), dim3(THREADS), 0, stream, a, n_parts, groups))
    if (nvec <= 128) {
      const int warps = n_parts >= 4 * sm_count() ? 8 : 1, blocks = (n_parts + warps - 1) / warps;
      if (nvec <= 32) SB_GROUPED(1, true, blocks, warps * 32);
      else if (nvec <= 64) SB_GROUPED(2, true, blocks, warps * 32);
      else SB_GROUPED(4, true, blocks, warps * 32);
      return 0;
    }
    const int threads = nvec <= 512 ? 256 : 512;
    const int vpt = (nvec + threads - 1) / threads;
    if (vpt <= 1) SB_GROUPED(1, false, n_parts, threads);
    else if (vpt <= 2) SB_GROUPED(2, false, n_parts, threads);
    else SB_GROUPED(4, false, n_parts, threads);
#undef SB_GROUPED
    return 0;
  }
  const size_t smem = (size_t)a.part * sizeof(float);
  if (smem > 200 * 1024) return SB_ERR_LIMIT;
  auto k = grouped_norm_kernel<TD, TO>;
  if (smem > 40 * 1024) cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  k<<<dim3(n_rows, groups), a.part <= 64 ? 64 : 256, smem, stream>>>(a);
  SB_LAUNCH_CHECK();
  return 0;
}

// ------------------------------------------------------------------------------------------ polynomial of normalised powers
// One block per row; z and out may be the same buffer. The three sums of squares in one pass, together in one reduction.
__device__ __forceinline__ void powers(float z, float& s1, float& s2, float& s3) {
  const float z2 = z * z, z4 = z2 * z2;
  s1 += z2;
  s2 += z4;
  s3 += z4 * z2;
}
__device__ __forceinline__ float3 block_sum3(float3 v, float (*red)[32]) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = (blockDim.x + 31) >> 5;
  v.x = warp_sum(v.x); v.y = warp_sum(v.y); v.z = warp_sum(v.z);
  if (lane == 0) { red[0][warp] = v.x; red[1][warp] = v.y; red[2][warp] = v.z; }
  __syncthreads();
  v.x = warp_sum(lane < n_warps ? red[0][lane] : 0.f);
  v.y = warp_sum(lane < n_warps ? red[1][lane] : 0.f);
  v.z = warp_sum(lane < n_warps ? red[2][lane] : 0.f);
  return v;
}
struct Poly {
  float a, b, c, e;
  __device__ __forceinline__ float at(float z) const { return z * (a + z * (b + z * c)) + e; }
};
__device__ __forceinline__ Poly poly_of(const float* coef, float3 sums, int n, float eps) {
  Poly f;
  f.a = coef[0] / sqrtf(sums.x / (float)n + eps);
  f.b = coef[1] / sqrtf(sums.y / (float)n + eps);
  f.c = coef[2] / sqrtf(sums.z / (float)n + eps);
  f.e = coef[3];
  return f;
}

// bfloat16 rows of a multiple of 8 elements that fit VPT pieces of 16 bytes a thread: read once, kept in registers.
template <int VPT>
__global__ void __launch_bounds__(512) poly_norm_vec_kernel(const bf16* z, const float* __restrict__ coef, float eps, bf16* out, int n) {
  __shared__ float red[3][32];
  pdl_launch_dependents();
  pdl_wait();
  const uint4* zr = reinterpret_cast<const uint4*>(z + (size_t)blockIdx.x * n);
  const int nvec = n >> 3;
  uint4 v[VPT];
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    v[k] = i < nvec ? zr[i] : make_uint4(0, 0, 0, 0);
  }
  float3 s = make_float3(0.f, 0.f, 0.f);
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&v[k]);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 f = __bfloat1622float2(h[j]);
      powers(f.x, s.x, s.y, s.z);
      powers(f.y, s.x, s.y, s.z);
    }
  }
  const Poly f = poly_of(coef, block_sum3(s, red), n, eps);
  uint4* orow = reinterpret_cast<uint4*>(out + (size_t)blockIdx.x * n);
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < nvec) {
      __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&v[k]);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 u = __bfloat1622float2(h[j]);
        h[j] = __floats2bfloat162_rn(f.at(u.x), f.at(u.y));
      }
      orow[i] = v[k];
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256) poly_norm_kernel(const T* z, const float* __restrict__ coef, float eps, T* out, int n) {
  __shared__ float red[3][32];
  const T* zr = z + (size_t)blockIdx.x * n;
  float3 s = make_float3(0.f, 0.f, 0.f);
  for (int i = threadIdx.x; i < n; i += blockDim.x) powers(to_float(zr[i]), s.x, s.y, s.z);
  const Poly f = poly_of(coef, block_sum3(s, red), n, eps);
  T* orow = out + (size_t)blockIdx.x * n;
  for (int i = threadIdx.x; i < n; i += blockDim.x) orow[i] = from_float<T>(f.at(to_float(zr[i])));
}

}  // namespace

// x float [*, dim] or null; delta [*, dim] of delta_dtype or null; through float [dim] or null (the weight of the norm the delta goes
// through first); rows int [n_rows] or null (only these rows, x stays as it is); weight float [dim], or null: no second norm; out [n_rows, dim] of out_dtype.
SB_EXPORT int sb_add_grouped_rmsnorm(float* x, const void* delta, int delta_dtype, const float* through, const int* rows, const float* weight,
                                     void* out, int out_dtype, int n_rows, int dim, int groups, float eps, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (dim <= 0 || groups <= 0 || dim % groups || groups > 65535 || !out || (!x && !delta) || (through && !delta)) return SB_ERR_SHAPE;
  const bool df = delta == nullptr || delta_dtype == SB_DTYPE_F32;
  if (!df && delta_dtype != SB_DTYPE_BF16) return SB_ERR_DTYPE;
  const NormArgs a = {x, delta, through, rows, weight, out, dim, dim / groups, eps};
  if (out_dtype == SB_DTYPE_F32)
    return df ? launch_grouped_norm<float, float>(a, n_rows, groups, stream) : launch_grouped_norm<bf16, float>(a, n_rows, groups, stream);
  if (out_dtype == SB_DTYPE_BF16)
    return df ? launch_grouped_norm<float, bf16>(a, n_rows, groups, stream) : launch_grouped_norm<bf16, bf16>(a, n_rows, groups, stream);
  return SB_ERR_DTYPE;
}

// z, out [n_rows, n] (contiguous, may be the same buffer), coef float [4].
SB_EXPORT int sb_poly_norm(const void* z, const float* coef, float eps, void* out, int n_rows, int n, int dtype, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (n <= 0 || !coef) return SB_ERR_SHAPE;
  if (dtype == SB_DTYPE_BF16) {
    const int nvec = n / 8;
    if (n % 8 == 0 && nvec <= 512 * 8 && aligned16(z) && aligned16(out)) {
      // many rows: small blocks with much in flight; few: as many threads as there is work for
      const bool many = n_rows >= 4 * sm_count();
      const int threads = nvec <= 32 ? 32 : (nvec <= 128 ? 64 : (many && nvec <= 1024 ? 128 : (nvec <= 512 || (many && nvec <= 2048) ? 256 : 512)));
      const int vpt = (nvec + threads - 1) / threads;
      if (vpt <= 2) SB_PDL_CHECK(launch_pdl(poly_norm_vec_kernel<2>, dim3(n_rows), dim3(threads), 0, stream, (const bf16*)z, coef, eps, (bf16*)out, n));
      else if (vpt <= 4) SB_PDL_CHECK(launch_pdl(poly_norm_vec_kernel<4>, dim3(n_rows), dim3(threads), 0, stream, (const bf16*)z, coef, eps, (bf16*)out, n));
      else SB_PDL_CHECK(launch_pdl(poly_norm_vec_kernel<8>, dim3(n_rows), dim3(threads), 0, stream, (const bf16*)z, coef, eps, (bf16*)out, n));
      return 0;
    }
    poly_norm_kernel<bf16><<<n_rows, 256, 0, stream>>>((const bf16*)z, coef, eps, (bf16*)out, n);
  } else if (dtype == SB_DTYPE_F32) {
    poly_norm_kernel<float><<<n_rows, 256, 0, stream>>>((const float*)z, coef, eps, (float*)out, n);
  } else {
    return SB_ERR_DTYPE;
  }
  SB_LAUNCH_CHECK();
  return 0;
}
