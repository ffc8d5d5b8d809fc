// What the passes of talking_attention.cu and talking_attention_tc.cu share: the launch's arguments and the score.
#pragma once
#include "common.cuh"

namespace talk {

constexpr int BN = 64;               // keys per tile of the scratch buffer
constexpr float LOG2E = 1.4426950408889634f;
constexpr float FIXED_CAP = 60.f;    // a cap up to this bounds every exponential: no maximum is taken (2^87 at most)

struct Params {
  const void* q; int q_stride;
  const void* kc; const void* vc;
  const int* block_table; int bt_width;
  const int* cu_q; const int* kv_len; const int* positions;
  int H, G, per, ps, ps_shift, num_pages;    // query heads, kv heads, query heads of a kv head; page size (its log2, or -1)
  float scale, cap, cap_in;                  // cap 0: none; cap_in = scale / cap
  int fixed;                                 // exponentials against 0: the cap bounds them
  int chunk;
  const float* sinks;                        // [H] or null
  const void* talk;                          // [Hp, Hp] (bfloat16, zeros beyond H) or [H, H] (float32), row = output head
  float* e; float2* stats; void* w;          // scratch: [tokens, H, pitch] floats, [tokens, H, pitch / 64], [tokens, H, pitch]
  int pitch, t_lo, t_hi;                     // the launch covers tokens [t_lo, t_hi) of the step
  int zero_ahead;                            // mixed weights are written as zeros up to this many positions beyond a token's own
  void* out;                                 // [T, H * D]
  const int* wide_rows; int deep_on;         // requests the wide shape covers (null: all); deep_on: the deep shape takes the small ones
  int n_splits; float* part; int* tickets;   // values, deep: key splits, [R, G, splits, 16, D] floats, [R, G] zeros
};

__device__ __forceinline__ int first_key(const Params& p, int pos) { return p.chunk > 0 ? (pos / p.chunk) * p.chunk : 0; }

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// A raw product as a score in units of log2: scaled, capped. tanh(z) = 1 - 2 / (1 + e^(2z)); its error is about 2^-23 of the cap.
__device__ __forceinline__ float capped_log2(float raw, float two_in_log2, float cap_log2) {
  return fmaf(-2.f * cap_log2, rcp(1.f + ex2(raw * two_in_log2)), cap_log2);
}
__device__ __forceinline__ float score_log2(const Params& p, float raw) {
  return p.cap > 0.f ? capped_log2(raw, p.cap_in * (2.f * LOG2E), p.cap * LOG2E) : raw * (p.scale * LOG2E);
}

// Scores and values of the wide requests on tcgen05 (head sizes 64 and 128). max_keys, max_q, n_requests size grids.
bool tc_takes(int H, int G, int ps, int q_stride, int chunk);
int tc_tokens_per_tile(int H, int G);
int tc_scores(const Params& p, int n_tokens, int max_keys, int max_q, int n_requests, int* error, cudaStream_t stream);
int tc_values(const Params& p, int max_q, int n_requests, int* error, cudaStream_t stream);

}  // namespace talk
