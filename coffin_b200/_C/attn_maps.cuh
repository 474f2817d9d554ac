// Arguments of the multi-map attention kernels (attn_maps.cu, attn_maps_flash.cu).
//
// A head may have several score maps over the same values (differential attention has two): query heads are laid
// out head by head as [map 0, map 1, ...] of `dim` each, key heads likewise, values once per key/value head.
// Scores are scaled, multiplied by a position-dependent query temperature and optionally capped by
// cap * tanh(score / cap); key and value sizes are independent.
//
// Optional parts, each switched on by its field: a sliding window (a query sees itself and the window - 1 tokens before
// it), a sink per head (an entry of the softmax without key or value), interleaved rotary positions on queries and keys
// (taken when rows are appended and when a decode query is read), values mixed with another layer's, and an output gate
// per element.  Further: chunks (a query sees the tokens of its own chunk), an RMS norm of queries and keys per head ahead of the
// turn, values cached turned by their position with heads turned back by the query's, a score penalty that grows with the
// logarithm of the distance, and keys that are their own values: the pages hold keys as projected, read once for both
// products, and one factor per key stands for its norm.
#pragma once
#include "act_type.cuh"

struct AttnMapsArgs {
  const void* proj; int64_t ldp;         // projection rows: q at column 0, k at k_col, v at v_col
  int64_t k_col, v_col;
  void* kpool; void* vpool;              // [slots, G * maps, dim], [slots, G, vdim]
  const int* tables; int64_t ldbt;       // block tables [segments, ldbt] (blocks of 64 tokens)
  const int* row_seg;                    // segment of every row (null: row r is segment r)
  const int* positions;                  // position of every row (< 0: padding)
  const int* seg_row; const int* seg_pos;   // segments of consecutive tokens (prefill kernel)
  float* part_o; float* part_ml;         // [rows, H * maps, nsplit, vdim], [.., 2]: unnormalised sums, (max, denominator)
  int H, G, maps, dim, vdim, nsplit;
  float scale, cap;                      // cap <= 0: no cap
  float temp_coef; int temp_every;       // temp_every <= 0: no temperature
  int64_t ldk, ldv;                      // row strides of the pools (0: dense, G * maps * dim and G * vdim)
  // one map, prompt kernels: the finished head (divided by its denominator, times sigmoid(gate)) goes straight to
  // bf16 rows instead of part_o / part_ml (null: no)
  void* act; int64_t lda; const float* gates; int64_t ldg;
  int window;                            // keys pos - window + 1 .. pos are visible (<= 0: all up to pos)
  int rot_half;                          // pairs (2 i, 2 i + 1), i < rot_half, of queries and keys turn (0: none)
  const float* sink;                     // [H * maps] in score units, or null
  const float2* cs;                      // (cos, sin) [rows, rot_half]
  const void* v0; int64_t ldv0;          // values of another layer, rows like proj (null: none):
  float v_own, v_mix;                    //   v = v_own * own + v_mix * v0
  const void* egate; int64_t lde;        // one map: output gate pre-activations [rows, H * vdim], rows like proj (null: none)
  int chunk;                             // > 0: keys of the query's own chunk of this many tokens, counted from position 0
  int norm; float eps;                   // norm: queries and keys are divided by their root mean square per head, then
  const float* qn; const float* kn;      //   weighted [dim] (null: not)
  const float2* vcs;                     // (cos, sin) [rows, vdim / 2]: values are cached turned, heads turned back (null: no)
  float* kr;                             // one map: factors [blocks, G, 64] of the scores of the keys, which are cached as
                                         //   projected and are the values too (vpool is not used) (null: no)
  const float* r1; const float* r2;      // [H]: score -= r1 ln(1 + r2 distance) (null: no)
  float oscale;                          // one map: factor of the finished head
  float bound;                           // > 0: no score is larger, and no row's largest below -bound (norms bound them; at most
                                         //   kMaxBound): the reference of every softmax instead of a running maximum
};
// 2^(-2 bound log2 e) stays well inside the range of fp32, and of a bf16 remainder 2^-9 below it
constexpr float kMaxBound = 34.f;

// first key that the query at `pos` sees
__host__ __device__ __forceinline__ int first_key(const AttnMapsArgs& a, int pos) {
  const int w = a.window > 0 && pos >= a.window ? pos - a.window + 1 : 0;
  return a.chunk > 0 ? max(w, pos - pos % a.chunk) : w;
}
// norm, value turns, key factors and distance penalties: what the plain forms of append and decode leave out
__host__ __device__ __forceinline__ bool extended(const AttnMapsArgs& a) { return a.norm || a.vcs || a.kr || a.r1; }
// finite stand-in for "no key seen yet": exponentials of differences with it are 0 or 1, never NaN
constexpr float kNoKey = -1e30f;

constexpr int kPage = 64;
__host__ __device__ __forceinline__ int64_t pool_ldk(const AttnMapsArgs& a) { return a.ldk ? a.ldk : (int64_t)a.G * a.maps * a.dim; }
__host__ __device__ __forceinline__ int64_t pool_ldv(const AttnMapsArgs& a) { return a.ldv ? a.ldv : (int64_t)a.G * a.vdim; }

__device__ __forceinline__ float query_temp(const AttnMapsArgs& a, int pos) {
  return a.temp_every > 0 ? 1.f + a.temp_coef * logf((float)((pos + 1) / a.temp_every + 1)) : 1.f;
}
// entry c of a projected row (entry `in_head` of its head) after the turn
template <typename T>
__device__ __forceinline__ float turned(const T* p, int c, int in_head, const float2* cs, int half) {
  const float x = act_load(p + c);
  if (in_head >> 1 >= half) return x;
  const float2 t = cs[in_head >> 1];
  const float y = act_load(p + (in_head & 1 ? c - 1 : c + 1));
  return in_head & 1 ? x * t.x + y * t.y : x * t.x - y * t.y;
}
__device__ __forceinline__ float mixed(float own, float other, const AttnMapsArgs& a) {
  return a.v0 ? a.v_own * own + a.v_mix * other : own;
}
// factor slot of key `key` of a block, key/value head g
__device__ __forceinline__ int64_t factor_at(const AttnMapsArgs& a, int64_t block, int g) { return (block * a.G + g) * kPage; }
// entries (2 m, 2 m + 1) of a finished head, turned back by the query's angle
__device__ __forceinline__ void turn_back(float& x, float& y, const float2 t) {
  const float u = x;
  x = u * t.x + y * t.y;
  y = y * t.x - u * t.y;
}
__device__ __forceinline__ float lg2(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// tanh through one exponential: |error| ~ 1e-7
__device__ __forceinline__ float cap_score(float s, float cap, float inv_cap) {
  const float e = exp2f(s * inv_cap * 2.885390081777927f);       // exp(2 s / cap)
  return cap - __fdividef(2.f * cap, e + 1.f);
}
