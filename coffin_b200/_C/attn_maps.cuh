// Arguments of the multi-map attention kernels (attn_maps.cu, attn_maps_flash.cu).
//
// A head may have several score maps over the same values (differential attention has two): query heads are laid
// out head by head as [map 0, map 1, ...] of `dim` each, key heads likewise, values once per key/value head.
// Scores are scaled, multiplied by a position-dependent query temperature and optionally capped by
// cap * tanh(score / cap); key and value sizes are independent.
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
};

constexpr int kPage = 64;
__host__ __device__ __forceinline__ int64_t pool_ldk(const AttnMapsArgs& a) { return a.ldk ? a.ldk : (int64_t)a.G * a.maps * a.dim; }
__host__ __device__ __forceinline__ int64_t pool_ldv(const AttnMapsArgs& a) { return a.ldv ? a.ldv : (int64_t)a.G * a.vdim; }

__device__ __forceinline__ float query_temp(const AttnMapsArgs& a, int pos) {
  return a.temp_every > 0 ? 1.f + a.temp_coef * logf((float)((pos + 1) / a.temp_every + 1)) : 1.f;
}
// tanh through one exponential: |error| ~ 1e-7
__device__ __forceinline__ float cap_score(float s, float cap, float inv_cap) {
  const float e = exp2f(s * inv_cap * 2.885390081777927f);       // exp(2 s / cap)
  return cap - __fdividef(2.f * cap, e + 1.f);
}
