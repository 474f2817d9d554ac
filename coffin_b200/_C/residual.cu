// A plain fp32 residual [rows, W]: embedding, and one kernel per sublayer boundary.
//
// The boundary adds what the sublayer left - a dense row, or the weighted expert rows of a routed feed-forward found
// through their sorted positions plus a multiple of the sublayer's own input (experts that return their input) - and
// leaves the RMS-normalised row for the next projection.  What is added may be RMS-normed with a gain of its own first (a norm
// behind every sublayer), and the token's embedding may be added with it (layers that run again).  A row crosses HBM once per sublayer and its sum is never rounded.
// Residuals of several streams and depth averages are streams.cu's and depth.cu's.
#include "act_type.cuh"

namespace {

constexpr int kMaxSlots = 64;

struct ResidualArgs {
  float* x;
  const void* y; int64_t ldy;            // dense output rows, or null
  const void* ys; int64_t ldys;          // expert output rows, sorted by expert, or null
  const int* pos; const float* w; int k; // [rows, k]: sorted row of every slot (< 0: none) and its weight
  const float* idw;                      // [rows]: weight of the sublayer's input, or null
  const void* hin; int64_t ldhin;        // that input (may be the rows h is written to)
  const float* gain; void* h; int64_t ldh;
  const int* rows;                       // residual row behind output row i (null: i)
  const float* post;                     // gain of the norm over what is added, or null
  const void* embed; const int64_t* tokens; int64_t vocab;   // table and tokens of the rows, or null
  int W; float eps; int store;
};

template <typename TA, int V> struct Vec;
template <typename TA> struct Vec<TA, 4> {
  static __device__ __forceinline__ void load(const TA* p, float* f) {
    const float4 v = act_load4(p);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
  }
  static __device__ __forceinline__ void store(TA* p, const float* f) { act_store4(p, make_float4(f[0], f[1], f[2], f[3])); }
};
template <typename TA> struct Vec<TA, 1> {
  static __device__ __forceinline__ void load(const TA* p, float* f) { f[0] = act_load(p); }
  static __device__ __forceinline__ void store(TA* p, const float* f) { act_store(p, f[0]); }
};

// V columns per access, up to IT accesses per thread; the row stays in registers between the sum and the norm.
template <typename TA, int V, int IT, bool POST>
__global__ void __launch_bounds__(1024) residual_step_kernel(const ResidualArgs a) {
  __shared__ float red[32];
  __shared__ int pos_s[kMaxSlots];
  __shared__ float w_s[kMaxSlots];
  const int tid = threadIdx.x, NT = blockDim.x;
  griddep_launch();
  griddep_wait();
  const int64_t r = a.rows ? a.rows[blockIdx.x] : (int64_t)blockIdx.x;
  if (r < 0) return;
  if (a.ys) {
    if (tid < a.k) { pos_s[tid] = a.pos[r * a.k + tid]; w_s[tid] = a.w[r * a.k + tid]; }
    __syncthreads();
  }
  float* xr = a.x + r * a.W;
  const TA* y = a.y ? reinterpret_cast<const TA*>(a.y) + r * a.ldy : nullptr;
  const TA* hin = reinterpret_cast<const TA*>(a.hin) + r * a.ldhin;
  const TA* ys = reinterpret_cast<const TA*>(a.ys);
  const float idw = a.idw ? a.idw[r] : 0.f;
  const TA* er = nullptr;
  if (POST && a.embed) {
    const int64_t tok = a.tokens[r];
    er = reinterpret_cast<const TA*>(a.embed) + (tok < 0 ? 0 : (tok >= a.vocab ? a.vocab - 1 : tok)) * a.W;
  }
  float u[IT][V], add[POST ? IT : 1][V], ss = 0.f, sa = 0.f;
#pragma unroll
  for (int t = 0; t < IT; ++t) {
    const int i = (tid + t * NT) * V;
#pragma unroll
    for (int v = 0; v < V; ++v) u[t][v] = 0.f;
    if (i >= a.W) continue;
    Vec<float, V>::load(xr + i, u[t]);
    float* s = add[POST ? t : 0];
    float f[V];
#pragma unroll
    for (int v = 0; v < V; ++v) s[v] = 0.f;
    if (y) Vec<TA, V>::load(y + i, s);
    if (ys) {
#pragma unroll 4
      for (int j = 0; j < a.k; ++j) {
        if (pos_s[j] < 0) continue;
        Vec<TA, V>::load(ys + (int64_t)pos_s[j] * a.ldys + i, f);
#pragma unroll
        for (int v = 0; v < V; ++v) s[v] = fmaf(w_s[j], f[v], s[v]);
      }
    }
    if (idw != 0.f) {
      Vec<TA, V>::load(hin + i, f);
#pragma unroll
      for (int v = 0; v < V; ++v) s[v] = fmaf(idw, f[v], s[v]);
    }
    if (POST) {
#pragma unroll
      for (int v = 0; v < V; ++v) sa = fmaf(s[v], s[v], sa);
      continue;
    }
    if (y || ys) {
#pragma unroll
      for (int v = 0; v < V; ++v) u[t][v] += s[v];
      if (a.store) Vec<float, V>::store(xr + i, u[t]);
    }
#pragma unroll
    for (int v = 0; v < V; ++v) ss = fmaf(u[t][v], u[t][v], ss);
  }
  if (POST) {
    const float ra = a.post ? 1.f / sqrtf(block_sum(sa, red) / (float)a.W + a.eps) : 1.f;
#pragma unroll
    for (int t = 0; t < IT; ++t) {
      const int i = (tid + t * NT) * V;
      if (i >= a.W) continue;
      float g[V];
#pragma unroll
      for (int v = 0; v < V; ++v) g[v] = 1.f;
      if (a.post) Vec<float, V>::load(a.post + i, g);
#pragma unroll
      for (int v = 0; v < V; ++v) u[t][v] = fmaf(add[t][v], g[v] * ra, u[t][v]);
      if (er) {
        Vec<TA, V>::load(er + i, g);
#pragma unroll
        for (int v = 0; v < V; ++v) u[t][v] += g[v];
      }
      if (a.store) Vec<float, V>::store(xr + i, u[t]);
#pragma unroll
      for (int v = 0; v < V; ++v) ss = fmaf(u[t][v], u[t][v], ss);
    }
  }
  if (!a.h) return;
  const float rstd = 1.f / sqrtf(block_sum(ss, red) / (float)a.W + a.eps);
  TA* hr = reinterpret_cast<TA*>(a.h) + (int64_t)blockIdx.x * a.ldh;
#pragma unroll
  for (int t = 0; t < IT; ++t) {
    const int i = (tid + t * NT) * V;
    if (i >= a.W) continue;
    float g[V];
    Vec<float, V>::load(a.gain + i, g);
#pragma unroll
    for (int v = 0; v < V; ++v) g[v] *= u[t][v] * rstd;
    Vec<TA, V>::store(hr + i, g);
  }
}

template <typename TA>
__global__ void __launch_bounds__(256) residual_embed_kernel(const TA* __restrict__ embed, const int64_t* __restrict__ tokens,
                                                             float* __restrict__ x, int W, int64_t V, float scale) {
  griddep_launch();
  griddep_wait();
  const int64_t r = blockIdx.x;
  int64_t tok = tokens[r];
  tok = tok < 0 ? 0 : (tok >= V ? V - 1 : tok);
  for (int i = threadIdx.x; i < W; i += 256) x[r * W + i] = act_load(embed + tok * W + i) * scale;
}

template <typename TA, bool POST>
int step_launch(const ResidualArgs& a, int64_t n, cudaStream_t st) {
  const bool v4 = a.W % 4 == 0 && a.ldh % 4 == 0 && a.ldy % 4 == 0 && a.ldys % 4 == 0 && a.ldhin % 4 == 0;
  const int per = v4 ? (a.W + 3) / 4 : a.W;
  const int nt = per >= 1024 ? 1024 : (per + 31) / 32 * 32;
  const dim3 grid((unsigned)n), block((unsigned)nt);
  if (v4) {
    if (per <= nt) return (int)cb_launch(residual_step_kernel<TA, 4, 1, POST>, grid, block, 0, st, a);
    if (per <= 2 * nt) return (int)cb_launch(residual_step_kernel<TA, 4, 2, POST>, grid, block, 0, st, a);
    if (per <= 4 * nt) return (int)cb_launch(residual_step_kernel<TA, 4, 4, POST>, grid, block, 0, st, a);
    return CB_ERR_SHAPE;
  }
  if (per <= 4 * nt) return (int)cb_launch(residual_step_kernel<TA, 1, 4, POST>, grid, block, 0, st, a);
  if (per <= 16 * nt) return (int)cb_launch(residual_step_kernel<TA, 1, 16, POST>, grid, block, 0, st, a);
  return CB_ERR_SHAPE;
}

}  // namespace

// One sublayer boundary over `n` rows of x [.., W]: x += y (y null: nothing) + sum_j w[r, j] ys[pos[r, j]] (ys null: nothing)
// + idw[r] hin[r] (idw null: nothing), the sum of the added terms RMS-normed and multiplied by post first (post null: not), and
// embed[token[r]] (embed null: nothing); then h = rmsnorm(x) * gain (h null: no norm).  rows (int32 [n], optional): residual
// row behind output row i (with store 0: x is left as it is).  f32: activations are fp32 instead of bf16.  W <= 16384.
CB_EXPORT int cb_residual_step(void* x, const void* y, int64_t ldy, const void* ys, int64_t ldys, const void* pos, const void* w, int64_t k,
                               const void* idw, const void* hin, int64_t ldhin, const void* gain, void* h, int64_t ldh, const void* rows,
                               int64_t n, int64_t W, float eps, int64_t store, const void* post, const void* embed, const void* tokens,
                               int64_t vocab, int64_t f32, void* stream) {
  if (!x || n < 1 || W < 1 || (h && !gain) || (rows && store)) return CB_ERR_ARG;
  if ((post && !y && !ys) || (embed && (!tokens || vocab < 1))) return CB_ERR_ARG;
  if ((ys && (!pos || !w || k < 1 || k > kMaxSlots)) || (idw && !hin)) return CB_ERR_ARG;
  ResidualArgs a;
  a.x = (float*)x; a.y = y; a.ldy = ldy; a.ys = ys; a.ldys = ldys; a.pos = (const int*)pos; a.w = (const float*)w; a.k = (int)k;
  a.idw = (const float*)idw; a.hin = hin; a.ldhin = ldhin; a.gain = (const float*)gain; a.h = h; a.ldh = ldh; a.rows = (const int*)rows;
  a.W = (int)W; a.eps = eps; a.store = (int)store;
  a.post = (const float*)post; a.embed = embed; a.tokens = (const int64_t*)tokens; a.vocab = vocab;
  cudaStream_t st = (cudaStream_t)stream;
  if (post || embed) return f32 ? step_launch<float, true>(a, n, st) : step_launch<bf16, true>(a, n, st);
  return f32 ? step_launch<float, false>(a, n, st) : step_launch<bf16, false>(a, n, st);
}

// x[t] = embed[token[t]] * scale
CB_EXPORT int cb_residual_embed(const void* embed, const void* tokens, void* x, int64_t T, int64_t W, int64_t V, float scale, int64_t f32,
                                void* stream) {
  if (!embed || !tokens || !x || T < 1 || W < 1 || V < 1) return CB_ERR_ARG;
  const dim3 grid((unsigned)T), block(256);
  if (f32)
    return (int)cb_launch(residual_embed_kernel<float>, grid, block, 0, (cudaStream_t)stream, (const float*)embed, (const int64_t*)tokens,
                          (float*)x, (int)W, V, scale);
  return (int)cb_launch(residual_embed_kernel<bf16>, grid, block, 0, (cudaStream_t)stream, (const bf16*)embed, (const int64_t*)tokens,
                        (float*)x, (int)W, V, scale);
}
