// Routing of a mixture of experts with a correction of the choice, experts that return their input, and shared experts
// that ride with the routed ones.
//
// The router's logits cover `experts` stored experts and, behind them, `identity` ones without weights.  Scores are their
// softmax; the `top` largest of score + correction are chosen; a chosen output weighs score / (sum of the chosen scores +
// 1e-20) * scale.  A token's slots are its `top` choices and then `always` further stored experts (the parts of a shared
// expert) with weight one.  A slot that chose an identity expert holds no expert (-1); its weight goes to idw, a multiple
// of the token's input.  All of it is fp32.
//
// For few rows one CTA also builds the list of units for the grouped GEMV: up to 8 rows of one expert, so that every
// chosen expert is streamed once whatever the number of its rows.  Many rows go through moe.cu's dispatch.
#include "act_type.cuh"

namespace {

constexpr int kPer = 16, kMaxOut = 32 * kPer;          // router outputs
constexpr int kUnit = 8, kMaxRows = 64, kMaxTop = 32;

struct RouteArgs {
  const float* logits; int64_t ldl;
  const float* corr;                     // [experts + identity]
  const int* positions;                  // < 0: padding row, no slots (null: none)
  int T, experts, identity, top, always;
  float scale;
  int* idx; float* w; float* idw;        // [T, top + always], [T, top + always], [T]
};

// One warp: slots of row `t`; lane j < top holds choice j (expert or -1) on return.
__device__ __forceinline__ int route_row(const RouteArgs& a, int64_t t, int lane) {
  const int n = a.experts + a.identity, kt = a.top + a.always;
  const bool pad = a.positions && a.positions[t] < 0;
  const float* row = a.logits + t * a.ldl;
  float s[kPer], c[kPer], mx = -INFINITY, sum = 0.f;
#pragma unroll
  for (int i = 0; i < kPer; ++i) {
    const int e = lane + 32 * i;
    s[i] = e < n ? row[e] : -INFINITY;
    mx = fmaxf(mx, s[i]);
  }
  mx = warp_max(mx);
#pragma unroll
  for (int i = 0; i < kPer; ++i) {
    s[i] = lane + 32 * i < n ? expf(s[i] - mx) : 0.f;
    sum += s[i];
  }
  sum = warp_sum(sum);
#pragma unroll
  for (int i = 0; i < kPer; ++i) {
    const int e = lane + 32 * i;
    s[i] /= sum;
    c[i] = e < n ? s[i] + a.corr[e] : -INFINITY;
  }
  float my = 0.f, chosen = 0.f;
  int mine = -1;
  for (int k = 0; k < a.top; ++k) {
    float best = -INFINITY;
    int bi = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < kPer; ++i)
      if (c[i] > best) { best = c[i]; bi = lane + 32 * i; }       // ties keep the lowest index
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ob > best || (ob == best && oi < bi)) { best = ob; bi = oi; }
    }
    if (bi >= n) bi = 0;                                         // logits that are not numbers: any in-range expert
    float v = 0.f;
#pragma unroll
    for (int i = 0; i < kPer; ++i)
      if (i == bi >> 5) {
        v = s[i];
        if ((bi & 31) == lane) c[i] = -INFINITY;
      }
    v = __shfl_sync(0xffffffffu, v, bi & 31);
    chosen += v;
    if (lane == k) { my = v; mine = bi; }
  }
  const float wt = my / (chosen + 1e-20f) * a.scale;
  const bool ident = lane < a.top && mine >= a.experts;
  const float iw = warp_sum(ident ? wt : 0.f);
  if (ident || pad) mine = -1;
  if (lane < a.top) {
    a.idx[t * kt + lane] = mine;
    a.w[t * kt + lane] = mine < 0 ? 0.f : wt;
  }
  for (int j = lane; j < a.always; j += 32) {
    a.idx[t * kt + a.top + j] = pad ? -1 : a.experts + j;
    a.w[t * kt + a.top + j] = pad ? 0.f : 1.f;
  }
  if (lane == 0) a.idw[t] = pad ? 0.f : iw;
  return mine;
}

__global__ void __launch_bounds__(256) routed_topk_kernel(const RouteArgs a) {
  griddep_launch();
  griddep_wait();
  const int64_t t = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (t < a.T) route_row(a, t, threadIdx.x & 31);
}

struct UnitList { int* pos; int* src; int* count; int* row0; int* rows; int* expert; int max_units; };

// Routing of up to kMaxRows rows and their units, one CTA: a warp per row, counts and prefixes per expert in shared memory.
__global__ void __launch_bounds__(1024) routed_units_kernel(const RouteArgs a, const UnitList u) {
  extern __shared__ int sm[];
  const int kt = a.top + a.always, S = a.T * kt, E = a.experts + a.always;
  int* ex = sm;                  // [S] expert of every slot
  int* rank = ex + S;            // [S] its place among the expert's slots
  int* cnt = rank + S;           // [E]
  int* off = cnt + E;            // [E] first sorted row
  int* uoff = off + E;           // [E] first unit
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  for (int e = tid; e < E; e += 1024) cnt[e] = 0;
  griddep_launch();
  griddep_wait();
  __syncthreads();
  for (int t = warp; t < a.T; t += 32) {
    const int mine = route_row(a, t, lane);
    const bool pad = a.positions && a.positions[t] < 0;
    for (int j = lane; j < kt; j += 32) {
      const int e = j < a.top ? mine : (pad ? -1 : a.experts + j - a.top);
      ex[t * kt + j] = e;
      rank[t * kt + j] = e >= 0 ? atomicAdd(cnt + e, 1) : 0;
    }
  }
  __syncthreads();
  if (warp == 0) {
    int rows = 0, units = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + lane, n = e < E ? cnt[e] : 0, nu = (n + kUnit - 1) / kUnit;
      int pr = n, pu = nu;
#pragma unroll
      for (int d = 1; d < 32; d <<= 1) {
        const int ur = __shfl_up_sync(0xffffffffu, pr, d), uu = __shfl_up_sync(0xffffffffu, pu, d);
        if (lane >= d) { pr += ur; pu += uu; }
      }
      if (e < E) { off[e] = rows + pr - n; uoff[e] = units + pu - nu; }
      rows += __shfl_sync(0xffffffffu, pr, 31);
      units += __shfl_sync(0xffffffffu, pu, 31);
    }
    if (lane == 0) *u.count = min(units, u.max_units);
  }
  __syncthreads();
  for (int e = tid; e < E; e += 1024) {
    int k = uoff[e];
    for (int i = 0; i < cnt[e]; i += kUnit, ++k)
      if (k < u.max_units) { u.row0[k] = off[e] + i; u.rows[k] = min(kUnit, cnt[e] - i); u.expert[k] = e; }
  }
  for (int s = tid; s < S; s += 1024) {
    const int e = ex[s];
    const int r = e >= 0 ? off[e] + rank[s] : -1;
    u.pos[s] = r;
    if (r >= 0) u.src[r] = s / kt;
  }
}

// y[r] = act(W[expert] x[r or src[r]]) over units of up to 8 rows, true fp32: a warp per output column.
__global__ void __launch_bounds__(256) routed_linear_f32_kernel(const float* __restrict__ W, int64_t stride, const float* __restrict__ x,
                                                                int64_t ldx, float* __restrict__ y, int64_t ldy, int N, int K,
                                                                const int* __restrict__ count, const int* __restrict__ row0,
                                                                const int* __restrict__ rows, const int* __restrict__ expert,
                                                                const int* __restrict__ src, int relu2) {
  griddep_launch();
  griddep_wait();
  const int n = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (n >= N) return;
  for (int u = blockIdx.y; u < *count; u += gridDim.y) {
    const int r0 = row0[u], m = rows[u];
    const float* w = W + (int64_t)expert[u] * stride + (int64_t)n * K;
    for (int i = 0; i < m; ++i) {
      const float* xr = x + (int64_t)(src ? src[r0 + i] : r0 + i) * ldx;
      float s = 0.f;
      for (int k = lane; k < K; k += 32) s = fmaf(w[k], xr[k], s);
      s = warp_sum(s);
      if (relu2) { s = fmaxf(s, 0.f); s *= s; }
      if (lane == 0) y[(int64_t)(r0 + i) * ldy + n] = s;
    }
  }
}

int route_args(RouteArgs* a, const void* logits, int64_t ldl, const void* corr, const void* positions, int64_t T, int64_t experts,
               int64_t identity, int64_t top, int64_t always, float scale, void* idx, void* w, void* idw) {
  if (!logits || !corr || !idx || !w || !idw || T < 1 || experts < 1 || identity < 0 || always < 0) return CB_ERR_ARG;
  if (experts + identity > kMaxOut || top < 1 || top > kMaxTop || top > experts + identity || always > kMaxTop) return CB_ERR_SHAPE;
  a->logits = (const float*)logits; a->ldl = ldl; a->corr = (const float*)corr; a->positions = (const int*)positions;
  a->T = (int)T; a->experts = (int)experts; a->identity = (int)identity; a->top = (int)top; a->always = (int)always; a->scale = scale;
  a->idx = (int*)idx; a->w = (float*)w; a->idw = (float*)idw;
  return 0;
}

}  // namespace

// Slots of `T` rows: idx / w [T, top + always] (idx -1: no stored expert), idw [T].
CB_EXPORT int cb_routed_topk(const void* logits, int64_t ldl, const void* corr, const void* positions, int64_t T, int64_t experts,
                             int64_t identity, int64_t top, int64_t always, float scale, void* idx, void* w, void* idw, void* stream) {
  RouteArgs a;
  const int rc = route_args(&a, logits, ldl, corr, positions, T, experts, identity, top, always, scale, idx, w, idw);
  if (rc) return rc;
  return (int)cb_launch(routed_topk_kernel, dim3((unsigned)((T + 7) / 8)), dim3(256), 0, (cudaStream_t)stream, a);
}

// The same for T <= 64 rows, with the sorted order (pos [T * slots], src [T * slots]) and the units of up to 8 rows of an expert.
CB_EXPORT int cb_routed_units(const void* logits, int64_t ldl, const void* corr, const void* positions, int64_t T, int64_t experts,
                              int64_t identity, int64_t top, int64_t always, float scale, void* idx, void* w, void* idw, void* pos,
                              void* src, void* count, void* row0, void* rows, void* expert, int64_t max_units, void* stream) {
  RouteArgs a;
  const int rc = route_args(&a, logits, ldl, corr, positions, T, experts, identity, top, always, scale, idx, w, idw);
  if (rc) return rc;
  if (T > kMaxRows) return CB_ERR_SHAPE;
  if (!pos || !src || !count || !row0 || !rows || !expert || max_units < 1) return CB_ERR_ARG;
  const UnitList u = {(int*)pos, (int*)src, (int*)count, (int*)row0, (int*)rows, (int*)expert, (int)max_units};
  const size_t smem = sizeof(int) * (size_t)(2 * T * (top + always) + 3 * (experts + always));
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(routed_units_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return (int)cb_launch(routed_units_kernel, dim3(1), dim3(1024), smem, (cudaStream_t)stream, a, u);
}

// fp32 expert product over a unit list (any number of units): y[r] = W[expert] x[src[r]] (src null: x[r]), squared relu with relu2.
CB_EXPORT int cb_routed_linear_f32(const void* W, int64_t stride, const void* x, int64_t ldx, void* y, int64_t ldy, int64_t N, int64_t K,
                                   const void* count, const void* row0, const void* rows, const void* expert, const void* src,
                                   int64_t max_units, int64_t relu2, void* stream) {
  if (!W || !x || !y || !count || !row0 || !rows || !expert || N < 1 || K < 1 || max_units < 1) return CB_ERR_ARG;
  const dim3 grid((unsigned)((N + 7) / 8), (unsigned)(max_units < 4096 ? max_units : 4096));
  return (int)cb_launch(routed_linear_f32_kernel, grid, dim3(256), 0, (cudaStream_t)stream, (const float*)W, stride, (const float*)x, ldx,
                        (float*)y, ldy, (int)N, (int)K, (const int*)count, (const int*)row0, (const int*)rows, (const int*)expert,
                        (const int*)src, (int)relu2);
}
