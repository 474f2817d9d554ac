// Routing of a mixture of experts with a correction of the choice, experts that return their input, and shared experts
// that ride with the routed ones.
//
// The router's logits cover `experts` stored experts and, behind them, `identity` ones without weights.  Scores are their
// softmax; the `top` largest of score + correction are chosen; a chosen output weighs score / (sum of the chosen scores +
// 1e-20) * scale.  With by_logit the correction is part of the logits: the largest of logit + correction are chosen, and weigh
// their softmax over the chosen ones, times scale.  A token's slots are its `top` choices and then `always` further stored experts (the parts of a shared
// expert) with weight one.  A slot that chose an identity expert holds no expert (-1); its weight goes to idw, a multiple
// of the token's input.  All of it is fp32.
//
// For few rows one CTA also builds the list of units for the grouped GEMV: up to 8 rows of one expert, so that every
// chosen expert is streamed once whatever the number of its rows.  Many rows go through moe.cu's dispatch.
#include "act_type.cuh"

namespace {

constexpr int kMaxOut = 512;                           // router outputs
constexpr int kUnit = 8, kMaxRows = 64, kMaxTop = 32;

struct RouteArgs {
  const float* logits; int64_t ldl;
  const float* corr;                     // [experts + identity]
  const int* positions;                  // < 0: padding row, no slots (null: none)
  int T, experts, identity, top, always;
  float scale;
  int* idx; float* w; float* idw;        // [T, top + always], [T, top + always], [T]
  int by_logit;
};

// unsigned integers in the order of the floats
__device__ __forceinline__ unsigned order_key(float x) {
  const unsigned u = __float_as_uint(x);
  return u & 0x80000000u ? ~u : u | 0x80000000u;
}

// One warp: slots of row `t`; lane j < top holds choice j (expert or -1) on return.  A lane keeps outputs lane + 32 i, i < PER.
template <int PER>
__device__ __forceinline__ int route_row(const RouteArgs& a, const float* row, int64_t t, int lane) {
  const int n = a.experts + a.identity, kt = a.top + a.always;
  const bool pad = a.positions && a.positions[t] < 0;
  float s[PER], mx = -INFINITY, sum = 0.f;
  unsigned c[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int e = lane + 32 * i;
    s[i] = e < n ? row[e] : -INFINITY;
    c[i] = e < n ? __float_as_uint(a.corr[e]) : 0u;
    if (a.by_logit && e < n) {
      s[i] += __uint_as_float(c[i]);
      c[i] = order_key(s[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < PER; ++i) mx = fmaxf(mx, s[i]);
  mx = warp_max(mx);
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    s[i] = expf(s[i] - mx);
    sum += s[i];
  }
  const float inv = 1.f / warp_sum(sum);
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    s[i] *= inv;
    if (!a.by_logit) c[i] = lane + 32 * i < n ? order_key(s[i] + __uint_as_float(c[i])) : 0u;      // 0: below every number
  }
  float my = 0.f, chosen = 0.f;
  int mine = -1;
#pragma unroll 1
  for (int k = 0; k < a.top; ++k) {
    unsigned best = 0u;
    int at = 0;
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (c[i] > best) { best = c[i]; at = i; }
    const unsigned top = __reduce_max_sync(0xffffffffu, best);
    const int me = best == top ? lane + 32 * at : 0x7fffffff;                     // ties keep the lowest index
    const int bi = min((int)__reduce_min_sync(0xffffffffu, (unsigned)me), n - 1);
    float v = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (lane + 32 * i == bi) { v = s[i]; c[i] = 0u; }
    v = __shfl_sync(0xffffffffu, v, bi & 31);
    chosen += v;
    if (lane == k) { my = v; mine = bi; }
  }
  const float wt = my * (a.scale / (chosen + 1e-20f));
  const bool ident = lane < a.top && mine >= a.experts;
  const float iw = a.identity ? warp_sum(ident ? wt : 0.f) : 0.f;
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

template <int PER>
__global__ void __launch_bounds__(128) routed_topk_kernel(const RouteArgs a) {
  griddep_launch();
  griddep_wait();
  const int64_t t = (int64_t)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (t < a.T) route_row<PER>(a, a.logits + t * a.ldl, t, threadIdx.x & 31);
}

struct UnitList { int* pos; int* src; int* count; int* row0; int* rows; int* expert; int max_units; };

// Routing of up to kMaxRows rows and their units by one CTA: a warp per row, counts per expert in shared memory.  The first slot
// that an expert was given takes its rows and units from running totals: experts come in no fixed order, and need none.
// `fresh`: the logits were written by this kernel.
template <int PER>
__device__ __forceinline__ void route_units(const RouteArgs& a, const UnitList& u, int* sm, bool fresh) {
  const int kt = a.top + a.always, S = a.T * kt, E = a.experts + a.always;
  int* ex = sm;                  // [S] expert of every slot
  int* rank = ex + S;            // [S] its place among the expert's slots
  int* cnt = rank + S;           // [E]
  int* off = cnt + E;            // [E] first sorted row
  __shared__ int rows_s, units_s;
  const int tid = threadIdx.x, NT = blockDim.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) { rows_s = 0; units_s = 0; }
  for (int e = tid; e < E; e += NT) cnt[e] = 0;
  __syncthreads();
  for (int t = warp; t < a.T; t += NT / 32) {
    const float* row = a.logits + (int64_t)t * a.ldl;
    float* copy = reinterpret_cast<float*>(off + E) + warp * kMaxOut;
    if (fresh) {                                                // written by other CTAs: past L1
      for (int e = lane; e < a.experts + a.identity; e += 32) copy[e] = __ldcg(row + e);
      __syncwarp();
      row = copy;
    }
    const int mine = route_row<PER>(a, row, t, lane);
    const bool pad = a.positions && a.positions[t] < 0;
    for (int j = lane; j < kt; j += 32) {
      const int e = j < a.top ? mine : (pad ? -1 : a.experts + j - a.top);
      ex[t * kt + j] = e;
      rank[t * kt + j] = e >= 0 ? atomicAdd(cnt + e, 1) : 0;
    }
  }
  __syncthreads();
  for (int s = tid; s < S; s += NT) {
    const int e = ex[s];
    if (e < 0 || rank[s]) continue;
    const int n = cnt[e], r0 = atomicAdd(&rows_s, n);
    int k = atomicAdd(&units_s, (n + kUnit - 1) / kUnit);
    off[e] = r0;
    for (int i = 0; i < n && k < u.max_units; i += kUnit, ++k) { u.row0[k] = r0 + i; u.rows[k] = min(kUnit, n - i); u.expert[k] = e; }
  }
  __syncthreads();
  for (int s = tid; s < S; s += NT) {
    const int e = ex[s], r = e >= 0 ? off[e] + rank[s] : -1;
    u.pos[s] = r;
    if (r >= 0) u.src[r] = s / kt;
  }
  if (tid == 0) *u.count = min(units_s, u.max_units);
}

template <int PER>
__global__ void __launch_bounds__(512) routed_units_kernel(const RouteArgs a, const UnitList u) {
  extern __shared__ int sm[];
  griddep_launch();
  griddep_wait();
  route_units<PER>(a, u, sm, false);
}

// The same with the router's product in front, for up to 8 bf16 rows: four warps share an output by K, weights requested ahead
// of the dependency; the last CTA to finish routes.
struct RouterProduct { const bf16* W; const bf16* h; int64_t ldh; int K; float* logits; unsigned* ticket; };
constexpr int kAhead = 4, kOut = 2, kSlices = 4;       // 16-byte pieces requested ahead per lane; outputs of a CTA, warps of an output
template <int PER, int ROWS>
__global__ void __launch_bounds__(32 * kOut * kSlices) routed_step_kernel(const RouteArgs a, const UnitList u, const RouterProduct p) {
  extern __shared__ int sm[];
  __shared__ float part[kOut][kSlices][ROWS];
  __shared__ bool last;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, o = warp / kSlices, sl = warp % kSlices;
  const int e = blockIdx.x * kOut + o, n = a.experts + a.identity, nc = p.K >> 3, per = (nc + kSlices - 1) / kSlices;
  const int c0 = sl * per, c1 = min(nc, c0 + per);
  const uint4 z = make_uint4(0, 0, 0, 0);
  const bf16* w = p.W + (int64_t)min(e, n - 1) * p.K;
  uint4 wv[kAhead];
  griddep_launch();
#pragma unroll
  for (int i = 0; i < kAhead; ++i) wv[i] = c0 + lane + 32 * i < c1 ? ld_stream(w + (c0 + lane + 32 * i) * 8) : z;
  griddep_wait();
  float acc[ROWS];
#pragma unroll
  for (int t = 0; t < ROWS; ++t) acc[t] = 0.f;
  for (int c = c0; c < c1; c += 32 * kAhead) {
    if (c != c0) {
#pragma unroll
      for (int i = 0; i < kAhead; ++i) wv[i] = c + lane + 32 * i < c1 ? ld_stream(w + (c + lane + 32 * i) * 8) : z;
    }
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      const int at = c + lane + 32 * i;
      if (at >= c1) continue;
      uint4 hv[ROWS];
#pragma unroll
      for (int t = 0; t < ROWS; ++t) hv[t] = t < a.T ? *reinterpret_cast<const uint4*>(p.h + t * p.ldh + at * 8) : z;
      float f[8], g[8];
      bf16x8_to_float(wv[i], f);
#pragma unroll
      for (int t = 0; t < ROWS; ++t) {
        bf16x8_to_float(hv[t], g);
#pragma unroll
        for (int k = 0; k < 8; ++k) acc[t] = fmaf(f[k], g[k], acc[t]);
      }
    }
  }
#pragma unroll
  for (int t = 0; t < ROWS; ++t) {
    const float v = warp_sum(acc[t]);
    if (lane == 0) part[o][sl][t] = v;
  }
  __syncthreads();
  if (threadIdx.x < kOut * ROWS) {
    const int oo = threadIdx.x / ROWS, t = threadIdx.x % ROWS, out = blockIdx.x * kOut + oo;
    float v = 0.f;
#pragma unroll
    for (int s = 0; s < kSlices; ++s) v += part[oo][s][t];
    if (out < n && t < a.T) __stcg(p.logits + t * a.ldl + out, v);
    __threadfence();
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    last = atomicAdd(p.ticket, 1u) == gridDim.x - 1;
    if (last) *p.ticket = 0;
  }
  __syncthreads();
  if (!last) return;
  __threadfence();
  route_units<PER>(a, u, sm, true);
}

// y[r] = act(W[expert] x[r or src[r]]) over units of up to 8 rows, true fp32: a warp per output column.  act 2: squared relu;
// 3: silu(gate) * up, an expert's N gate rows before its N up rows.
__global__ void __launch_bounds__(256) routed_linear_f32_kernel(const float* __restrict__ W, int64_t stride, const float* __restrict__ x,
                                                                int64_t ldx, float* __restrict__ y, int64_t ldy, int N, int K,
                                                                const int* __restrict__ count, const int* __restrict__ row0,
                                                                const int* __restrict__ rows, const int* __restrict__ expert,
                                                                const int* __restrict__ src, int act) {
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
      if (act == 2) { s = fmaxf(s, 0.f); s *= s; }
      if (act == 3) {
        const float* wu = w + (int64_t)N * K;
        float u = 0.f;
        for (int k = lane; k < K; k += 32) u = fmaf(wu[k], xr[k], u);
        s = silu_x(s) * warp_sum(u);
      }
      if (lane == 0) y[(int64_t)(r0 + i) * ldy + n] = s;
    }
  }
}

int route_args(RouteArgs* a, const void* logits, int64_t ldl, const void* corr, const void* positions, int64_t T, int64_t experts,
               int64_t identity, int64_t top, int64_t always, float scale, int64_t by_logit, void* idx, void* w, void* idw) {
  a->by_logit = (int)by_logit;
  if (!logits || !corr || !idx || !w || !idw || T < 1 || experts < 1 || identity < 0 || always < 0) return CB_ERR_ARG;
  if (experts + identity > kMaxOut || top < 1 || top > kMaxTop || top > experts + identity || always > kMaxTop) return CB_ERR_SHAPE;
  a->logits = (const float*)logits; a->ldl = ldl; a->corr = (const float*)corr; a->positions = (const int*)positions;
  a->T = (int)T; a->experts = (int)experts; a->identity = (int)identity; a->top = (int)top; a->always = (int)always; a->scale = scale;
  a->idx = (int*)idx; a->w = (float*)w; a->idw = (float*)idw;
  return 0;
}

size_t units_smem(const RouteArgs& a, int copies) {
  return sizeof(int) * (size_t)(2 * a.T * (a.top + a.always) + 2 * (a.experts + a.always)) + sizeof(float) * (size_t)copies * kMaxOut;
}
template <int PER>
int launch_units(const RouteArgs& a, const UnitList& u, const RouterProduct* p, cudaStream_t st) {
  if (!p) return (int)cb_launch(routed_units_kernel<PER>, dim3(1), dim3((unsigned)(a.T >= 16 ? 512 : 32 * a.T)), units_smem(a, 0), st, a, u);
  const dim3 grid((unsigned)((a.experts + a.identity + kOut - 1) / kOut));
  const size_t smem = units_smem(a, 8);
  if (a.T == 1) return (int)cb_launch(routed_step_kernel<PER, 1>, grid, dim3(256), smem, st, a, u, *p);
  if (a.T <= 4) return (int)cb_launch(routed_step_kernel<PER, 4>, grid, dim3(256), smem, st, a, u, *p);
  return (int)cb_launch(routed_step_kernel<PER, 8>, grid, dim3(256), smem, st, a, u, *p);
}
#define CB_PER(CALL)                                             \
  const int per_ = (int)((experts + identity + 31) / 32);        \
  if (per_ <= 1) return CALL(1);                                 \
  if (per_ <= 4) return CALL(4);                                 \
  if (per_ <= 10) return CALL(10);                               \
  return CALL(16)

}  // namespace

// Slots of `T` rows: idx / w [T, top + always] (idx -1: no stored expert), idw [T].
CB_EXPORT int cb_routed_topk(const void* logits, int64_t ldl, const void* corr, const void* positions, int64_t T, int64_t experts,
                             int64_t identity, int64_t top, int64_t always, float scale, int64_t by_logit, void* idx, void* w, void* idw,
                             void* stream) {
  RouteArgs a;
  const int rc = route_args(&a, logits, ldl, corr, positions, T, experts, identity, top, always, scale, by_logit, idx, w, idw);
  if (rc) return rc;
#define CB_TOPK(N) (int)cb_launch(routed_topk_kernel<N>, dim3((unsigned)((T + 3) / 4)), dim3(128), 0, (cudaStream_t)stream, a)
  CB_PER(CB_TOPK);
#undef CB_TOPK
}

// The same for T <= 64 rows, with the sorted order (pos [T * slots], src [T * slots]) and the units of up to 8 rows of an expert.
// router / h / ticket given (T <= 8, bf16): logits = router h^T first, by the same launch; ticket: a zeroed counter.
CB_EXPORT int cb_routed_units(const void* logits, int64_t ldl, const void* corr, const void* positions, int64_t T, int64_t experts,
                              int64_t identity, int64_t top, int64_t always, float scale, int64_t by_logit, void* idx, void* w, void* idw, void* pos,
                              void* src, void* count, void* row0, void* rows, void* expert, int64_t max_units, const void* router,
                              const void* h, int64_t ldh, int64_t K, void* ticket, void* stream) {
  RouteArgs a;
  const int rc = route_args(&a, logits, ldl, corr, positions, T, experts, identity, top, always, scale, by_logit, idx, w, idw);
  if (rc) return rc;
  if (T > kMaxRows || units_smem(a, router ? 8 : 0) > 44 * 1024) return CB_ERR_SHAPE;
  if (!pos || !src || !count || !row0 || !rows || !expert || max_units < 1) return CB_ERR_ARG;
  const UnitList u = {(int*)pos, (int*)src, (int*)count, (int*)row0, (int*)rows, (int*)expert, (int)max_units};
  RouterProduct p = {(const bf16*)router, (const bf16*)h, ldh, (int)K, (float*)const_cast<void*>(logits), (unsigned*)ticket};
  if (router && (!h || !ticket || T > 8)) return CB_ERR_ARG;
  if (router && (K % 8 || ldh % 8 || (((uintptr_t)router | (uintptr_t)h) & 15))) return CB_ERR_SHAPE;
#define CB_UNITS(N) launch_units<N>(a, u, router ? &p : nullptr, (cudaStream_t)stream)
  CB_PER(CB_UNITS);
#undef CB_UNITS
}

// fp32 expert product over a unit list (any number of units): y[r] = act(W[expert] x[src[r]]) (src null: x[r]); act as cb_gemv_units.
CB_EXPORT int cb_routed_linear_f32(const void* W, int64_t stride, const void* x, int64_t ldx, void* y, int64_t ldy, int64_t N, int64_t K,
                                   const void* count, const void* row0, const void* rows, const void* expert, const void* src,
                                   int64_t max_units, int64_t act, void* stream) {
  if (!W || !x || !y || !count || !row0 || !rows || !expert || N < 1 || K < 1 || max_units < 1) return CB_ERR_ARG;
  const dim3 grid((unsigned)((N + 7) / 8), (unsigned)(max_units < 4096 ? max_units : 4096));
  return (int)cb_launch(routed_linear_f32_kernel, grid, dim3(256), 0, (cudaStream_t)stream, (const float*)W, stride, (const float*)x, ldx,
                        (float*)y, ldy, (int)N, (int)K, (const int*)count, (const int*)row0, (const int*)rows, (const int*)expert,
                        (const int*)src, (int)act);
}
