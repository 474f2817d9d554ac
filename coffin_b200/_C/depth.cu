// Depth-averaged residual: after every layer the residual becomes a fixed weighted sum of the embedding output and of all
// layer results so far.
//
// A row keeps its results side by side, x [rows, planes, W] fp32: plane 0 is the embedding output, plane i + 1 the
// result of layer i.  The running residual of layer i lives in plane i + 1 from the start (its sublayers add to it in
// place), so a result is never copied.  The averages are taken in blocks: the last layer of a block reads all planes once and
// leaves, for every layer of the next block, the sum of what exists by then in the plane where that layer's average will go;
// inside a block only the partial sum and the few newer planes are read.  One kernel per sublayer boundary: add the sublayer's output, at a layer's end take
// the weighted sum over the planes into the next one, and normalise for the next projection - layer norm (weight, no
// bias) or RMS norm.  Sums and norms are fp32.  Few rows: a cluster of CTAs shares a row's columns and exchanges
// the two sums of the norm through distributed shared memory.
#include "act_type.cuh"
#include "sm100.cuh"

namespace {

constexpr int kT = 256, kWide = 640, kMaxPlanes = 1024, kPrep = 8;

__device__ __forceinline__ float ld_dsmem(const float* p, uint32_t rank) {
  const uint32_t a = sm100::map_to_cta((uint32_t)__cvta_generic_to_shared(p), rank);
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(a) : "memory");
  return v;
}

struct DepthArgs {
  float* x; int64_t ldx;               // row stride (planes * W)
  int plane;                           // the running residual
  const void* y; int64_t ldy;          // sublayer output to add (null: none)
  const float* dwa; int64_t ldw;       // weights of planes 0 .. plane, rows of the following layers behind (null: not a layer's end)
  int first;                           // planes < first are summed up in plane + 1 already (0: nothing is there)
  int prep;                            // following layers whose sums over planes 0 .. plane go to planes plane + 2 ..
  const float* gain; void* h; int64_t ldh;     // normalised rows (h null: none)
  const int* rows;                     // which row feeds output row i (null: row i)
  int W, cols;                         // columns per CTA
  float eps;
  int center, store;
};

// acc += sum over planes j0, j0 + step, ... < n of w[j] * x[j][i .. i + V)
template <int V>
__device__ __forceinline__ void plane_sum(float* acc, const float* __restrict__ xi, int64_t W, const float* w, int j0, int step, int n) {
  constexpr int U = 8;                           // planes requested together
  for (int j = j0; j < n; j += U * step) {
    float f[U][V];
#pragma unroll
    for (int k = 0; k < U; ++k) {
      const bool ok = j + k * step < n;
      const float* p = xi + (int64_t)(j + k * step) * W;
      if (V == 4) {
        const float4 q = ok ? *reinterpret_cast<const float4*>(p) : make_float4(0.f, 0.f, 0.f, 0.f);
        f[k][0] = q.x; f[k][1 % V] = q.y; f[k][2 % V] = q.z; f[k][3 % V] = q.w;
      } else {
        f[k][0] = ok ? *p : 0.f;
      }
    }
#pragma unroll
    for (int k = 0; k < U; ++k) {
      const float c = j + k * step < n ? w[j + k * step] : 0.f;
#pragma unroll
      for (int v = 0; v < V; ++v) acc[v] = fmaf(c, f[k][v], acc[v]);
    }
  }
}
template <int V> __device__ __forceinline__ void ld_f32(float* d, const float* p) {
  if (V == 4) { const float4 q = *reinterpret_cast<const float4*>(p); d[0] = q.x; d[1 % V] = q.y; d[2 % V] = q.z; d[3 % V] = q.w; }
  else d[0] = *p;
}
template <int V> __device__ __forceinline__ void st_f32(float* p, const float* d) {
  if (V == 4) *reinterpret_cast<float4*>(p) = make_float4(d[0], d[1 % V], d[2 % V], d[3 % V]);
  else *p = d[0];
}

// PREP: the sums for the next block of layers as well
template <typename TA, int V, bool PREP>
__global__ void __launch_bounds__(PREP ? kT : kWide, PREP ? 3 : 2) depth_step_kernel(const DepthArgs a) {
  extern __shared__ float v_s[];       // this CTA's columns of the (averaged) residual, then the weights
  __shared__ float red[32];
  __shared__ float cl[2];
  float* w_s = v_s + a.cols;           // [1 + prep][plane + 1]
  const int np1 = a.plane + 1, nT = blockDim.x;
  const int ns = gridDim.x, c0 = blockIdx.x * a.cols, c1 = min(a.W, c0 + a.cols), nc = c1 - c0;
  if (a.dwa)
    for (int k = 0; k <= (PREP ? a.prep : 0); ++k)
      for (int j = threadIdx.x; j <= a.plane; j += nT) w_s[k * np1 + j] = a.dwa[k * a.ldw + j];
  griddep_launch();
  griddep_wait();
  const int64_t r = a.rows ? a.rows[blockIdx.y] : (int64_t)blockIdx.y;
  if (r < 0) return;                   // the same for every CTA of a cluster
  __syncthreads();
  float* xr = a.x + r * a.ldx;
  float* cur = xr + (int64_t)a.plane * a.W;
  const TA* yr = a.y ? reinterpret_cast<const TA*>(a.y) + r * a.ldy : nullptr;
  float s = 0.f;
  auto own = [&](float* u, int i) {    // the running residual with the sublayer's output
    ld_f32<V>(u, cur + i);
    if (!yr) return;
    if (V == 4) {
      const float4 f = act_load4(yr + i);
      u[0] += f.x; u[1 % V] += f.y; u[2 % V] += f.z; u[3 % V] += f.w;
    } else {
      u[0] += act_load(yr + i);
    }
    if (a.store) st_f32<V>(cur + i, u);
  };
  auto keep = [&](const float* u, int i) {
#pragma unroll
    for (int v = 0; v < V; ++v) { v_s[i + v] = u[v]; s += a.center ? u[v] : u[v] * u[v]; }
  };
  for (int i = c0 + threadIdx.x * V; i < c1; i += nT * V) {
    float u[V];
    own(u, i);
    if (a.dwa) {
      float acc[V];
#pragma unroll
      for (int v = 0; v < V; ++v) acc[v] = w_s[a.plane] * u[v];
      if (PREP) {
        float pre[kPrep][V];
#pragma unroll
        for (int k = 0; k < kPrep; ++k)
#pragma unroll
          for (int v = 0; v < V; ++v) pre[k][v] = k < a.prep ? w_s[(1 + k) * np1 + a.plane] * u[v] : 0.f;
        constexpr int U = 4;
        for (int j = 0; j < a.plane; j += U) {
          float f[U][V];
#pragma unroll
          for (int q = 0; q < U; ++q) {
#pragma unroll
            for (int v = 0; v < V; ++v) f[q][v] = 0.f;
            if (j + q < a.plane) ld_f32<V>(f[q], xr + (int64_t)(j + q) * a.W + i);
          }
#pragma unroll
          for (int q = 0; q < U; ++q) {
            const int jj = min(j + q, a.plane);                // past the end: the values are zero
#pragma unroll
            for (int v = 0; v < V; ++v) acc[v] = fmaf(w_s[jj], f[q][v], acc[v]);
#pragma unroll
            for (int k = 0; k < kPrep; ++k) {
              const float w = k < a.prep ? w_s[(1 + k) * np1 + jj] : 0.f;
#pragma unroll
              for (int v = 0; v < V; ++v) pre[k][v] = fmaf(w, f[q][v], pre[k][v]);
            }
          }
        }
#pragma unroll
        for (int k = 0; k < kPrep; ++k)
          if (k < a.prep && a.store) st_f32<V>(cur + (int64_t)(2 + k) * a.W + i, pre[k]);
      } else {
        if (a.first) {
          ld_f32<V>(u, cur + a.W + i);
#pragma unroll
          for (int v = 0; v < V; ++v) acc[v] += u[v];
        }
        plane_sum<V>(acc, xr + i, a.W, w_s, a.first, 1, a.plane);
      }
#pragma unroll
      for (int v = 0; v < V; ++v) u[v] = acc[v];
      if (a.store) st_f32<V>(cur + a.W + i, u);
    }
    keep(u, i - c0);
  }
  if (!a.h) return;
  // mean and squared deviations of this CTA's columns, then of the row (RMS norm: plain squares about zero)
  s = block_sum(s, red);
  float mean = 0.f, m2 = s;
  if (a.center) {
    mean = s / (float)nc;
    float d2 = 0.f;
    for (int i = threadIdx.x; i < nc; i += nT) { const float d = v_s[i] - mean; d2 = fmaf(d, d, d2); }
    m2 = block_sum(d2, red);
  }
  if (ns > 1) {
    if (threadIdx.x == 0) { cl[0] = mean; cl[1] = m2; }
    sm100::cluster_sync_all();
    float mq[8], vq[8], tot = 0.f;
#pragma unroll
    for (int q = 0; q < 8; ++q) {
      mq[q] = q < ns ? ld_dsmem(&cl[0], q) : 0.f;
      vq[q] = q < ns ? ld_dsmem(&cl[1], q) : 0.f;
      tot += mq[q] * (float)max(0, min(a.W, (q + 1) * a.cols) - q * a.cols);
    }
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");    // this CTA has read what it needs
    mean = tot / (float)a.W;
    m2 = 0.f;
#pragma unroll
    for (int q = 0; q < 8; ++q) {
      const float d = mq[q] - mean;
      m2 += vq[q] + (a.center ? d * d * (float)max(0, min(a.W, (q + 1) * a.cols) - q * a.cols) : 0.f);
    }
    if (!a.center) mean = 0.f;
  }
  const float rstd = 1.f / sqrtf(m2 / (float)a.W + a.eps);
  TA* hr = reinterpret_cast<TA*>(a.h) + (int64_t)blockIdx.y * a.ldh;
  for (int i = threadIdx.x * V; i < nc; i += nT * V) {
    if (V == 4) {
      const float4 g = *reinterpret_cast<const float4*>(a.gain + c0 + i);
      act_store4(hr + c0 + i, make_float4((v_s[i] - mean) * rstd * g.x, (v_s[i + 1 % V] - mean) * rstd * g.y,
                                          (v_s[i + 2 % V] - mean) * rstd * g.z, (v_s[i + 3 % V] - mean) * rstd * g.w));
    } else {
      act_store(hr + c0 + i, (v_s[i] - mean) * rstd * a.gain[c0 + i]);
    }
  }
  if (ns > 1) asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");     // nobody leaves while its sums may still be read
}

// planes 0 and 1 of row t = embed[token[t]] * scale
template <typename TA>
__global__ void __launch_bounds__(kT) depth_embed_kernel(const TA* __restrict__ embed, const int64_t* __restrict__ tokens,
                                                         float* __restrict__ x, int64_t ldx, int W, int64_t V, float scale) {
  griddep_launch();
  griddep_wait();
  const int64_t r = blockIdx.x;
  int64_t tok = tokens[r];
  tok = tok < 0 ? 0 : (tok >= V ? V - 1 : tok);
  const TA* e = embed + tok * W;
  float* xr = x + r * ldx;
  if (W % 4 == 0 && ldx % 4 == 0) {
    for (int i = threadIdx.x * 4; i < W; i += kT * 4) {
      float4 v = act_load4(e + i);
      v.x *= scale; v.y *= scale; v.z *= scale; v.w *= scale;
      *reinterpret_cast<float4*>(xr + i) = v;
      *reinterpret_cast<float4*>(xr + W + i) = v;
    }
    return;
  }
  for (int i = threadIdx.x; i < W; i += kT) xr[i] = xr[W + i] = act_load(e + i) * scale;
}

template <typename TA>
int launch_depth(DepthArgs a, int64_t n, cudaStream_t st) {
  const bool v4 = a.W % 4 == 0 && a.ldx % 4 == 0 && a.ldh % 4 == 0 && a.ldy % 4 == 0;
  // a row with many planes to read is shared by a cluster of CTAs while SMs are idle; otherwise few rows get wide blocks
  int ns = 1;
  if (a.dwa && a.plane - a.first > 12)
    while (ns < 8 && n * ns * 2 <= 148 && a.W / (ns * 2) >= 256) ns <<= 1;
  a.cols = ((a.W + ns - 1) / ns + 3) & ~3;
  ns = (a.W + a.cols - 1) / a.cols;
  const int units = v4 ? (a.cols + 3) / 4 : a.cols;
  int threads = kT;
  if (!a.prep && n <= 148) {
    threads = (units + 31) & ~31;
    threads = threads < kT ? kT : (threads > kWide ? kWide : threads);
  }
  auto kern = a.prep ? (v4 ? depth_step_kernel<TA, 4, true> : depth_step_kernel<TA, 1, true>)
                     : (v4 ? depth_step_kernel<TA, 4, false> : depth_step_kernel<TA, 1, false>);
  const size_t smem = ((size_t)a.cols + (a.dwa ? (size_t)(1 + a.prep) * (a.plane + 1) : 0)) * sizeof(float);
  if (smem > 200 * 1024) return CB_ERR_SHAPE;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)ns, (unsigned)n);
  cfg.blockDim = dim3((unsigned)threads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  int na = 0;
  if (ns > 1) {
    attr[na].id = cudaLaunchAttributeClusterDimension;
    attr[na].val.clusterDim.x = (unsigned)ns; attr[na].val.clusterDim.y = 1; attr[na].val.clusterDim.z = 1;
    ++na;
  }
  if (g_cb_use_pdl) {
    attr[na].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[na].val.programmaticStreamSerializationAllowed = 1;
    ++na;
  }
  cfg.attrs = attr;
  cfg.numAttrs = na;
  if (g_cb_trace_names) cb_trace_name((const void*)kern);
  return (int)cudaLaunchKernelEx(&cfg, kern, a);
}

}  // namespace

// One sublayer boundary over `n` rows of x [*, ldx]: plane `plane` += y (y null: nothing), with dwa the weighted sum of
// planes 0 .. plane goes to plane + 1 (first > 0: planes < first are summed up there already), the sums of the next `prep`
// layers over these planes to the planes behind (their weights in the rows of dwa, ldw apart), and h = norm(the result) * gain
// (center: layer norm, else RMS norm).  `rows`
// (int32 [n]): which row feeds output row i; `store` 0: x is left as it is.  f32: y and h are fp32 instead of bf16.
CB_EXPORT int cb_depth_step(void* x, int64_t ldx, int64_t plane, const void* y, int64_t ldy, const void* dwa, int64_t ldw,
                            int64_t first, int64_t prep, const void* gain, void* h, int64_t ldh, const void* rows, int64_t n, int64_t W, float eps, int64_t center, int64_t store,
                            int64_t f32, void* stream) {
  if (!x || n < 1 || n > 65535 || W < 1 || plane < 0 || plane >= kMaxPlanes || (h && !gain) || (rows && store)) return CB_ERR_ARG;
  if (prep < 0 || prep > kPrep || first < 0 || first > plane || ((prep || first) && !dwa) || (prep && first)) return CB_ERR_ARG;
  if (ldx < (plane + (dwa && store ? 2 + prep : (first ? 2 : 1))) * W) return CB_ERR_ARG;
  DepthArgs a;
  a.x = (float*)x; a.ldx = ldx; a.plane = (int)plane; a.y = y; a.ldy = ldy; a.dwa = (const float*)dwa; a.ldw = ldw;
  a.first = (int)first; a.prep = (int)prep; a.gain = (const float*)gain;
  a.h = h; a.ldh = ldh; a.rows = (const int*)rows; a.W = (int)W; a.cols = 0; a.eps = eps; a.center = (int)center; a.store = (int)store;
  return f32 ? launch_depth<float>(a, n, (cudaStream_t)stream) : launch_depth<bf16>(a, n, (cudaStream_t)stream);
}

CB_EXPORT int cb_depth_embed(const void* embed, const void* tokens, void* x, int64_t ldx, int64_t T, int64_t W, int64_t V, float scale,
                             int64_t f32, void* stream) {
  if (!embed || !tokens || !x || T < 1 || W < 1 || ldx < 2 * W) return CB_ERR_ARG;
  cudaStream_t st = (cudaStream_t)stream;
  if (f32)
    return (int)cb_launch(depth_embed_kernel<float>, dim3((unsigned)T), dim3(kT), 0, st, (const float*)embed, (const int64_t*)tokens,
                          (float*)x, ldx, (int)W, V, scale);
  return (int)cb_launch(depth_embed_kernel<bf16>, dim3((unsigned)T), dim3(kT), 0, st, (const bf16*)embed, (const int64_t*)tokens,
                        (float*)x, ldx, (int)W, V, scale);
}
