// Depth-averaged residual: after every layer the residual becomes a fixed weighted sum of the embedding output and of all
// layer results so far.
//
// A row keeps its results side by side, x [rows, planes, W] fp32: plane 0 is the embedding output, plane i + 1 the
// result of layer i.  The running residual of layer i lives in plane i + 1 from the start (its sublayers add to it in
// place), so a result is never copied.  One kernel per sublayer boundary: add the sublayer's output, at a layer's end take
// the weighted sum over the planes into the next one, and normalise for the next projection - layer norm (weight, no
// bias) or RMS norm.  Sums and norms are fp32.  Few rows: a cluster of CTAs shares a row's columns and exchanges
// the two sums of the norm through distributed shared memory.
#include "act_type.cuh"
#include "sm100.cuh"

namespace {

constexpr int kT = 256;

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
  const float* dwa;                    // weights of planes 0 .. plane (null: not a layer's end)
  const float* gain; void* h; int64_t ldh;     // normalised rows (h null: none)
  const int* rows;                     // which row feeds output row i (null: row i)
  int W, cols;                         // columns per CTA
  float eps;
  int center, store;
};

template <typename TA, int V>
__global__ void __launch_bounds__(kT) depth_step_kernel(const DepthArgs a) {
  extern __shared__ float v_s[];       // this CTA's columns of the (averaged) residual
  __shared__ float red[32], w_s[256];
  __shared__ float cl[2];
  const int ns = gridDim.x, c0 = blockIdx.x * a.cols, c1 = min(a.W, c0 + a.cols);
  if (a.dwa)
    for (int j = threadIdx.x; j <= a.plane && j < 256; j += kT) w_s[j] = a.dwa[j];
  griddep_launch();
  griddep_wait();
  const int64_t r = a.rows ? a.rows[blockIdx.y] : (int64_t)blockIdx.y;
  if (r < 0) return;                   // the same for every CTA of a cluster
  __syncthreads();
  float* xr = a.x + r * a.ldx;
  float* cur = xr + (int64_t)a.plane * a.W;
  const TA* yr = a.y ? reinterpret_cast<const TA*>(a.y) + r * a.ldy : nullptr;
  float s = 0.f;
  for (int i = c0 + threadIdx.x * V; i < c1; i += kT * V) {
    float u[V];
    if (V == 4) {
      const float4 f = *reinterpret_cast<const float4*>(cur + i);
      u[0] = f.x; u[1 % V] = f.y; u[2 % V] = f.z; u[3 % V] = f.w;
    } else {
      u[0] = cur[i];
    }
    if (yr) {
      if (V == 4) {
        const float4 f = act_load4(yr + i);
        u[0] += f.x; u[1 % V] += f.y; u[2 % V] += f.z; u[3 % V] += f.w;
      } else {
        u[0] += act_load(yr + i);
      }
      if (a.store) {
        if (V == 4) *reinterpret_cast<float4*>(cur + i) = make_float4(u[0], u[1 % V], u[2 % V], u[3 % V]);
        else cur[i] = u[0];
      }
    }
    if (a.dwa) {
      float acc[V];
      const float wl = a.plane < 256 ? w_s[a.plane] : a.dwa[a.plane];
#pragma unroll
      for (int v = 0; v < V; ++v) acc[v] = wl * u[v];
      const float* p = xr + i;
      int j = 0;
      for (; j + 8 <= a.plane; j += 8) {                         // eight planes requested together
        float f[8][V];
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          if (V == 4) {
            const float4 q = *reinterpret_cast<const float4*>(p + (int64_t)(j + k) * a.W);
            f[k][0] = q.x; f[k][1 % V] = q.y; f[k][2 % V] = q.z; f[k][3 % V] = q.w;
          } else {
            f[k][0] = p[(int64_t)(j + k) * a.W];
          }
        }
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          const float w = j + k < 256 ? w_s[j + k] : a.dwa[j + k];
#pragma unroll
          for (int v = 0; v < V; ++v) acc[v] = fmaf(w, f[k][v], acc[v]);
        }
      }
#pragma unroll 1
      for (; j < a.plane; ++j) {
        const float w = j < 256 ? w_s[j] : a.dwa[j];
        if (V == 4) {
          const float4 q = *reinterpret_cast<const float4*>(p + (int64_t)j * a.W);
          acc[0] = fmaf(w, q.x, acc[0]); acc[1 % V] = fmaf(w, q.y, acc[1 % V]);
          acc[2 % V] = fmaf(w, q.z, acc[2 % V]); acc[3 % V] = fmaf(w, q.w, acc[3 % V]);
        } else {
          acc[0] = fmaf(w, p[(int64_t)j * a.W], acc[0]);
        }
      }
#pragma unroll
      for (int v = 0; v < V; ++v) u[v] = acc[v];
      if (a.store) {
        if (V == 4) *reinterpret_cast<float4*>(cur + a.W + i) = make_float4(u[0], u[1 % V], u[2 % V], u[3 % V]);
        else cur[a.W + i] = u[0];
      }
    }
#pragma unroll
    for (int v = 0; v < V; ++v) { v_s[i - c0 + v] = u[v]; s += a.center ? u[v] : u[v] * u[v]; }
  }
  if (!a.h) return;
  // first sum: the mean (layer norm) or the mean square; second: squared deviations
  auto row_sum = [&](float v, int k) {
    v = block_sum(v, red);
    if (ns == 1) return v;
    if (threadIdx.x == 0) cl[k] = v;
    sm100::cluster_sync_all();
    float t = 0.f;
    for (int q = 0; q < ns; ++q) t += ld_dsmem(&cl[k], q);
    return t;
  };
  float m = row_sum(s, 0) / (float)a.W, mean = 0.f, rstd;
  if (a.center) {
    mean = m;
    float d2 = 0.f;
    for (int i = threadIdx.x * V; i < c1 - c0; i += kT * V)      // each thread re-reads what it wrote
#pragma unroll
      for (int v = 0; v < V; ++v) { const float d = v_s[i + v] - mean; d2 = fmaf(d, d, d2); }
    m = row_sum(d2, 1) / (float)a.W;
  }
  rstd = 1.f / sqrtf(m + a.eps);
  TA* hr = reinterpret_cast<TA*>(a.h) + (int64_t)blockIdx.y * a.ldh;
  for (int i = threadIdx.x * V; i < c1 - c0; i += kT * V) {
    if (V == 4) {
      const float4 g = *reinterpret_cast<const float4*>(a.gain + c0 + i);
      act_store4(hr + c0 + i, make_float4((v_s[i] - mean) * rstd * g.x, (v_s[i + 1 % V] - mean) * rstd * g.y,
                                          (v_s[i + 2 % V] - mean) * rstd * g.z, (v_s[i + 3 % V] - mean) * rstd * g.w));
    } else {
      act_store(hr + c0 + i, (v_s[i] - mean) * rstd * a.gain[c0 + i]);
    }
  }
  if (ns > 1) sm100::cluster_sync_all();         // nobody leaves while its sums may still be read
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
  for (int i = threadIdx.x; i < W; i += kT) {
    const float v = act_load(embed + tok * W + i) * scale;
    x[r * ldx + i] = v;
    x[r * ldx + W + i] = v;
  }
}

template <typename TA>
int launch_depth(DepthArgs a, int64_t n, cudaStream_t st) {
  const bool v4 = a.W % 4 == 0 && a.ldx % 4 == 0 && a.ldh % 4 == 0 && a.ldy % 4 == 0;
  int ns = 1;
  while (ns < 8 && n * ns * 2 <= 148 && a.W / (ns * 2) >= 256) ns <<= 1;
  a.cols = ((a.W + ns - 1) / ns + 3) & ~3;
  ns = (a.W + a.cols - 1) / a.cols;
  auto kern = v4 ? depth_step_kernel<TA, 4> : depth_step_kernel<TA, 1>;
  const size_t smem = (size_t)a.cols * sizeof(float);
  if (smem > 200 * 1024) return CB_ERR_SHAPE;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)ns, (unsigned)n);
  cfg.blockDim = dim3(kT);
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
// planes 0 .. plane goes to plane + 1, and h = norm(the result) * gain (center: layer norm, else RMS norm).  `rows`
// (int32 [n]): which row feeds output row i; `store` 0: x is left as it is.  f32: y and h are fp32 instead of bf16.
CB_EXPORT int cb_depth_step(void* x, int64_t ldx, int64_t plane, const void* y, int64_t ldy, const void* dwa, const void* gain,
                            void* h, int64_t ldh, const void* rows, int64_t n, int64_t W, float eps, int64_t center, int64_t store,
                            int64_t f32, void* stream) {
  if (!x || n < 1 || n > 65535 || W < 1 || plane < 0 || (h && !gain) || (rows && store)) return CB_ERR_ARG;
  if (ldx < (plane + (dwa && store ? 2 : 1)) * W) return CB_ERR_ARG;
  DepthArgs a;
  a.x = (float*)x; a.ldx = ldx; a.plane = (int)plane; a.y = y; a.ldy = ldy; a.dwa = (const float*)dwa; a.gain = (const float*)gain;
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
