// Static hyper-connections: the residual is `S` fp32 streams instead of one vector.
//
// A sublayer reads a fixed mix of the streams (u = sum_s in[s] x_s), and its output y is written back into all
// of them together with a fixed S x S mixing of the old ones (x_t <- sum_s mix[s, t] x_s + out[t] y).  The
// write-back of one sublayer and the read + RMS norm of the next touch the same rows, so they are one kernel:
// the streams cross HBM once per sublayer.  Sums, norm and streams are fp32; only the normalised row that
// feeds the next projection leaves in the activation type.  The input-dependent lanes of the Qwen4-exp family
// are qwen4.cu's hyper_norm / hyper_up.
#include "act_type.cuh"

namespace {

constexpr int kT = 256;

template <int S, typename TA, int V>
__global__ void __launch_bounds__(kT) streams_step_kernel(float* __restrict__ x, const TA* __restrict__ y, int64_t ldy,
                                                          const float* __restrict__ mix, const float* __restrict__ outw,
                                                          const float* __restrict__ inw, const float* __restrict__ gain,
                                                          TA* __restrict__ h, int64_t ldh, const int* __restrict__ rows,
                                                          int W, float eps, int store) {
  extern __shared__ float u_s[];        // the mixed row
  __shared__ float red[32];
  float m[S][S], o[S], in[S];
#pragma unroll
  for (int s = 0; s < S; ++s) {
    in[s] = inw ? inw[s] : 1.f;
    o[s] = outw ? outw[s] : 0.f;
#pragma unroll
    for (int t = 0; t < S; ++t) m[s][t] = mix ? mix[s * S + t] : (s == t ? 1.f : 0.f);
  }
  griddep_launch();
  griddep_wait();
  const int64_t r = rows ? rows[blockIdx.x] : (int64_t)blockIdx.x;
  if (r < 0) return;
  float* xr = x + r * S * W;
  const TA* yr = y ? y + r * ldy : nullptr;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < W; i += kT * V) {
    float xs[S][V], yv[V], u[V];
    if (V == 4) {
#pragma unroll
      for (int s = 0; s < S; ++s) {
        const float4 f = *reinterpret_cast<const float4*>(xr + (int64_t)s * W + i);
        xs[s][0] = f.x; xs[s][1 % V] = f.y; xs[s][2 % V] = f.z; xs[s][3 % V] = f.w;
      }
      float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
      if (yr) f = act_load4(yr + i);
      yv[0] = f.x; yv[1 % V] = f.y; yv[2 % V] = f.z; yv[3 % V] = f.w;
    } else {
#pragma unroll
      for (int s = 0; s < S; ++s) xs[s][0] = xr[(int64_t)s * W + i];
      yv[0] = yr ? act_load(yr + i) : 0.f;
    }
#pragma unroll
    for (int v = 0; v < V; ++v) u[v] = 0.f;
    if (yr) {
      float nx[S][V];
#pragma unroll
      for (int t = 0; t < S; ++t) {
#pragma unroll
        for (int v = 0; v < V; ++v) {
          float a = o[t] * yv[v];
#pragma unroll
          for (int s = 0; s < S; ++s) a = fmaf(m[s][t], xs[s][v], a);
          nx[t][v] = a;
        }
        if (store) {
          if (V == 4) *reinterpret_cast<float4*>(xr + (int64_t)t * W + i) = make_float4(nx[t][0], nx[t][1 % V], nx[t][2 % V], nx[t][3 % V]);
          else xr[(int64_t)t * W + i] = nx[t][0];
        }
      }
#pragma unroll
      for (int s = 0; s < S; ++s)
#pragma unroll
        for (int v = 0; v < V; ++v) u[v] = fmaf(in[s], nx[s][v], u[v]);
    } else {
#pragma unroll
      for (int s = 0; s < S; ++s)
#pragma unroll
        for (int v = 0; v < V; ++v) u[v] = fmaf(in[s], xs[s][v], u[v]);
    }
#pragma unroll
    for (int v = 0; v < V; ++v) { u_s[i + v] = u[v]; ss = fmaf(u[v], u[v], ss); }
  }
  if (!h) return;
  const float rstd = 1.f / sqrtf(block_sum(ss, red) / (float)W + eps);
  TA* hr = h + (int64_t)blockIdx.x * ldh;
  for (int i = threadIdx.x * V; i < W; i += kT * V) {            // each thread re-reads what it wrote
    if (V == 4) {
      const float4 g = *reinterpret_cast<const float4*>(gain + i);
      act_store4(hr + i, make_float4(u_s[i] * rstd * g.x, u_s[i + 1] * rstd * g.y, u_s[i + 2] * rstd * g.z, u_s[i + 3] * rstd * g.w));
    } else {
      act_store(hr + i, u_s[i] * rstd * gain[i]);
    }
  }
}

// x[t, s, :] = embed[token[t]] + pos[position[t]] for every stream s
template <typename TA>
__global__ void __launch_bounds__(kT) streams_embed_kernel(const TA* __restrict__ embed, const TA* __restrict__ pos,
                                                           const int64_t* __restrict__ tokens, const int* __restrict__ positions,
                                                           float* __restrict__ x, int S, int W, int64_t V, int64_t P) {
  griddep_launch();
  griddep_wait();
  const int64_t r = blockIdx.x;
  int64_t tok = tokens[r];
  tok = tok < 0 ? 0 : (tok >= V ? V - 1 : tok);
  int64_t p = positions[r];
  p = p < 0 ? 0 : (p >= P ? P - 1 : p);
  for (int i = threadIdx.x; i < W; i += kT) {
    float v = act_load(embed + tok * W + i);
    if (pos) v += act_load(pos + p * W + i);
    for (int s = 0; s < S; ++s) x[(r * S + s) * W + i] = v;
  }
}

template <int S, typename TA>
int step_launch(float* x, const void* y, int64_t ldy, const float* mix, const float* outw, const float* inw, const float* gain,
                void* h, int64_t ldh, const int* rows, int64_t n, int64_t W, float eps, int64_t store, cudaStream_t st) {
  const bool v4 = W % 4 == 0 && ldh % 4 == 0 && ldy % 4 == 0;
  auto kern = v4 ? streams_step_kernel<S, TA, 4> : streams_step_kernel<S, TA, 1>;
  const size_t smem = (size_t)W * sizeof(float);
  if (smem > 200 * 1024) return CB_ERR_SHAPE;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return (int)cb_launch(kern, dim3((unsigned)n), dim3(kT), smem, st, x, (const TA*)y, ldy, mix, outw, inw, gain, (TA*)h, ldh, rows,
                        (int)W, eps, (int)store);
}

}  // namespace

// One sublayer boundary over `n` rows: apply the pending write-back (y, mix, outw; y null: none), then
// h = rmsnorm(sum_s inw[s] x_s) * gain.  `inw` null: plain sum of the streams (the end of the stack).  `rows`
// (int32 [n], optional): which stream row feeds output row i.  `store` 0: the streams are not updated.
// `h` null: write-back only.  f32: activations (y, h) are fp32 instead of bf16.
CB_EXPORT int cb_streams_step(void* x, const void* y, int64_t ldy, const void* mix, const void* outw, const void* inw,
                              const void* gain, void* h, int64_t ldh, const void* rows, int64_t n, int64_t S, int64_t W,
                              float eps, int64_t store, int64_t f32, void* stream) {
  if (!x || n < 1 || W < 1 || S < 1 || S > 8 || (y && (!mix || !outw)) || (h && !gain)) return CB_ERR_ARG;
  if (rows && store) return CB_ERR_ARG;
  cudaStream_t st = (cudaStream_t)stream;
#define CB_STEP(N)                                                                                                              \
  case N:                                                                                                                       \
    return f32 ? step_launch<N, float>((float*)x, y, ldy, (const float*)mix, (const float*)outw, (const float*)inw,             \
                                       (const float*)gain, h, ldh, (const int*)rows, n, W, eps, store, st)                      \
               : step_launch<N, bf16>((float*)x, y, ldy, (const float*)mix, (const float*)outw, (const float*)inw,              \
                                      (const float*)gain, h, ldh, (const int*)rows, n, W, eps, store, st);
  switch (S) { CB_STEP(1) CB_STEP(2) CB_STEP(3) CB_STEP(4) CB_STEP(5) CB_STEP(6) CB_STEP(7) CB_STEP(8) }
#undef CB_STEP
  return CB_ERR_ARG;
}

CB_EXPORT int cb_streams_embed(const void* embed, const void* pos, const void* tokens, const void* positions, void* x, int64_t T,
                               int64_t S, int64_t W, int64_t V, int64_t P, int64_t f32, void* stream) {
  if (!embed || !tokens || !positions || !x || T < 1 || S < 1 || W < 1) return CB_ERR_ARG;
  cudaStream_t st = (cudaStream_t)stream;
  if (f32)
    return (int)cb_launch(streams_embed_kernel<float>, dim3((unsigned)T), dim3(kT), 0, st, (const float*)embed, (const float*)pos,
                          (const int64_t*)tokens, (const int*)positions, (float*)x, (int)S, (int)W, V, P);
  return (int)cb_launch(streams_embed_kernel<bf16>, dim3((unsigned)T), dim3(kT), 0, st, (const bf16*)embed, (const bf16*)pos,
                        (const int64_t*)tokens, (const int*)positions, (float*)x, (int)S, (int)W, V, P);
}
