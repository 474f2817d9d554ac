// fp32 projections: C[M, N] = A[M, K] x W[N, K]^T in true 32-bit (no TF32), any sizes and strides.
//
// The serving mode multiplies bf16 on the tensor cores; this kernel is the 32-bit mode of a model (the sharper
// numerics check of everything around the products).  64 x 64 tiles, 4 x 4 outputs per thread, operands
// staged through shared memory.
#include "act_type.cuh"

namespace {

constexpr int TM = 64, TN = 64, TK = 16;

__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ A, int64_t lda, const float* __restrict__ W,
                                                       int64_t ldw, float* __restrict__ C, int64_t ldc, int64_t M, int64_t N,
                                                       int64_t K) {
  __shared__ float as[TK][TM + 4], ws[TK][TN + 4];
  griddep_launch();
  griddep_wait();
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int64_t m0 = (int64_t)blockIdx.y * TM, n0 = (int64_t)blockIdx.x * TN;
  float acc[4][4] = {};
  for (int64_t k0 = 0; k0 < K; k0 += TK) {
    for (int e = tid; e < TM * TK; e += 256) {
      const int r = e / TK, k = e % TK;
      as[k][r] = (m0 + r < M && k0 + k < K) ? A[(m0 + r) * lda + k0 + k] : 0.f;
      ws[k][r] = (n0 + r < N && k0 + k < K) ? W[(n0 + r) * ldw + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < TK; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = as[k][ty * 4 + i]; b[i] = ws[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int64_t r = m0 + ty * 4 + i, c = n0 + tx * 4 + j;
      if (r < M && c < N) C[r * ldc + c] = acc[i][j];
    }
}

__global__ void __launch_bounds__(256) swiglu_f32_kernel(const float* __restrict__ gu, int64_t ldg, float* __restrict__ out,
                                                         int64_t ldo, int64_t I) {
  griddep_launch();
  griddep_wait();
  const float* g = gu + (int64_t)blockIdx.x * ldg;
  float* o = out + (int64_t)blockIdx.x * ldo;
  for (int64_t i = threadIdx.x; i < I; i += 256) o[i] = silu_x(g[i]) * g[I + i];
}

__global__ void __launch_bounds__(256) xielu_f32_kernel(const float* __restrict__ x, int64_t ldx, float* __restrict__ out, int64_t ldo,
                                                        int64_t I, float a, float b) {
  griddep_launch();
  griddep_wait();
  const float* r = x + (int64_t)blockIdx.x * ldx;
  float* o = out + (int64_t)blockIdx.x * ldo;
  for (int64_t i = threadIdx.x; i < I; i += 256) o[i] = xielu_x(r[i], a, b);
}

}  // namespace

CB_EXPORT int cb_gemm_f32(const void* A, int64_t lda, const void* W, int64_t ldw, void* C, int64_t ldc, int64_t M, int64_t N,
                          int64_t K, void* stream) {
  if (!A || !W || !C || M < 1 || N < 1 || K < 1) return CB_ERR_ARG;
  const dim3 grid((unsigned)((N + TN - 1) / TN), (unsigned)((M + TM - 1) / TM));
  if (grid.y > 65535) return CB_ERR_SHAPE;
  return (int)cb_launch(gemm_f32_kernel, grid, dim3(256), 0, (cudaStream_t)stream, (const float*)A, lda, (const float*)W, ldw,
                        (float*)C, ldc, M, N, K);
}

// out[M, I] = silu(gu[:, :I]) * gu[:, I:2I], fp32
CB_EXPORT int cb_swiglu_f32(const void* gu, int64_t ldg, void* out, int64_t ldo, int64_t M, int64_t I, void* stream) {
  if (!gu || !out || M < 1 || I < 1) return CB_ERR_ARG;
  return (int)cb_launch(swiglu_f32_kernel, dim3((unsigned)M), dim3(256), 0, (cudaStream_t)stream, (const float*)gu, ldg,
                        (float*)out, ldo, I);
}

// out = xIELU(x) with the coefficients (a, b) of its two branches, fp32 (may be in place)
CB_EXPORT int cb_xielu_f32(const void* x, int64_t ldx, void* out, int64_t ldo, int64_t M, int64_t I, float a, float b, void* stream) {
  if (!x || !out || M < 1 || I < 1) return CB_ERR_ARG;
  return (int)cb_launch(xielu_f32_kernel, dim3((unsigned)M), dim3(256), 0, (cudaStream_t)stream, (const float*)x, ldx, (float*)out,
                        ldo, I, a, b);
}
