// Rotary positions of the row-batch families: the angles of a batch, and neighbouring pairs of head parts turned by them.
#include "act_type.cuh"

namespace {

// cs[row, i] = (cos, sin) of position * freq_i, freq in turns (fp64: the turn count is reduced exactly, whatever the position)
__global__ void __launch_bounds__(256) rope_rows_kernel(const int* __restrict__ positions, const double* __restrict__ turns,
                                                        float2* __restrict__ cs, int rows, int half) {
  griddep_launch();
  griddep_wait();
  const int e = blockIdx.x * 256 + threadIdx.x;
  if (e >= rows * half) return;
  const double t = (double)max(positions[e / half], 0) * turns[e % half];
  float s, c;
  sincospif(2.f * (float)(t - rint(t)), &s, &c);
  cs[e] = make_float2(c, s);
}

// rotated query parts: src [rows, heads] at column off of each head -> dst (the same place, or the absorbed query)
template <typename TS, typename TA>
__global__ void __launch_bounds__(256) rope_heads_kernel(const TS* __restrict__ src, int64_t lds, int64_t hs, TA* __restrict__ dst,
                                                         int64_t ldd, int64_t hd, const float2* __restrict__ cs, int half, int rot, int H,
                                                         int rows) {
  griddep_launch();
  griddep_wait();
  const int np = (rot + 1) / 2;
  const int64_t e = (int64_t)blockIdx.x * 256 + threadIdx.x;
  if (e >= (int64_t)rows * H * np) return;
  const int i = (int)(e % np), h = (int)(e / np % H);
  const int64_t row = e / np / H;
  const TS* s = src + row * lds + h * hs + 2 * i;
  TA* d = dst + row * ldd + h * hd + 2 * i;
  const bool two = 2 * i + 1 < rot;
  float u = act_load(s), v = two ? act_load(s + 1) : 0.f;
  if (i < half) {
    const float2 c = cs[row * half + i];
    const float x = u * c.x - v * c.y;
    v = v * c.x + u * c.y;
    u = x;
  }
  act_store(d, u);
  if (two) act_store(d + 1, v);
}

}  // namespace

// (cos, sin) of position * turns[i] turns, for `rows` rows: cs [rows, half, 2] fp32; turns fp64 [half].
CB_EXPORT int cb_rope_rows(const void* positions, const void* turns, void* cs, int64_t rows, int64_t half, void* stream) {
  if (!positions || !turns || !cs || rows < 1 || half < 1 || rows * half > (int64_t)1 << 30) return CB_ERR_ARG;
  return (int)cb_launch(rope_rows_kernel, dim3((unsigned)((rows * half + 255) / 256)), dim3(256), 0, (cudaStream_t)stream,
                        (const int*)positions, (const double*)turns, (float2*)cs, (int)rows, (int)half);
}

// Rotated parts of `H` heads: dst[t, h] = rotate(src[t, h]) (row strides lds / ldd, head strides hs / hd); may be in place.
CB_EXPORT int cb_rope_heads(const void* src, int64_t lds, int64_t hs, void* dst, int64_t ldd, int64_t hd, const void* cs, int64_t half,
                            int64_t rot, int64_t H, int64_t rows, int64_t f32, void* stream) {
  if (!src || !dst || rows < 1 || H < 1 || rot < 1 || 2 * half > rot || (half && !cs)) return CB_ERR_ARG;
  const dim3 grid((unsigned)((rows * H * ((rot + 1) / 2) + 255) / 256)), block(256);
  cudaStream_t st = (cudaStream_t)stream;
  if (f32)
    return (int)cb_launch(rope_heads_kernel<float, float>, grid, block, 0, st, (const float*)src, lds, hs, (float*)dst, ldd, hd,
                          (const float2*)cs, (int)half, (int)rot, (int)H, (int)rows);
  return (int)cb_launch(rope_heads_kernel<bf16, bf16>, grid, block, 0, st, (const bf16*)src, lds, hs, (bf16*)dst, ldd, hd,
                        (const float2*)cs, (int)half, (int)rot, (int)H, (int)rows);
}
