// Products of expert units: up to 8 rows of one expert share one pass over its weights, dot products on the tensor cores.
//
// How many units there are is known on the device only (routed.cu), so the grid does not follow it: the work items, all
// 16-row blocks of all units, are divided evenly among the CTAs that are resident.  A CTA's eight warps share a block by
// K; the next block's weights are requested before the sums of the current one are exchanged.  As in gemv_mma.cu a lane's
// 16-byte pieces of weight rows g and g + 8 are its A fragments of two MMAs, with the k index permuted alike in B.
//
// Two of these run back to back (ups, then downs) over one unit list.  The first releases its dependents after its own wait, so
// the list is complete when the second starts: with `early` it reads the list (past L1) and requests weights ahead of its wait.
#include "act_type.cuh"

namespace {

constexpr int kT = 256, kWarps = kT / 32, kU = 4, kPad = 32;     // kU: pairs of 32 elements in flight per lane
constexpr int kMS = 20, kPart = 8 * kMS;                         // sums of one warp: [8 rows][16 outputs], padded

struct UnitArgs {
  const bf16* W; int64_t stride;         // [experts, N, K]
  const bf16* x; int64_t ldx; bf16* y; int64_t ldy;
  const int* count; const int* row0; const int* rows; const int* expert;
  const int* src;                        // row of x behind sorted row r (null: r)
  int N, K, act, early, max_rows;
};

__device__ __forceinline__ void mma(float* c, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// GATED: an expert has N gate rows, then N up rows; a block is 8 outputs, its gate rows are fragments g, its up rows g + 8.
template <bool GATED>
__global__ void __launch_bounds__(kT, 3) gemv_units_kernel(const UnitArgs a) {
  constexpr int kOut = GATED ? 8 : 16;                           // outputs of a block
  extern __shared__ __align__(16) unsigned char smem[];
  float* part = reinterpret_cast<float*>(smem);                  // [2][kWarps][kPart]
  bf16* xs = reinterpret_cast<bf16*>(part + 2 * kWarps * kPart); // [max_rows][K + kPad]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int nchunk = a.K >> 3, npair = (nchunk + 3) >> 2, per = (npair + kWarps - 1) / kWarps;
  const int p0 = warp * per, p1 = min(npair, p0 + per), nblk = (a.N + kOut - 1) / kOut, ldxs = a.K + kPad;
  if (!a.early) griddep_wait();
  griddep_launch();
  const int64_t total = (int64_t)__ldcg(a.count) * nblk;
  const int lo = (int)(total * blockIdx.x / gridDim.x), hi = (int)(total * (blockIdx.x + 1) / gridDim.x);
  const uint4 z = make_uint4(0, 0, 0, 0);
  uint4 wl[kU], wh[kU];
  // rows of block `blk` that this lane loads, of expert e
  auto block = [&](int e, int blk, const bf16** lo_, const bf16** hi_) {
    const bf16* w = a.W + (int64_t)e * a.stride;
    *lo_ = w + (int64_t)min(blk * kOut + g, a.N - 1) * a.K;
    *hi_ = w + (int64_t)(GATED ? a.N + min(blk * kOut + g, a.N - 1) : min(blk * kOut + g + 8, a.N - 1)) * a.K;
  };
  auto load = [&](const bf16* l, const bf16* h, int p) {
#pragma unroll
    for (int u = 0; u < kU; ++u) {
      const int c = (p + u) * 4 + t;
      const bool ok = p + u < p1 && c < nchunk;
      wl[u] = ok ? ld_stream(l + c * 8) : z;
      wh[u] = ok ? ld_stream(h + c * 8) : z;
    }
  };
  int unit = lo / nblk, blk = lo % nblk, e = 0, r0 = 0, M = 0, staged = -1;
  const bf16 *l = nullptr, *h = nullptr;
  if (lo < hi) {
    e = __ldcg(a.expert + unit);
    block(e, blk, &l, &h);
    load(l, h, p0);
  }
  if (a.early) griddep_wait();
  for (int it = lo; it < hi; ++it) {
    if (unit != staged) {
      staged = unit;
      r0 = __ldcg(a.row0 + unit);
      M = min(__ldcg(a.rows + unit), a.max_rows);
      __syncthreads();
      for (int m = 0; m < M; ++m) {
        const bf16* row = a.x + (int64_t)(a.src ? a.src[r0 + m] : r0 + m) * a.ldx;
        for (int c = tid; c < nchunk; c += kT) *reinterpret_cast<uint4*>(xs + m * ldxs + c * 8) = *reinterpret_cast<const uint4*>(row + c * 8);
      }
      __syncthreads();
    }
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    const bf16* xr = xs + g * ldxs;
    for (int p = p0; p < p1; p += kU) {
      if (p != p0) load(l, h, p);
#pragma unroll
      for (int u = 0; u < kU; ++u) {
        const int c = (p + u) * 4 + t;
        const uint4 v = p + u < p1 && c < nchunk && g < M ? *reinterpret_cast<const uint4*>(xr + c * 8) : z;
        mma(acc, wl[u].x, wh[u].x, wl[u].y, wh[u].y, v.x, v.y);
        mma(acc, wl[u].z, wh[u].z, wl[u].w, wh[u].w, v.z, v.w);
      }
    }
    const int n0 = blk * kOut, rr = r0, MM = M;
    if (it + 1 < hi) {
      if (++blk == nblk) {
        blk = 0;
        e = __ldcg(a.expert + ++unit);
      }
      block(e, blk, &l, &h);
      load(l, h, p0);
    }
    float* mine = part + ((it & 1) * kWarps + warp) * kPart;
#pragma unroll
    for (int i = 0; i < 4; ++i) mine[(2 * t + (i & 1)) * kMS + g + (i >> 1) * 8] = acc[i];
    __syncthreads();
    if (tid < 8 * kOut) {
      const int m = tid / kOut, r = tid % kOut;
      if (m < MM && n0 + r < a.N) {
        const float* q = part + (it & 1) * kWarps * kPart + m * kMS + r;
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < kWarps; ++w) v += q[w * kPart];
        if (GATED) {
          float up = 0.f;
#pragma unroll
          for (int w = 0; w < kWarps; ++w) up += q[w * kPart + 8];
          v = silu_s(v) * up;
        } else if (a.act) v = epi_act(a.act, v, 0.f, 0.f);
        a.y[(int64_t)(rr + m) * a.ldy + n0 + r] = __float2bfloat16(v);
      }
    }
  }
}

}  // namespace

// y[r] = act(W[expert(r)] x[src[r]]) (src null: x[r]) for the sorted rows of the unit list; units hold at most max_rows <= 8 rows.
// act 2: squared relu (0: none); 3: silu(gate) * up, W holds N gate rows, then N up rows of every expert.  early: the kernel before this one is the same product over the same list (see above).
CB_EXPORT int cb_gemv_units(const void* W, int64_t stride, const void* x, int64_t ldx, void* y, int64_t ldy, int64_t max_units,
                            int64_t max_rows, int64_t N, int64_t K, int64_t act, const void* count, const void* row0, const void* rows,
                            const void* expert, const void* src, int64_t early, void* stream) {
  if (!W || !x || !y || !count || !row0 || !rows || !expert) return CB_ERR_ARG;
  if (K % 8 || ldx % 8 || stride % 8 || (((uintptr_t)W | (uintptr_t)x) & 15) || N < 1 || K < 8 || max_units < 1 || max_rows < 1 || max_rows > 8)
    return CB_ERR_SHAPE;
  UnitArgs a;
  a.W = (const bf16*)W; a.stride = stride; a.x = (const bf16*)x; a.ldx = ldx; a.y = (bf16*)y; a.ldy = ldy;
  a.count = (const int*)count; a.row0 = (const int*)row0; a.rows = (const int*)rows; a.expert = (const int*)expert; a.src = (const int*)src;
  a.N = (int)N; a.K = (int)K; a.act = act == 3 ? 0 : (int)act; a.early = (int)early; a.max_rows = (int)max_rows;
  const size_t smem = sizeof(float) * 2 * kWarps * kPart + sizeof(bf16) * (size_t)max_rows * (K + kPad);
  if (smem > 220 * 1024) return CB_ERR_SHAPE;
  auto kern = act == 3 ? gemv_units_kernel<true> : gemv_units_kernel<false>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  int64_t per_sm = (int64_t)(224 * 1024 / (smem + 1024));
  per_sm = per_sm < 1 ? 1 : (per_sm > 3 ? 3 : per_sm);
  const int64_t per_block = act == 3 ? 8 : 16, items = max_units * ((N + per_block - 1) / per_block), grid = items < 148 * per_sm ? items : 148 * per_sm;
  int64_t carve = (per_sm * (int64_t)(smem + 1024) * 100 + 228 * 1024 - 1) / (228 * 1024);
  return (int)cb_launch_carve((int)(carve > 100 ? 100 : carve), kern, dim3((unsigned)grid), dim3(kT), smem, (cudaStream_t)stream, a);
}
