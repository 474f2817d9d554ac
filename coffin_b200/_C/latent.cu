// Latent attention: queries and keys / values behind low-rank latents, one rotated key part shared by all heads.
//
// A token leaves one row in the pages, [ latent c | rotated key part ], whatever the number of heads.  Two ways to read it:
//   absorbed : q~_h = W_uk_h^T q_h meets the latent itself, the weighted sum of latents goes through W_uv_h afterwards.
//              One key / value head for all query heads: decoding, and portions of few tokens.
//   expanded : keys and values of every head are multiplied out of the pages' rows (one GEMM whose weight carries
//              identity rows for the shared part) and the prompt kernels of attn_maps_flash.cu / attn_maps_tc.cu run on them.
// Here: the norm / rotate / append kernel, the gather of page rows, the per-head products of the
// absorbed form (tensor cores; plain form for 32-bit) and its split-key decode kernel.  Norms, angles, scores and softmax
// are fp32; the attention weights enter the second product as bf16 head + remainder.
#include "act_type.cuh"

namespace {

constexpr int kPage = 64;
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void cp16(void* s, const void* g, bool ok) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(s);
  const int n = ok ? 16 : 0;                                     // 0 source bytes: the destination is zero-filled
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(a), "l"(g), "r"(n) : "memory");
}
__device__ __forceinline__ void ldsm4(uint32_t* r, const void* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm4t(uint32_t* r, const void* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t split_head(float& x, float& y) {
  const uint32_t h = pack_bf162(x, y);
  x -= __uint_as_float(h << 16);
  y -= __uint_as_float(h & 0xffff0000u);
  return h;
}

// ---- norm, rotate, append ----------------------------------------------------------------------
struct LatentArgs {
  const void* proj; int64_t ldp;         // projection rows: query latent at column 0, then c, then the rotated part
  int64_t c_col, r_col;
  const float* norm_q; const float* norm_c;
  void* cq; int64_t ldq;                 // normed query latents
  void* pool; int64_t ldk;               // page rows [slots, ldk]: c at column 0, rotated part at column cp
  const int* tables; int64_t ldbt;       // block tables [segments, ldbt]
  const int* row_seg;                    // segment of every row (null: row r is segment r)
  const int* positions;                  // < 0: padding
  const float2* cs; int half;            // angles [rows, half]
  int q_rank, kv_rank, rot, cp;
  float eps;
  // queries without a latent (q_rank 0): the projection rows hold H heads of hq columns whose rotated part starts at column
  // r_off; it is turned in place for the rows before `split` and into qa [rows - split, H, ldk] at column cp from there on
  int H, split; int64_t hq, r_off; void* qa; int64_t ldqa;
};

constexpr int kPT = 256, kPV = 8;        // values a thread keeps in registers
template <typename TP, typename TA>
__global__ void __launch_bounds__(kPT) latent_rows_kernel(const LatentArgs a) {
  __shared__ float red[32];
  const int row = blockIdx.x, part = blockIdx.y;                 // part 0: query latent or heads, 1: c and the rotated part
  griddep_launch();
  griddep_wait();
  const int pos = a.positions[row];
  if (pos < 0) return;
  if (!part && !a.q_rank) {
    TP* q = reinterpret_cast<TP*>(const_cast<void*>(a.proj)) + (int64_t)row * a.ldp + a.r_off;
    TA* qa = reinterpret_cast<TA*>(a.qa) + (int64_t)(row - a.split) * a.ldqa + a.cp;
    const int np = (a.rot + 1) / 2;
    for (int e = threadIdx.x; e < a.H * np; e += kPT) {
      const int h = e / np, i = e % np;
      const bool two = 2 * i + 1 < a.rot;
      TP* s = q + h * a.hq + 2 * i;
      float u = act_load(s), v = two ? act_load(s + 1) : 0.f;
      if (i < a.half) {
        const float2 cs = a.cs[(int64_t)row * a.half + i];
        const float x = u * cs.x - v * cs.y;
        v = v * cs.x + u * cs.y;
        u = x;
      }
      if (row < a.split) {
        act_store(s, u);
        if (two) act_store(s + 1, v);
      } else {
        act_store(qa + h * a.ldk + 2 * i, u);
        if (two) act_store(qa + h * a.ldk + 2 * i + 1, v);
      }
    }
    return;
  }
  const TP* p = reinterpret_cast<const TP*>(a.proj) + (int64_t)row * a.ldp + (part ? a.c_col : 0);
  const int n = part ? a.kv_rank : a.q_rank;
  const float* w = part ? a.norm_c : a.norm_q;
  TA* out = part ? reinterpret_cast<TA*>(a.pool) : reinterpret_cast<TA*>(a.cq) + (int64_t)row * a.ldq;
  if (part) {
    const int seg = a.row_seg ? a.row_seg[row] : row;
    out += ((int64_t)a.tables[(int64_t)seg * a.ldbt + pos / kPage] * kPage + pos % kPage) * a.ldk;
  }
  float ss = 0.f, v[kPV];
#pragma unroll
  for (int i = 0; i < kPV; ++i) {
    const int c = threadIdx.x + i * kPT;
    v[i] = c < n ? act_load(p + c) : 0.f;
  }
#pragma unroll
  for (int i = 0; i < kPV; ++i) ss = fmaf(v[i], v[i], ss);
  for (int c = threadIdx.x + kPV * kPT; c < n; c += kPT) { const float x = act_load(p + c); ss = fmaf(x, x, ss); }
  const float r = 1.f / sqrtf(block_sum(ss, red) / (float)n + a.eps);
#pragma unroll
  for (int i = 0; i < kPV; ++i) {
    const int c = threadIdx.x + i * kPT;
    if (c < n) act_store(out + c, v[i] * r * w[c]);
  }
  for (int c = threadIdx.x + kPV * kPT; c < n; c += kPT) act_store(out + c, act_load(p + c) * r * w[c]);
  if (part) {
    const TP* q = reinterpret_cast<const TP*>(a.proj) + (int64_t)row * a.ldp + a.r_col;
    for (int i = threadIdx.x; 2 * i < a.rot; i += kPT) {
      float u = act_load(q + 2 * i), v = 2 * i + 1 < a.rot ? act_load(q + 2 * i + 1) : 0.f;
      if (i < a.half) {
        const float2 cs = a.cs[(int64_t)row * a.half + i];
        const float x = u * cs.x - v * cs.y;
        v = v * cs.x + u * cs.y;
        u = x;
      }
      act_store(out + a.cp + 2 * i, u);
      if (2 * i + 1 < a.rot) act_store(out + a.cp + 2 * i + 1, v);
    }
  }
}

// ---- page rows, gathered -----------------------------------------------------------------------
// dst rows [base[s] + j] = page row of token j of segment s, counted from its page first[s] on, in 16-byte pieces
__global__ void __launch_bounds__(256) latent_gather_kernel(const uint4* __restrict__ pool, int64_t ld16, const int* __restrict__ tables,
                                                            int64_t ldbt, const int* __restrict__ base, const int* __restrict__ lens,
                                                            const int* __restrict__ first, uint4* __restrict__ dst) {
  griddep_launch();
  griddep_wait();
  const int pg = blockIdx.x, s = blockIdx.y, left = lens[s] - pg * kPage;
  if (left <= 0) return;
  const uint4* src = pool + (int64_t)tables[(int64_t)s * ldbt + first[s] + pg] * kPage * ld16;
  uint4* d = dst + ((int64_t)base[s] + pg * kPage) * ld16;
  const int n = (int)(kPage * ld16), ok = (int)(min(left, kPage) * ld16);
  for (int e = threadIdx.x; e < n; e += 256) d[e] = e < ok ? src[e] : make_uint4(0, 0, 0, 0);
}

// ---- per-head products -------------------------------------------------------------------------
// y[t, h, n] = sum_k w[h, n, k] x[t, h, k] (* sigmoid(gate[t, h])): one warp per 16 rows of a head's weight (KS warps share
// them by k), the weight rows straight from 16-byte loads as A fragments, up to 8 NT tokens as columns.
constexpr int kHT = 128;
struct HeadArgs {
  const void* w; const void* x; int64_t ldx, hx;       // row and head strides of x
  void* y; int64_t ldy, hy;
  const float* gate; int64_t ldg;
  int T, H, N, K;
};
template <int NT, int KS>
__global__ void __launch_bounds__(kHT) head_linear_kernel(const HeadArgs a) {
  constexpr int U = 4, BPC = 4 / KS;                   // quads of 8-element chunks in flight; 16-row blocks per CTA
  __shared__ float part[KS > 1 ? 4 : 1][NT][16][9];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t4 = lane & 3;
  const int h = blockIdx.y, ks = warp % KS, n0 = ((int)blockIdx.x * BPC + warp / KS) * 16, t0 = blockIdx.z * 8 * NT;
  const int nq = (a.K + 31) >> 5, per = (nq + KS - 1) / KS, q0 = ks * per, q1 = min(nq, q0 + per);
  const bf16* w = reinterpret_cast<const bf16*>(a.w) + (int64_t)h * a.N * a.K;
  const bf16* wlo = w + (int64_t)min(n0 + g, a.N - 1) * a.K;
  const bf16* whi = w + (int64_t)min(n0 + g + 8, a.N - 1) * a.K;
  const uint4 z = make_uint4(0, 0, 0, 0);
  uint4 lo[U], hi[U];
  auto load = [&](int q) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int c = ((q + u) * 4 + t4) * 8;
      const bool ok = q + u < q1 && c < a.K && n0 < a.N;
      lo[u] = ok ? ld_stream(wlo + c) : z;
      hi[u] = ok ? ld_stream(whi + c) : z;
    }
  };
  griddep_launch();
  load(q0);                                            // the weights do not depend on the previous kernel
  griddep_wait();
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  const bf16* x = reinterpret_cast<const bf16*>(a.x) + h * a.hx;
  for (int q = q0; q < q1; q += U) {
    if (q != q0) load(q);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int c = ((q + u) * 4 + t4) * 8;
      const bool ok = q + u < q1 && c < a.K;
      const uint32_t a0[4] = {lo[u].x, hi[u].x, lo[u].y, hi[u].y}, a1[4] = {lo[u].z, hi[u].z, lo[u].w, hi[u].w};
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        const int t = t0 + i * 8 + g;
        const uint4 v = ok && t < a.T ? *reinterpret_cast<const uint4*>(x + (int64_t)t * a.ldx + c) : z;
        mma(acc[i], a0, v.x, v.y);
        mma(acc[i], a1, v.z, v.w);
      }
    }
  }
  if (KS > 1) {
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) part[warp][i][g + (e >> 1) * 8][2 * t4 + (e & 1)] = acc[i][e];
    __syncthreads();
    if (ks) return;
  }
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int n = n0 + g + (e >> 1) * 8, t = t0 + i * 8 + 2 * t4 + (e & 1);
      if (n >= a.N || t >= a.T) continue;
      float v = acc[i][e];
      if (KS > 1) {
#pragma unroll
        for (int k = 1; k < KS; ++k) v += part[warp + k][i][g + (e >> 1) * 8][2 * t4 + (e & 1)];
      }
      if (a.gate) v *= sigmoid_x(a.gate[(int64_t)t * a.ldg + h]);
      act_store(reinterpret_cast<bf16*>(a.y) + (int64_t)t * a.ldy + h * a.hy + n, v);
    }
}

// the same in 32-bit: a warp per output
__global__ void __launch_bounds__(256) head_linear_f32_kernel(const HeadArgs a) {
  griddep_launch();
  griddep_wait();
  const int lane = threadIdx.x & 31, n = blockIdx.x * 8 + (threadIdx.x >> 5), h = blockIdx.y;
  const int64_t t = blockIdx.z;
  if (n >= a.N) return;
  const float* w = reinterpret_cast<const float*>(a.w) + ((int64_t)h * a.N + n) * a.K;
  const float* x = reinterpret_cast<const float*>(a.x) + t * a.ldx + h * a.hx;
  float s = 0.f;
  for (int k = lane; k < a.K; k += 32) s = fmaf(w[k], x[k], s);
  s = warp_sum(s);
  if (a.gate) s *= sigmoid_x(a.gate[t * a.ldg + h]);
  if (lane == 0) reinterpret_cast<float*>(a.y)[t * a.ldy + h * a.hy + n] = s;
}

// ---- decode ------------------------------------------------------------------------------------
// One CTA per (key split, group of 16 MT heads, row), sixteen warps: the pages of the split go through a two-stage cp.async ring and
// serve every head of the group - scores over the whole page row, weighted sums over its first cp columns.  Leaves
// unnormalised sums and (max, denominator) for latent_merge_kernel.
struct LatentDecodeArgs {
  const void* q; int64_t ldq;            // absorbed queries [rows, H, ldk]
  const void* pool; int64_t ldk;         // page rows
  const int* tables; int64_t ldbt; const int* row_seg; const int* positions;
  float* part_o; float* part_ml;         // [rows, H, nsplit, cp], [.., 2]
  int H, cp, nsplit, window;             // window <= 0: none
  float scale;
};
constexpr int kDT = 512, kPS = kPage + 4;
template <int MT, int NP2>               // NP2: 16-column pairs of the values per warp (cp <= 256 NP2)
__global__ void __launch_bounds__(kDT, 1) latent_decode_kernel(const LatentDecodeArgs a) {
  constexpr int PP = kPage + 8, NH = 16 * MT, KS = 4 / MT;      // KS: slices of the page row that share a score
  extern __shared__ __align__(128) unsigned char smem[];
  const int LW = (int)a.ldk, LK = LW + 8, KPAGE = kPage * LK;
  bf16* ks = reinterpret_cast<bf16*>(smem);            // [2][kPage][LK]
  bf16* qs = ks + 2 * KPAGE;                           // [NH][LK]
  bf16* pa = qs + NH * LK;                             // [2][NH][PP]: heads, remainders
  float* ps = reinterpret_cast<float*>(pa + 2 * NH * PP);        // [KS][NH][kPS] partial scores
  __shared__ float w_s[NH];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g4 = lane >> 2, t4 = lane & 3;
  const int split = blockIdx.x, row = blockIdx.z, h0 = blockIdx.y * NH, nh = min(NH, a.H - h0);
  griddep_launch();
  griddep_wait();
  const int pos = a.positions[row], seg = a.row_seg ? a.row_seg[row] : row;
  if (pos < 0) return;
  const int64_t vh0 = (int64_t)row * a.H + h0;
  const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0, page0 = lo / kPage;     // first visible key
  const int pages = pos / kPage + 1, per = (pages - page0 + a.nsplit - 1) / a.nsplit;
  const int pg0 = page0 + split * per, pg1 = min(pages, pg0 + per);
  if (pg0 >= pages) {
    if (tid < nh) a.part_ml[((vh0 + tid) * a.nsplit + split) * 2] = -INFINITY;
    return;
  }
  const int* bt = a.tables + (int64_t)seg * a.ldbt;
  const bf16* pool = reinterpret_cast<const bf16*>(a.pool);
  const int pieces = LW / 8;
  auto load = [&](int pg) {
    const bf16* src = pool + (int64_t)bt[pg] * kPage * LW;
    const int n = min(kPage, pos + 1 - pg * kPage);    // rows of the page that exist
    bf16* kd = ks + (pg & 1) * KPAGE;
    for (int r = warp; r < kPage; r += kDT / 32)
      for (int c = lane; c < pieces; c += 32) cp16(kd + r * LK + c * 8, r < n ? src + (int64_t)r * LW + c * 8 : src, r < n);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load(pg0);
  const bf16* q = reinterpret_cast<const bf16*>(a.q) + (int64_t)row * a.ldq + (int64_t)h0 * LW;
  for (int r = warp; r < NH; r += kDT / 32)
    for (int c = lane; c < pieces; c += 32)
      *reinterpret_cast<uint4*>(qs + r * LK + c * 8) = r < nh ? *reinterpret_cast<const uint4*>(q + (int64_t)r * LW + c * 8) : make_uint4(0, 0, 0, 0);
  float o[MT][NP2][2][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < NP2; ++i)
#pragma unroll
      for (int j = 0; j < 2; ++j) o[m][i][j][0] = o[m][i][j][1] = o[m][i][j][2] = o[m][i][j][3] = 0.f;
  float m_run[MT], l_run[MT];                          // of heads warp + 16 i
#pragma unroll
  for (int i = 0; i < MT; ++i) { m_run[i] = -INFINITY; l_run[i] = 0.f; }
  const float f = a.scale * kLog2e;
  const int ksteps = LW / 16, np = a.cp / 16;
  // scores: a warp takes 16 keys, one head tile and one slice of the page row
  const int kg = warp & 3, mt = (warp >> 2) % MT, sl = (warp >> 2) / MT;
  const int kper = (ksteps + KS - 1) / KS, k0 = sl * kper, k1 = min(ksteps, k0 + kper);
  for (int pg = pg0; pg < pg1; ++pg) {
    if (pg + 1 < pg1) {
      load(pg + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const bf16* kt = ks + (pg & 1) * KPAGE;
    {
      float s[2][2][4];                                // [chain][key half]
#pragma unroll
      for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int j = 0; j < 2; ++j) s[c][j][0] = s[c][j][1] = s[c][j][2] = s[c][j][3] = 0.f;
      const bf16* kr = kt + (kg * 16 + (lane & 7) + ((lane >> 4) << 3)) * LK + ((lane >> 3) & 1) * 8;
      const bf16* qr = qs + (mt * 16 + (lane & 15)) * LK + (lane >> 4) * 8;
      int k = k0;
#pragma unroll 3
      for (; k + 2 <= k1; k += 2) {
        uint32_t a0[4], a1[4], b0[4], b1[4];
        ldsm4(a0, qr + k * 16);
        ldsm4(b0, kr + k * 16);
        ldsm4(a1, qr + k * 16 + 16);
        ldsm4(b1, kr + k * 16 + 16);
        mma(s[0][0], a0, b0[0], b0[1]);
        mma(s[0][1], a0, b0[2], b0[3]);
        mma(s[1][0], a1, b1[0], b1[1]);
        mma(s[1][1], a1, b1[2], b1[3]);
      }
      if (k < k1) {
        uint32_t a0[4], b0[4];
        ldsm4(a0, qr + k * 16);
        ldsm4(b0, kr + k * 16);
        mma(s[0][0], a0, b0[0], b0[1]);
        mma(s[0][1], a0, b0[2], b0[3]);
      }
      float* pd = ps + (sl * NH + mt * 16 + g4) * kPS + kg * 16 + t4 * 2;
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        *reinterpret_cast<float2*>(pd + j * 8) = make_float2(s[0][j][0] + s[1][j][0], s[0][j][1] + s[1][j][1]);
        *reinterpret_cast<float2*>(pd + 8 * kPS + j * 8) = make_float2(s[0][j][2] + s[1][j][2], s[0][j][3] + s[1][j][3]);
      }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const int hd = warp + 16 * i, key = pg * kPage + 2 * lane;
      float2 x = make_float2(0.f, 0.f);
#pragma unroll
      for (int c = 0; c < KS; ++c) {
        const float2 p = *reinterpret_cast<const float2*>(ps + (c * NH + hd) * kPS + 2 * lane);
        x.x += p.x; x.y += p.y;
      }
      x.x = key <= pos && key >= lo ? x.x * f : -INFINITY;
      x.y = key + 1 <= pos && key + 1 >= lo ? x.y * f : -INFINITY;
      const float mn = fmaxf(m_run[i], warp_max(fmaxf(x.x, x.y)));     // finite: a walked page holds a visible key
      float e0 = ex2(x.x - mn), e1 = ex2(x.y - mn);
      const float w = ex2(m_run[i] - mn);
      l_run[i] = l_run[i] * w + e0 + e1;               // this lane's share
      m_run[i] = mn;
      *reinterpret_cast<uint32_t*>(pa + hd * PP + 2 * lane) = split_head(e0, e1);
      *reinterpret_cast<uint32_t*>(pa + (NH + hd) * PP + 2 * lane) = pack_bf162(e0, e1);
      if (lane == 0) w_s[hd] = w;
    }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float wl = w_s[m * 16 + g4], wh = w_s[m * 16 + g4 + 8];
#pragma unroll
      for (int i = 0; i < NP2; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j) { o[m][i][j][0] *= wl; o[m][i][j][1] *= wl; o[m][i][j][2] *= wh; o[m][i][j][3] *= wh; }
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      uint32_t ph[MT][4], pl[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        ldsm4(ph[m], pa + (m * 16 + (lane & 15)) * PP + k * 16 + (lane >> 4) * 8);
        ldsm4(pl[m], pa + ((MT + m) * 16 + (lane & 15)) * PP + k * 16 + (lane >> 4) * 8);
      }
#pragma unroll
      for (int i = 0; i < NP2; ++i) {
        const int cp = warp + 16 * i;
        if (cp < np) {
          uint32_t b[4];
          ldsm4t(b, kt + (k * 16 + (lane & 15)) * LK + cp * 16 + (lane >> 4) * 8);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma(o[m][i][0], ph[m], b[0], b[1]);
            mma(o[m][i][1], ph[m], b[2], b[3]);
          }
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma(o[m][i][0], pl[m], b[0], b[1]);
            mma(o[m][i][1], pl[m], b[2], b[3]);
          }
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < NP2; ++i) {
      if (warp + 16 * i >= np) continue;
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int hd = m * 16 + g4 + 8 * e, c = (warp + 16 * i) * 16 + j * 8 + t4 * 2;
          if (hd < nh)
            *reinterpret_cast<float2*>(a.part_o + ((vh0 + hd) * a.nsplit + split) * a.cp + c) = make_float2(o[m][i][j][2 * e], o[m][i][j][2 * e + 1]);
        }
    }
#pragma unroll
  for (int i = 0; i < MT; ++i) {
    const int hd = warp + 16 * i;
    const float l = warp_sum(l_run[i]);
    if (hd < nh && lane == 0) {
      float* ml = a.part_ml + ((vh0 + hd) * a.nsplit + split) * 2;
      ml[0] = m_run[i] * (1.f / kLog2e);
      ml[1] = l;
    }
  }
}

// merge of the key splits: 128 columns of one (row, head) per CTA, two groups of threads share the splits
template <typename TA>
__global__ void __launch_bounds__(256) latent_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                                           const int* __restrict__ positions, TA* __restrict__ out, int64_t ldo, int H,
                                                           int cp, int nsplit) {
  __shared__ float sum_s[128];
  const int tid = threadIdx.x, lane = tid & 31, h = blockIdx.y, c = blockIdx.x * 128 + (tid & 127), sg = tid >> 7;
  const int64_t row = blockIdx.z;
  griddep_launch();
  griddep_wait();
  if (positions[row] < 0) return;
  const int64_t vh = row * H + h;
  const float* ml = part_ml + vh * nsplit * 2;
  float2 v[2];                                         // splits lane and lane + 32
#pragma unroll
  for (int k = 0; k < 2; ++k)
    v[k] = lane + 32 * k < nsplit ? *reinterpret_cast<const float2*>(ml + 2 * (lane + 32 * k)) : make_float2(-INFINITY, 0.f);
  // splits are filled from the front
  const int used = __popc(__ballot_sync(0xffffffffu, v[0].x != -INFINITY)) + __popc(__ballot_sync(0xffffffffu, v[1].x != -INFINITY));
  const float M = warp_max(fmaxf(v[0].x, v[1].x));
  float fac[2];
#pragma unroll
  for (int k = 0; k < 2; ++k) fac[k] = v[k].x == -INFINITY ? 0.f : expf(v[k].x - M);
  const float inv = 1.f / warp_sum(fac[0] * v[0].y + fac[1] * v[1].y);
  const float* po = part_o + vh * nsplit * cp + min(c, cp - 1);
  float acc = 0.f;
#pragma unroll 8
  for (int s = sg; s < used; s += 2) acc = fmaf(__shfl_sync(0xffffffffu, s < 32 ? fac[0] : fac[1], s & 31), po[(int64_t)s * cp], acc);
  if (sg) sum_s[tid & 127] = acc;
  __syncthreads();
  if (!sg && c < cp) act_store(out + row * ldo + (int64_t)h * cp + c, (acc + sum_s[tid]) * inv);
}

size_t decode_smem(int mt, int64_t lw) {
  return sizeof(bf16) * (size_t)(2 * kPage * (lw + 8) + 16 * mt * (lw + 8) + 2 * 16 * mt * (kPage + 8)) + sizeof(float) * 64 * kPS;
}
template <int MT, int NP2>
int launch_decode(const LatentDecodeArgs& a, int rows, cudaStream_t st) {
  auto kern = latent_decode_kernel<MT, NP2>;
  const size_t smem = decode_smem(MT, a.ldk);
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  return (int)cb_launch(kern, dim3((unsigned)a.nsplit, (unsigned)((a.H + 16 * MT - 1) / (16 * MT)), (unsigned)rows), dim3(kDT), smem, st, a);
}
template <int NT>
int launch_heads(const HeadArgs& a, cudaStream_t st) {
  const unsigned tz = (unsigned)((a.T + 8 * NT - 1) / (8 * NT)), nb = (unsigned)((a.N + 15) / 16);
  if (a.K >= 256) return (int)cb_launch(head_linear_kernel<NT, 4>, dim3(nb, (unsigned)a.H, tz), dim3(kHT), 0, st, a);
  return (int)cb_launch(head_linear_kernel<NT, 1>, dim3((nb + 3) / 4, (unsigned)a.H, tz), dim3(kHT), 0, st, a);
}

}  // namespace

CB_EXPORT int cb_latent_args_size() { return (int)sizeof(LatentArgs); }

// `rows` projection rows: cq = rmsnorm(query latent), or the rotated query parts turned (q_rank 0); with own != 0 also
// rmsnorm(c) and the rotated part into the pages.
// p_f32: projection rows are fp32; f32: latents and pages are fp32 instead of bf16.
CB_EXPORT int cb_latent_rows(const void* args, int64_t rows, int64_t own, int64_t p_f32, int64_t f32, void* stream) {
  if (!args || rows < 1) return CB_ERR_ARG;
  const LatentArgs& a = *(const LatentArgs*)args;
  if (!a.proj || !a.positions || a.q_rank < 0 || (a.q_rank && (!a.norm_q || !a.cq))) return CB_ERR_ARG;
  if (!a.q_rank && (a.H < 1 || a.split < 0 || (a.split < rows && !a.qa) || (p_f32 && !f32) || 2 * a.half > a.rot || (a.half && !a.cs)))
    return CB_ERR_ARG;
  if (own && (!a.pool || !a.norm_c || !a.tables || a.kv_rank < 1 || a.kv_rank > a.cp || a.cp + a.rot > a.ldk || (a.half && !a.cs) || 2 * a.half > a.rot))
    return CB_ERR_ARG;
  const dim3 grid((unsigned)rows, own ? 2u : 1u), block(kPT);
  cudaStream_t st = (cudaStream_t)stream;
  if (f32) return (int)cb_launch(latent_rows_kernel<float, float>, grid, block, 0, st, a);
  if (p_f32) return (int)cb_launch(latent_rows_kernel<float, bf16>, grid, block, 0, st, a);
  return (int)cb_launch(latent_rows_kernel<bf16, bf16>, grid, block, 0, st, a);
}

// Page rows of `segs` sequences side by side: segment s fills rows base[s] .. base[s] + whole pages of lens[s] tokens, from
// page first[s] of its table on.
CB_EXPORT int cb_latent_gather(const void* pool, int64_t row_bytes, const void* tables, int64_t ldbt, const void* base, const void* lens,
                               const void* first, void* dst, int64_t segs, int64_t max_pages, void* stream) {
  if (!pool || !tables || !base || !lens || !first || !dst || segs < 1 || segs > 65535 || max_pages < 1) return CB_ERR_ARG;
  if (row_bytes % 16) return CB_ERR_SHAPE;
  return (int)cb_launch(latent_gather_kernel, dim3((unsigned)max_pages, (unsigned)segs), dim3(256), 0, (cudaStream_t)stream,
                        (const uint4*)pool, row_bytes / 16, (const int*)tables, ldbt, (const int*)base, (const int*)lens, (const int*)first, (uint4*)dst);
}

// y[t, h, :N] = w[h] x[t, h, :K] (* sigmoid(gate[t, h])), w [H, N, K]; bf16 (K % 8 == 0, 16-byte rows) or fp32.
CB_EXPORT int cb_head_linear(const void* w, const void* x, int64_t ldx, int64_t hx, void* y, int64_t ldy, int64_t hy, const void* gate,
                             int64_t ldg, int64_t T, int64_t H, int64_t N, int64_t K, int64_t f32, void* stream) {
  if (!w || !x || !y || T < 1 || H < 1 || H > 65535 || N < 1 || K < 1) return CB_ERR_ARG;
  HeadArgs a;
  a.w = w; a.x = x; a.ldx = ldx; a.hx = hx; a.y = y; a.ldy = ldy; a.hy = hy; a.gate = (const float*)gate; a.ldg = ldg;
  a.T = (int)T; a.H = (int)H; a.N = (int)N; a.K = (int)K;
  cudaStream_t st = (cudaStream_t)stream;
  if (f32) {
    if (T > 65535) return CB_ERR_SHAPE;
    return (int)cb_launch(head_linear_f32_kernel, dim3((unsigned)((N + 7) / 8), (unsigned)H, (unsigned)T), dim3(256), 0, st, a);
  }
  if (K % 8 || ldx % 8 || hx % 8 || ((uintptr_t)x & 15) || ((uintptr_t)w & 15)) return CB_ERR_SHAPE;
  if (T <= 8) return launch_heads<1>(a, st);
  if (T <= 16) return launch_heads<2>(a, st);
  if (T <= 32) return launch_heads<4>(a, st);
  return launch_heads<8>(a, st);
}

// Whether cb_latent_decode takes page rows of ldk columns with cp latent ones.
CB_EXPORT int cb_latent_decode_ok(int64_t ldk, int64_t cp) {
  return ldk % 16 == 0 && cp % 16 == 0 && cp >= 16 && cp <= 512 && cp <= ldk && decode_smem(2, ldk) <= 220 * 1024;
}

// Absorbed attention of `rows` queries [rows, H, ldk] against the pages (their own rows appended before): key splits into
// part_o [rows, H, nsplit, cp] / part_ml.  tiles: groups of 16 heads a CTA serves (1 or 2); window: tokens a query sees,
// itself included (<= 0: all up to it).
CB_EXPORT int cb_latent_decode(const void* q, int64_t ldq, const void* pool, int64_t ldk, const void* tables, int64_t ldbt,
                               const void* row_seg, const void* positions, void* part_o, void* part_ml, int64_t rows, int64_t H, int64_t cp,
                               int64_t nsplit, int64_t tiles, int64_t window, float scale, void* stream) {
  if (tiles < 1 || tiles > 2) return CB_ERR_ARG;
  if (!q || !pool || !tables || !positions || !part_o || !part_ml || rows < 1 || rows > 65535 || H < 1 || nsplit < 1 || nsplit > 64)
    return CB_ERR_ARG;
  if (!cb_latent_decode_ok(ldk, cp) || ldq % 8 || ((uintptr_t)q & 15) || ((uintptr_t)pool & 15)) return CB_ERR_SHAPE;
  LatentDecodeArgs a;
  a.q = q; a.ldq = ldq; a.pool = pool; a.ldk = ldk; a.tables = (const int*)tables; a.ldbt = ldbt; a.row_seg = (const int*)row_seg;
  a.positions = (const int*)positions; a.part_o = (float*)part_o; a.part_ml = (float*)part_ml; a.H = (int)H; a.cp = (int)cp;
  a.nsplit = (int)nsplit; a.window = (int)window; a.scale = scale;
  cudaStream_t st = (cudaStream_t)stream;
  const int r = (int)rows;
  if (tiles == 1) return cp <= 256 ? launch_decode<1, 1>(a, r, st) : launch_decode<1, 2>(a, r, st);
  return cp <= 256 ? launch_decode<2, 1>(a, r, st) : launch_decode<2, 2>(a, r, st);
}

// out[row, h, :cp] = average of the key splits left by cb_latent_decode.  f32: out is fp32 instead of bf16.
CB_EXPORT int cb_latent_merge(const void* part_o, const void* part_ml, const void* positions, void* out, int64_t ldo, int64_t rows, int64_t H,
                              int64_t cp, int64_t nsplit, int64_t f32, void* stream) {
  if (!part_o || !part_ml || !positions || !out || rows < 1 || rows > 65535 || H < 1 || H > 65535 || cp < 1 || nsplit < 1 || nsplit > 64) return CB_ERR_ARG;
  const dim3 grid((unsigned)((cp + 127) / 128), (unsigned)H, (unsigned)rows), block(256);
  cudaStream_t st = (cudaStream_t)stream;
  if (f32)
    return (int)cb_launch(latent_merge_kernel<float>, grid, block, 0, st, (const float*)part_o, (const float*)part_ml, (const int*)positions,
                          (float*)out, ldo, (int)H, (int)cp, (int)nsplit);
  return (int)cb_launch(latent_merge_kernel<bf16>, grid, block, 0, st, (const float*)part_o, (const float*)part_ml, (const int*)positions,
                        (bf16*)out, ldo, (int)H, (int)cp, (int)nsplit);
}
