// Recurrent mixers with a matrix state, one token at a time: the decode step, and the generic path of a prompt.
//
//   delta  : gated delta rule with one decay per head and key channel,
//              S <- g * S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//            behind a short causal convolution + SiLU and unit q / k vectors; o is RMS-normed per head,
//            weighted and multiplied by a low-rank sigmoid gate.
//   mLSTM  : matrix memory with exponential gates under a running maximum m,
//              S <- exp(f + m' - m) S + exp(i - m) k v^T;  n likewise with k;
//              o = S^T q / (max(|n.q|, exp(-m)) + 1e-6)
//            o is RMS-normed per head, weighted and multiplied by a sigmoid gate.
//   gated  : the forget gate f of a key channel (sigmoid above a lower bound) also decides what is written,
//              S <- f * S + (1 - f) v^T;  o = S^T silu(q)
//            o is RMS-normed per head and weighted.
//
// One cluster of CTAs per (head, sequence): every CTA owns `jc` value columns of the head's state in registers
// (the columns of S never interact), computes the head's q / k / decays itself, and only the RMS norm over the
// head's values crosses the cluster (one partial sum per CTA through distributed shared memory).  The read-out is
// taken without a second reduction: o = (gS)^T q + u (k.q).  Everything from the projections on is fp32.
// Launches: one per layer and step.  The scalar-decay delta net of the Qwen3.5 family is gdn.cu.
#include "linrec.cuh"
#include "sm100.cuh"

namespace {

constexpr int kT = 256;

__device__ __forceinline__ float ld_dsmem(const float* p, uint32_t rank) {
  const uint32_t a = sm100::map_to_cta((uint32_t)__cvta_generic_to_shared(p), rank);
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(a) : "memory");
  return v;
}

// dot of a weight row (storage type) with fp32 values in shared memory; n is a multiple of 4
template <typename TW>
__device__ __noinline__ float row_dot(const TW* __restrict__ w, const float* x, int64_t n) {
  float s0 = 0.f, s1 = 0.f;
  int64_t i = 0;
#pragma unroll 1
  for (; i + 8 <= n; i += 8) {
    const float4 a = act_load4(w + i), b = act_load4(w + i + 4);
    s0 = fmaf(a.x, x[i], s0); s0 = fmaf(a.y, x[i + 1], s0); s0 = fmaf(a.z, x[i + 2], s0); s0 = fmaf(a.w, x[i + 3], s0);
    s1 = fmaf(b.x, x[i + 4], s1); s1 = fmaf(b.y, x[i + 5], s1); s1 = fmaf(b.z, x[i + 6], s1); s1 = fmaf(b.w, x[i + 7], s1);
  }
  return s0 + s1;
}

// Low-rank factor times a short vector, rows x rank spread over the block in 16-byte pieces (2^lsh lanes per row).  The
// weights do not depend on the previous kernel, so the first PRE pieces of a thread are requested ahead of the
// dependency wait and used once the vector is there.
template <int PRE>
struct LowRank {
  uint4 w[PRE];
  const bf16* W;
  int rows, nch, lsh, iters;
  __device__ __forceinline__ void init(const bf16* W_, int rows_, int rank) {
    W = W_; rows = rows_; nch = rank >> 3;
    lsh = nch <= 1 ? 0 : 32 - __clz(nch - 1);
    iters = ((rows << lsh) + kT - 1) / kT;
#pragma unroll
    for (int i = 0; i < PRE; ++i) w[i] = i < iters ? piece(i) : make_uint4(0, 0, 0, 0);
  }
  __device__ __forceinline__ uint4 piece(int it) const {
    const int i = it * kT + (int)threadIdx.x, r = i >> lsh, c = i & ((1 << lsh) - 1);
    return r < rows && c < nch ? *reinterpret_cast<const uint4*>(W + ((int64_t)r * nch + c) * 8) : make_uint4(0, 0, 0, 0);
  }
  // out[r] = W[r, :] . x, by the first lane of a row.  A thread's pieces all multiply the same eight values of x.
  __device__ __forceinline__ void dot_piece(int it, const uint4& v, const float* xr, float* out) const {
    const int i = it * kT + (int)threadIdx.x, r = i >> lsh, c = i & ((1 << lsh) - 1);
    float f[8], s = 0.f;
    bf16x8_to_float(v, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) s = fmaf(f[e], xr[e], s);
    for (int o = 1; o < (1 << lsh); o <<= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    if (c == 0 && r < rows) out[r] = s;
  }
  __device__ __forceinline__ void run(const float* x, float* out) {
    const int c = (int)threadIdx.x & ((1 << lsh) - 1);
    float xr[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) xr[e] = c < nch ? x[c * 8 + e] : 0.f;
#pragma unroll 1
    for (int g = 0; g < iters; g += PRE) {
      if (g > 0) {
#pragma unroll
        for (int i = 0; i < PRE; ++i) w[i] = g + i < iters ? piece(g + i) : make_uint4(0, 0, 0, 0);
      }
#pragma unroll
      for (int i = 0; i < PRE; ++i)
        if (g + i < iters) dot_piece(g + i, w[i], xr, out);
    }
  }
};

// sums of three values over the block; every thread gets them
__device__ __forceinline__ void block_sum3(float& a, float& b, float& c, float* red) {
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5;
  a = warp_sum(a); b = warp_sum(b); c = warp_sum(c);
  __syncthreads();
  if (lane == 0) { red[w * 3] = a; red[w * 3 + 1] = b; red[w * 3 + 2] = c; }
  __syncthreads();
  a = b = c = 0.f;
#pragma unroll
  for (int i = 0; i < kT / 32; ++i) { a += red[i * 3]; b += red[i * 3 + 1]; c += red[i * 3 + 2]; }
}

// LOW: the low-rank factors are multiplied here (few rows), else their results are given
template <int KIND, typename TP, typename TA, int RMAX, bool LOW>
__global__ void __launch_bounds__(kT, RMAX <= 4 && !LOW ? 3 : (RMAX <= 16 ? 2 : 1)) linrec_step_kernel(const LinrecArgs a) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[32];
  __shared__ float cl_part;
  const int tid = threadIdx.x, h = blockIdx.y, seg = blockIdx.z, NS = gridDim.x, rank = blockIdx.x;
  const int dk = a.dk, dv = a.dv, jc = a.jc;
  float* sq = sm;                                      // [dk]
  float* sk = sq + dk;                                 // [dk]
  float* sg = sk + dk;                                 // [dk] decays (delta, gated) / n (mLSTM)
  float* sv = sg + dk;                                 // [jc]
  float* su = sv + jc;                                 // [jc]
  float* so = su + jc;                                 // [jc]
  float* sog = so + jc;                                // [jc] output gates
  float* low = sog + jc;                               // [ra + rg] low-rank activations (delta)
  const int lown = KIND == LINREC_DELTA ? (int)((a.dec ? 0 : a.ra) + (a.og ? 0 : a.rg)) : 0;
  float* part = low + ((lown + 3) & ~3);               // [RG][jc] x 2
  const int cq = jc >> 2, RG = kT / cq, q4 = tid % cq, rg = tid / cq;
  const bool act_thr = rg < RG;
  const int j0 = rank * jc, ncol = min(jc, dv - j0);   // ncol > 0 by construction of the grid
  constexpr bool kLow = KIND == LINREC_DELTA && sizeof(TA) == 2 && LOW;
  const bool low_a = kLow && !a.dec && a.ra <= 256, low_g = kLow && !a.og && a.rg <= 256;
  LowRank<kLow ? (RMAX <= 8 ? 8 : 4) : 1> lra;
  LowRank<kLow ? 4 : 1> lrg;
  if (low_a) lra.init(reinterpret_cast<const bf16*>(a.a2) + (int64_t)h * dk * a.ra, dk, (int)a.ra);
  if (low_g) lrg.init(reinterpret_cast<const bf16*>(a.g2) + ((int64_t)h * dv + j0) * a.rg, ncol, (int)a.rg);
  // parameters of this thread's channels, requested ahead of the dependency like the factors
  float4 pcw[2];                                       // convolution taps of channels tid and tid + kT (four taps)
  const int nch = 2 * dk + ncol;
  const bool taps4 = a.taps == 4;
  const int qb = h / (a.H / a.G) * dk;
  auto channel = [&](int e) {
    return e < dk ? (int64_t)(qb + e) : (e < 2 * dk ? a.k_col + qb + e - dk : a.v_col + (int64_t)h * dv + j0 + e - 2 * dk);
  };
  float p_dt = 0.f, p_ea = 0.f, p_bi = 0.f, p_bf = 0.f;
  if (KIND == LINREC_MLSTM) { p_bi = a.gate_b[h]; p_bf = a.gate_b[a.H + h]; }
  if (KIND == LINREC_GATED && tid < dk) { p_bf = a.gate_b[(int64_t)h * dk + tid]; p_bi = a.lower[(int64_t)h * dk + tid]; }
  if (KIND == LINREC_DELTA) {
#pragma unroll
    for (int u = 0; u < 2; ++u)
      pcw[u] = taps4 && tid + u * kT < nch ? *reinterpret_cast<const float4*>(a.conv_w + channel(tid + u * kT) * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    p_ea = expf(a.A_log[h]);
    if (tid < dk) p_dt = a.dt_bias[(int64_t)h * dk + tid];
  }
  const float* nw = a.norm_w + (KIND == LINREC_MLSTM ? (int64_t)h * dv : 0) + j0;
  const float p_nw = tid < ncol ? nw[tid] : 0.f;
  griddep_launch();
  griddep_wait();
  const int row0 = a.seg_row ? a.seg_row[seg] : seg;
  const int nrow = a.seg_row ? a.seg_row[seg + 1] - row0 : 1;
  const int slot = a.seg_slot[seg], pos0 = a.seg_pos[seg];
  if (slot < 0 || nrow < 1 || pos0 < 0) return;        // the same for every CTA of the cluster
  float* Sg = a.S + ((int64_t)slot * a.H + h) * dk * dv + j0;
  const bool vec = (dv & 3) == 0 && ncol == jc;
  float S[RMAX][4];
  const int nr = act_thr && q4 * 4 < ncol ? (dk - rg + RG - 1) / RG : 0;      // state rows of this thread
  float* const Sp = Sg + (int64_t)rg * dv + q4 * 4;
  const int64_t sstep = (int64_t)RG * dv;
  const int ne = min(4, ncol - q4 * 4);
  if (vec) {
#pragma unroll
    for (int i = 0; i < RMAX; ++i) {
      const float4 f = i < nr ? *reinterpret_cast<const float4*>(Sp + i * sstep) : make_float4(0.f, 0.f, 0.f, 0.f);
      S[i][0] = f.x; S[i][1] = f.y; S[i][2] = f.z; S[i][3] = f.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < RMAX; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[i][e] = i < nr && e < ne ? Sp[i * sstep + e] : 0.f;
  }
  float mrun = 0.f;
  if (KIND == LINREC_MLSTM) {
    mrun = a.m[(int64_t)slot * a.H + h];
    for (int c = tid; c < dk; c += kT) sg[c] = a.n[((int64_t)slot * a.H + h) * dk + c];
    // rank 0 rewrites n and m at the end: every CTA of the cluster has to have read them by then
    if (NS > 1) sm100::cluster_sync_all();
  }
  const TA* ring = reinterpret_cast<const TA*>(a.ring) + (int64_t)slot * (a.ring_mask + 1) * a.ring_w;
  const TP* prow0 = reinterpret_cast<const TP*>(a.proj) + (int64_t)row0 * a.ldp;

  for (int t = 0; t < nrow; ++t) {
    const int64_t row = row0 + t;
    const TP* pr = prow0 + (int64_t)t * a.ldp;
    float aa = 1.f, bb = 1.f, kq = 0.f, den = 1.f;
    // what channel `tid` needs from this row, requested together
    float x_a = 0.f, x_b = 0.f, x_v = 0.f, x_og = 0.f;
    const int64_t vch = (int64_t)h * dv + j0 + tid;
    const float gate0 = KIND == LINREC_GATED ? 0.f : a.gates[row * a.ldg + h], gate1 = KIND == LINREC_MLSTM ? a.gates[row * a.ldg + a.H + h] : 0.f;
    if (KIND == LINREC_DELTA) {
      if (tid < dk && a.dec) x_a = a.dec[row * a.ldd + (int64_t)h * dk + tid];
      if (tid < ncol && a.og) x_og = act_load(reinterpret_cast<const TA*>(a.og) + row * a.ldo + vch);
    } else if (KIND == LINREC_GATED) {
      if (tid < dk) {
        x_a = act_load(pr + (int64_t)h * dk + tid);
        x_b = a.gates[row * a.ldg + (int64_t)h * dk + tid];
      }
      if (tid < ncol) x_v = act_load(pr + a.v_col + vch);
    } else {
      if (tid < dk) {
        x_a = act_load(pr + (int64_t)h * dk + tid);
        x_b = act_load(pr + a.k_col + (int64_t)h * dk + tid);
      }
      if (tid < ncol) {
        x_v = act_load(pr + a.v_col + vch);
        x_og = act_load(reinterpret_cast<const TP*>(a.og) + row * a.ldo + vch);
      }
    }
    if (KIND == LINREC_DELTA) {
      // short convolution: channels q, k, v of this CTA spread over the block, four taps requested together (in a decode
      // step all but the newest come from the ring)
      auto tap = [&](int64_t ch, int j) {                // the row a tap reads is the same for every channel
        const int src = t - (a.taps - 1) + j, p = pos0 + src;
        float x = 0.f;
        if (src >= 0) x = act_round<TA>(act_load(prow0 + (int64_t)src * a.ldp + ch));
        else if (p >= 0) x = act_load(ring + (int64_t)(p & a.ring_mask) * a.ring_w + ch);
        return x;
      };
      auto put = [&](int e, float acc) { (e < 2 * dk ? sq : sv - 2 * dk)[e] = silu_s(acc); };       // sq and sk are adjacent
      if (taps4) {
        float x[2][4];
        const int64_t ch0 = channel(tid < nch ? tid : 0), ch1 = channel(tid + kT < nch ? tid + kT : 0);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          x[0][j] = tid < nch ? tap(ch0, j) : 0.f;
          x[1][j] = tid + kT < nch ? tap(ch1, j) : 0.f;
        }
#pragma unroll
        for (int u = 0; u < 2; ++u)
          if (tid + u * kT < nch)
            put(tid + u * kT, fmaf(pcw[u].w, x[u][3], fmaf(pcw[u].z, x[u][2], fmaf(pcw[u].y, x[u][1], pcw[u].x * x[u][0]))));
      }
#pragma unroll 1
      for (int e = tid + (taps4 ? 2 * kT : 0); e < nch; e += kT) {
        const int64_t ch = channel(e);
        float acc = 0.f;
#pragma unroll 1
        for (int j = 0; j < a.taps; ++j) acc = fmaf(a.conv_w[ch * a.taps + j], tap(ch, j), acc);
        put(e, acc);
      }
#pragma unroll 1
      for (int c = tid; c < lown; c += kT) {
        const int na = a.dec ? 0 : (int)a.ra;
        low[c] = act_round<TA>(act_load(pr + (c < na ? a.a1_col + c : a.g1_col + c - na)));
      }
      bb = sigmoid_s(gate0);                                // beta
      __syncthreads();
      float q2 = 0.f, k2 = 0.f, qk = 0.f;
      for (int c = tid; c < dk; c += kT) {
        const float qc = sq[c], kc = sk[c];
        q2 = fmaf(qc, qc, q2); k2 = fmaf(kc, kc, k2); qk = fmaf(qc, kc, qk);
      }
      block_sum3(q2, k2, qk, red);
      const float rq = 1.f / (sqrtf(q2 + 1e-6f) * sqrtf((float)dk)), rk = 1.f / sqrtf(k2 + 1e-6f);
      kq = qk * rq * rk;
      if (low_a) lra.run(low, sg);
      if (low_g) lrg.run(low + (a.dec ? 0 : a.ra), sog);
      if (low_a || low_g) __syncthreads();
      const TA* a2 = reinterpret_cast<const TA*>(a.a2);
      for (int c = tid; c < dk; c += kT) {
        sq[c] *= rq; sk[c] *= rk;
        const int64_t ch = (int64_t)h * dk + c;
        const float x = !LOW || a.dec ? (c == tid ? x_a : a.dec[row * a.ldd + ch]) : (low_a ? sg[c] : row_dot(a2 + ch * a.ra, low, a.ra));
        sg[c] = __expf(-p_ea * softplus_s(x + (c == tid ? p_dt : a.dt_bias[ch])));
      }
      const TA* g2 = reinterpret_cast<const TA*>(a.g2);
      const float* lg = low + (a.dec ? 0 : a.ra);
      for (int c = tid; c < ncol; c += kT) {
        const int64_t ch = (int64_t)h * dv + j0 + c;
        const float x = !LOW || a.og ? (c == tid ? x_og : act_load(reinterpret_cast<const TA*>(a.og) + row * a.ldo + ch)) : (low_g ? sog[c] : row_dot(g2 + ch * a.rg, lg, a.rg));
        sog[c] = sigmoid_s(x);
      }
    } else if (KIND == LINREC_GATED) {
      for (int c = tid; c < dk; c += kT) {
        const int64_t ch = (int64_t)h * dk + c;
        const bool own = c == tid;
        sq[c] = silu_x(own ? x_a : act_load(pr + ch));
        sg[c] = forget((own ? x_b : a.gates[row * a.ldg + ch]) + (own ? p_bf : a.gate_b[ch]), own ? p_bi : a.lower[ch], sk + c);
      }
      for (int c = tid; c < ncol; c += kT) sv[c] = c == tid ? x_v : act_load(pr + a.v_col + (int64_t)h * dv + j0 + c);
    } else {
      const float rs = 1.f / sqrtf((float)dk);
      const float zi = gate0 + p_bi, zf = gate1 + p_bf;
      const float ig = a.cap * tanhf(zi / a.cap), fc = a.cap * tanhf(zf / a.cap);
      const float fg = -softplus_x(-fc);
      const float mn = fmaxf(fg + mrun, ig);
      aa = expf(fg + mrun - mn);
      bb = expf(ig - mn);
      mrun = mn;
      float nq = 0.f, z1 = 0.f, z2 = 0.f;
      for (int c = tid; c < dk; c += kT) {
        const float qc = act_round<TA>(c == tid ? x_a : act_load(pr + (int64_t)h * dk + c)) * rs;
        const float kc = act_round<TA>(c == tid ? x_b : act_load(pr + a.k_col + (int64_t)h * dk + c)) * bb;
        sq[c] = qc; sk[c] = kc;
        const float nn = fmaf(aa, sg[c], kc);
        sg[c] = nn;
        nq = fmaf(nn, qc, nq);
      }
      for (int c = tid; c < ncol; c += kT) {
        const int64_t ch = (int64_t)h * dv + j0 + c;
        sv[c] = act_round<TA>(c == tid ? x_v : act_load(pr + a.v_col + ch));
        const float x = c == tid ? x_og : act_load(reinterpret_cast<const TP*>(a.og) + row * a.ldo + ch);
        sog[c] = sigmoid_s(x);
      }
      block_sum3(nq, z1, z2, red);
      den = fmaxf(fabsf(nq), expf(-mn)) + 1e-6f;
    }
    __syncthreads();
    // ---- state pass: partial sums of the read-outs over this thread's rows
    float pa[4] = {}, pb[4] = {};
    if (KIND != LINREC_DELTA) {
      float v4[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) v4[e] = q4 * 4 + e < ncol ? sv[q4 * 4 + e] : 0.f;
#pragma unroll
      for (int i = 0; i < RMAX; ++i) {
        const int r = rg + i * RG;
        if (i < nr) {
          const float k = sk[r], q = sq[r], g = KIND == LINREC_GATED ? sg[r] : aa;
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            S[i][e] = fmaf(g, S[i][e], k * v4[e]);
            pb[e] = fmaf(S[i][e], q, pb[e]);
          }
        }
      }
    } else {
#pragma unroll
      for (int i = 0; i < RMAX; ++i) {
        const int r = rg + i * RG;
        if (i < nr) {
          const float k = sk[r], q = sq[r], g = sg[r];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            S[i][e] *= g;
            pa[e] = fmaf(S[i][e], k, pa[e]);
            pb[e] = fmaf(S[i][e], q, pb[e]);
          }
        }
      }
    }
    if (act_thr) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        part[rg * jc + q4 * 4 + e] = pb[e];
        if (KIND == LINREC_DELTA) part[(RG + rg) * jc + q4 * 4 + e] = pa[e];
      }
    }
    __syncthreads();
    for (int c4 = tid; c4 < ((4 * jc + 31) & ~31); c4 += kT) {   // four lanes per column
      const int c = c4 >> 2;
      float b = 0.f, d = 0.f;
      if (c < jc)
        for (int r = c4 & 3; r < RG; r += 4) {
          b += part[r * jc + c];
          if (KIND == LINREC_DELTA) d += part[(RG + r) * jc + c];
        }
      b += __shfl_xor_sync(0xffffffffu, b, 1); b += __shfl_xor_sync(0xffffffffu, b, 2);
      d += __shfl_xor_sync(0xffffffffu, d, 1); d += __shfl_xor_sync(0xffffffffu, d, 2);
      if ((c4 & 3) || c >= jc) continue;
      if (c >= ncol) b = 0.f;
      if (KIND == LINREC_DELTA) {
        const float u = c < ncol ? bb * (sv[c] - d) : 0.f;
        su[c] = u;
        so[c] = fmaf(u, kq, b);
      } else {
        so[c] = b / den;
      }
    }
    __syncthreads();
    if (KIND == LINREC_DELTA) {
      float u4[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) u4[e] = act_thr ? su[q4 * 4 + e] : 0.f;
#pragma unroll
      for (int i = 0; i < RMAX; ++i) {
        const int r = rg + i * RG;
        if (i < nr) {
          const float k = sk[r];
#pragma unroll
          for (int e = 0; e < 4; ++e) S[i][e] = fmaf(k, u4[e], S[i][e]);
        }
      }
    }
    // ---- head norm and output gate
    float ss = 0.f;
    for (int c = tid; c < ncol; c += kT) ss = fmaf(so[c], so[c], ss);
    ss = block_sum(ss, red);
    if (NS > 1) {
      if (tid == 0) cl_part = ss;
      sm100::cluster_sync_all();
      ss = 0.f;
      for (int r = 0; r < NS; ++r) ss += ld_dsmem(&cl_part, r);
      sm100::cluster_sync_all();
    }
    const float rstd = 1.f / sqrtf(ss / (float)dv + a.eps);
    TA* out = reinterpret_cast<TA*>(a.act) + row * a.lda + (int64_t)h * dv + j0;
    for (int c = tid; c < ncol; c += kT) act_store(out + c, so[c] * rstd * (c == tid ? p_nw : nw[c]) * (KIND == LINREC_GATED ? 1.f : sog[c]));
    __syncthreads();
  }
  // ---- state back
  if (vec) {
#pragma unroll
    for (int i = 0; i < RMAX; ++i)
      if (i < nr) *reinterpret_cast<float4*>(Sp + i * sstep) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
  } else {
#pragma unroll
    for (int i = 0; i < RMAX; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (i < nr && e < ne) Sp[i * sstep + e] = S[i][e];
  }
  if (KIND == LINREC_MLSTM && rank == 0) {
    for (int c = tid; c < dk; c += kT) a.n[((int64_t)slot * a.H + h) * dk + c] = sg[c];
    if (tid == 0) a.m[(int64_t)slot * a.H + h] = mrun;
  }
  if (KIND == LINREC_DELTA && nrow == 1) {
    // one token: its raw rows enter the ring here (no reader of this step looks at that entry); longer segments
    // leave it to linrec_ring_kernel, which runs after every reader
    TA* w = reinterpret_cast<TA*>(a.ring) + ((int64_t)slot * (a.ring_mask + 1) + (pos0 & a.ring_mask)) * a.ring_w;
    if (rank == 0 && h % (a.H / a.G) == 0)
      for (int c = tid; c < dk; c += kT) {
        act_store(w + qb + c, act_load(prow0 + qb + c));
        act_store(w + a.k_col + qb + c, act_load(prow0 + a.k_col + qb + c));
      }
    for (int c = tid; c < ncol; c += kT) {
      const int64_t ch = a.v_col + (int64_t)h * dv + j0 + c;
      act_store(w + ch, act_load(prow0 + ch));
    }
  }
}

// the last rows of every segment of more than one token enter the convolution ring
template <typename TA>
__global__ void __launch_bounds__(256) linrec_ring_kernel(const TA* __restrict__ proj, int64_t ldp, const int* __restrict__ seg_row,
                                                          const int* __restrict__ seg_pos, const int* __restrict__ seg_slot,
                                                          TA* __restrict__ ring, int mask, int64_t w, int keep) {
  griddep_launch();
  griddep_wait();
  const int seg = blockIdx.y, row0 = seg_row[seg], n = seg_row[seg + 1] - row0, slot = seg_slot[seg];
  if (n < 2 || slot < 0) return;
  for (int i = 0; i < keep && i < n; ++i) {
    const int p = seg_pos[seg] + n - 1 - i;
    for (int64_t c = blockIdx.x * 256 + threadIdx.x; c < w; c += gridDim.x * 256)
      ring[((int64_t)slot * (mask + 1) + (p & mask)) * w + c] = proj[(int64_t)(row0 + n - 1 - i) * ldp + c];
  }
}

template <int KIND, typename TP, typename TA, int RMAX, bool LOW>
int launch_step(const LinrecArgs& a, int ns, int segs, size_t smem, cudaStream_t st) {
  auto kern = linrec_step_kernel<KIND, TP, TA, RMAX, LOW>;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)ns, (unsigned)a.H, (unsigned)segs);
  cfg.blockDim = dim3(kT);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  int na = 0;
  attr[na].id = cudaLaunchAttributeClusterDimension;
  attr[na].val.clusterDim.x = (unsigned)ns; attr[na].val.clusterDim.y = 1; attr[na].val.clusterDim.z = 1;
  ++na;
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

// value columns per CTA: a head is one CTA when 16 state rows per thread suffice, else the fewest slices that get there
// (32 rows per thread if nothing does); more slices, down to 16 columns, while the machine has idle SMs
int plan_cols(int64_t H, int64_t dk, int64_t dv, int64_t segs) {
  int best = 0, rows = 0;
  for (int ns = 1; ns <= 8; ++ns) {
    if (best && (ns & (ns - 1))) continue;             // slices by halving
    int jc = (int)((dv + ns - 1) / ns);
    jc = (jc + 3) & ~3;
    if ((dv + jc - 1) / jc != ns || jc > 4 * kT) continue;
    const int RG = kT / (jc / 4), r = (int)((dk + RG - 1) / RG);
    if (r > 32) continue;
    if (!best || rows > 16 || (H * ns * segs <= 160 && jc >= 16)) { best = jc; rows = r; }
  }
  return best;
}

template <int KIND, typename TP, typename TA>
int dispatch_step(LinrecArgs& a, int segs, cudaStream_t st) {
  a.jc = plan_cols(a.H, a.dk, a.dv, segs);
  if (!a.jc) return CB_ERR_SHAPE;
  const int ns = (a.dv + a.jc - 1) / a.jc, RG = kT / (a.jc / 4), rm = (a.dk + RG - 1) / RG;
  const int64_t lown = KIND == LINREC_DELTA ? (a.dec ? 0 : a.ra) + (a.og ? 0 : a.rg) : 0;
  const size_t smem = sizeof(float) * (size_t)(3 * a.dk + 4 * a.jc + ((lown + 3) & ~3) + 2 * RG * a.jc);
  if (smem > 200 * 1024) return CB_ERR_SHAPE;
#define CB_ROWS(R)                                                                        \
  if (rm <= R) {                                                                          \
    if (KIND == LINREC_DELTA && (!a.dec || !a.og)) return launch_step<KIND, TP, TA, R, KIND == LINREC_DELTA>(a, ns, segs, smem, st); \
    return launch_step<KIND, TP, TA, R, false>(a, ns, segs, smem, st);                    \
  }
  CB_ROWS(4) CB_ROWS(8) CB_ROWS(16) CB_ROWS(32)
#undef CB_ROWS
  return CB_ERR_SHAPE;
}

}  // namespace

CB_EXPORT int cb_linrec_args_size() { return (int)sizeof(LinrecArgs); }
// whether the token-by-token kernel takes a head of this size
CB_EXPORT int cb_linrec_supported(int64_t H, int64_t dk, int64_t dv) { return plan_cols(H, dk, dv, 1) > 0; }

// `segs` segments of the recurrence `kind` token by token.  p_f32: projection rows are fp32 (else the activation
// type); f32: activations, ring and low-rank weights are fp32 instead of bf16.
CB_EXPORT int cb_linrec_step(const void* args, int64_t kind, int64_t segs, int64_t p_f32, int64_t f32, void* stream) {
  if (!args || segs < 1 || segs > 65535) return CB_ERR_ARG;
  LinrecArgs a = *(const LinrecArgs*)args;
  if (!a.proj || !a.gates || !a.act || !a.seg_pos || !a.seg_slot || !a.S || a.H < 1 || a.G < 1 || a.H % a.G) return CB_ERR_ARG;
  cudaStream_t st = (cudaStream_t)stream;
  if (kind == LINREC_DELTA) {
    if (!a.ring || a.taps < 1 || a.taps > a.ring_mask + 1 || a.ra % 8 || a.rg % 8) return CB_ERR_ARG;
    if (f32) return dispatch_step<LINREC_DELTA, float, float>(a, (int)segs, st);
    return p_f32 ? dispatch_step<LINREC_DELTA, float, bf16>(a, (int)segs, st) : dispatch_step<LINREC_DELTA, bf16, bf16>(a, (int)segs, st);
  }
  if (kind == LINREC_MLSTM) {
    if (!a.n || !a.m || !a.og || !(a.cap > 0.f)) return CB_ERR_ARG;
    if (f32) return dispatch_step<LINREC_MLSTM, float, float>(a, (int)segs, st);
    return p_f32 ? dispatch_step<LINREC_MLSTM, float, bf16>(a, (int)segs, st) : dispatch_step<LINREC_MLSTM, bf16, bf16>(a, (int)segs, st);
  }
  if (kind == LINREC_GATED) {
    if (!a.gate_b || !a.lower || !a.norm_w || a.G != a.H) return CB_ERR_ARG;
    if (f32) return dispatch_step<LINREC_GATED, float, float>(a, (int)segs, st);
    return p_f32 ? dispatch_step<LINREC_GATED, float, bf16>(a, (int)segs, st) : dispatch_step<LINREC_GATED, bf16, bf16>(a, (int)segs, st);
  }
  return CB_ERR_ARG;
}

// Convolution ring of the segments with more than one token, after everything that reads it.
CB_EXPORT int cb_linrec_ring(const void* proj, int64_t ldp, const void* seg_row, const void* seg_pos, const void* seg_slot,
                             int64_t segs, void* ring, int64_t ring_depth, int64_t ring_w, int64_t taps, int64_t f32, void* stream) {
  if (!proj || !seg_row || !seg_pos || !seg_slot || !ring || segs < 1 || segs > 65535 || taps > ring_depth) return CB_ERR_ARG;
  if (taps < 2) return CB_OK;
  const dim3 grid((unsigned)((ring_w + 1023) / 1024), (unsigned)segs);
  cudaStream_t st = (cudaStream_t)stream;
  if (f32)
    return (int)cb_launch(linrec_ring_kernel<float>, grid, dim3(256), 0, st, (const float*)proj, ldp, (const int*)seg_row,
                          (const int*)seg_pos, (const int*)seg_slot, (float*)ring, (int)(ring_depth - 1), ring_w, (int)(taps - 1));
  return (int)cb_launch(linrec_ring_kernel<bf16>, grid, dim3(256), 0, st, (const bf16*)proj, ldp, (const int*)seg_row,
                        (const int*)seg_pos, (const int*)seg_slot, (bf16*)ring, (int)(ring_depth - 1), ring_w, (int)(taps - 1));
}
