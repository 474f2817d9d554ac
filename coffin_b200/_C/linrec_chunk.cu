// Recurrent mixers over prompts: the recurrences of linrec.cu in chunks of 16 tokens on the tensor cores.
//
// Inside a chunk everything is relative to the state S_0 at its start (decays are products of factors <= 1, taken
// pairwise as differences of cumulative logarithms, so nothing overflows however strong they are):
//
//   delta :  u = T (v - S_0^T k~),  o = S_0^T q~ + B u,  S <- G S_0 + k^ u^T
//            k~_t = G_t k_t,  q~_t = G_t q_t,  k^_s = (G / G_s) k_s,  B_ts = sum_c q_t k_s G_t / G_s  (s <= t),
//            T = (I + diag(beta) A)^-1 diag(beta),  A_ts = sum_c k_t k_s G_t / G_s  (s < t)
//   mLSTM :  u = v and the same with scalar decays under the running maximum; its normaliser n is one more value
//            column, v = 1.
//   gated :  u = v, k = 1 - f, decays per channel, no normaliser.
//
// `prep` (one CTA per chunk and head) computes those factors in fp32; `scan` (two warps per 16 value columns) walks
// the chunks with S^T in accumulator registers.  A gated state is linear in its start, so where heads are few its scan is cut into
// blocks of chunks that run side by side: `states` leaves what every block adds and how much of its start it keeps, and a
// block of the scan folds the blocks before it first.  The 32-bit quantities enter the products as a bf16 head plus a bf16
// remainder (three products, 16 mantissa bits), the sums and the state are fp32; `finish` applies the head norm and
// the output gate.  A segment may start and end anywhere: its last chunk is padded with neutral tokens.
#include "linrec.cuh"

namespace {

constexpr int C = 16;
constexpr float kLog2e = 1.4426950408889634f;

struct ChunkArgs {
  LinrecArgs r;
  unsigned char* image;      // per (chunk, head): the operand block that scan stages (layout below)
  float* v;                  // delta: convolved values [rows, H * dv]
  float* o; int64_t ldo_;    // read-outs [rows, H * dv]
  float* gi; float* gf; float* gm; float* gb;   // mLSTM, [rows, H]: input log gate, forget log gate, m after / before the token
  float* nq;                 // mLSTM: n . q [rows, H]
  int segs;
  // gated, blocks of `per` chunks (0: not cut): [entries, H, slices * kST, NT] float4 - the segment's first state, then what the
  // blocks leave from nothing (the first from that state) - and the products of the blocks' decays [entries, H, DK]
  float4* part; float* keep; int per;
};
__host__ __device__ __forceinline__ int64_t entry_index(int row0, int seg, int per) { return (int64_t)(row0 / (16 * per)) + 2 * seg; }

// operand block, bf16 units, row pitch P = DK + 8:  X head [NX][P] | X remainder | K^ head [16][P] | K^ remainder |
// T head [16][24] | T remainder | B head | B remainder | G fp32 [DK].   NX = 32 (k~ then q~) for delta, else 16 (q~).
template <int KIND, int DK> struct Image {
  static constexpr int P = DK + 8, NX = KIND == LINREC_DELTA ? 32 : 16;
  static constexpr int xh = 0, xl = xh + NX * P, kh = xl + NX * P, kl = kh + C * P, th = kl + C * P, tl = th + C * 24, bh = tl + C * 24,
                       bl = bh + C * 24, g = bl + C * 24, total = g + 2 * DK;
  static constexpr size_t bytes = (size_t)total * 2;
};

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t split_head(float& x, float& y) {
  const uint32_t h = pack_bf162(x, y);
  x -= __uint_as_float(h << 16);
  y -= __uint_as_float(h & 0xffff0000u);
  return h;
}
__device__ __forceinline__ void put2(bf16* head, bf16* rem, float x, float y) {
  *reinterpret_cast<uint32_t*>(head) = split_head(x, y);
  *reinterpret_cast<uint32_t*>(rem) = pack_bf162(x, y);
}
__device__ __forceinline__ void put1(bf16* head, bf16* rem, float x) {
  const bf16 h = __float2bfloat16(x);
  *head = h;
  *rem = __float2bfloat16(x - __bfloat162float(h));
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
__device__ __forceinline__ float2 ld2(const bf16* p) {
  const uint32_t v = *reinterpret_cast<const uint32_t*>(p);
  return make_float2(__uint_as_float(v << 16), __uint_as_float(v & 0xffff0000u));
}
// operand blocks of a segment are consecutive; blocks of different segments never coincide
__device__ __forceinline__ int64_t block_index(int row0, int seg, int chunk) { return (int64_t)(row0 >> 4) + seg + chunk; }

// ---- prep: delta -------------------------------------------------------------------------------
constexpr int kPT = 128;
template <int DK, int TAPS>
__global__ void __launch_bounds__(kPT, 7) chunk_prep_delta_kernel(const ChunkArgs ca) {
  using I = Image<LINREC_DELTA, DK>;
  constexpr int LD = DK + 4;
  const LinrecArgs& a = ca.r;
  extern __shared__ __align__(16) float sm[];
  float* sq = sm;                    // [C][LD]
  float* sk = sq + C * LD;
  float* sL = sk + C * LD;           // cumulative log2 decays, inclusive
  __shared__ float sA[C][C + 1], beta[C], rq[C], rk[C];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.y, seg = blockIdx.z;
  griddep_launch();
  griddep_wait();
  const int row0 = a.seg_row[seg], n = a.seg_row[seg + 1] - row0, slot = a.seg_slot[seg], pos0 = a.seg_pos[seg];
  const int c0 = blockIdx.x * C;
  if (c0 >= n || slot < 0) return;
  const int m = min(C, n - c0);
  const bf16* proj = reinterpret_cast<const bf16*>(a.proj);
  const bf16* ring = reinterpret_cast<const bf16*>(a.ring) + (int64_t)slot * (a.ring_mask + 1) * a.ring_w;
  const int qb = (h / (a.H / a.G)) * a.dk;
  bf16* im = reinterpret_cast<bf16*>(ca.image + (block_index(row0, seg, blockIdx.x) * a.H + h) * I::bytes);

  // short convolution + SiLU, a channel pair per thread
  auto raw = [&](int rel, int64_t ch) -> float2 {                // rel: token of the segment, possibly before it
    if (rel >= 0) return ld2(proj + (int64_t)(row0 + rel) * a.ldp + ch);
    const int p = pos0 + rel;
    if (p < 0) return make_float2(0.f, 0.f);
    return ld2(ring + (int64_t)(p & a.ring_mask) * a.ring_w + ch);
  };
  const int np = a.dk + (a.dv >> 1);                             // pairs: q, k, v
  for (int e = tid; e < np; e += kPT) {
    const int kd = a.dk >> 1;
    const int part = e < kd ? 0 : (e < a.dk ? 1 : 2);
    const int c = 2 * (part == 0 ? e : (part == 1 ? e - kd : e - a.dk));
    const int64_t ch = part == 0 ? qb + c : (part == 1 ? a.k_col + qb + c : a.v_col + (int64_t)h * a.dv + c);
    auto emit = [&](int t, float x, float y) {
      x = silu_s(x); y = silu_s(y);
      if (t >= m) x = y = 0.f;
      if (part == 0) { sq[t * LD + c] = x; sq[t * LD + c + 1] = y; }
      else if (part == 1) { sk[t * LD + c] = x; sk[t * LD + c + 1] = y; }
      else if (t < m) *reinterpret_cast<float2*>(ca.v + (int64_t)(row0 + c0 + t) * a.H * a.dv + (int64_t)h * a.dv + c) = make_float2(x, y);
    };
    if (TAPS > 0) {
      constexpr int N = TAPS > 0 ? TAPS : 1;
      float wx[N], wy[N];
      float2 x[C + N - 1];
#pragma unroll
      for (int j = 0; j < N; ++j) { wx[j] = a.conv_w[ch * N + j]; wy[j] = a.conv_w[(ch + 1) * N + j]; }
#pragma unroll
      for (int i = 0; i < C + N - 1; ++i) x[i] = i - (N - 1) < m ? raw(c0 + i - (N - 1), ch) : make_float2(0.f, 0.f);
#pragma unroll
      for (int t = 0; t < C; ++t) {
        float ax = 0.f, ay = 0.f;
#pragma unroll
        for (int j = 0; j < N; ++j) { ax = fmaf(wx[j], x[t + j].x, ax); ay = fmaf(wy[j], x[t + j].y, ay); }
        emit(t, ax, ay);
      }
    } else {
      for (int t = 0; t < C; ++t) {
        float ax = 0.f, ay = 0.f;
        if (t < m)
          for (int j = 0; j < a.taps; ++j) {
            const float2 x = raw(c0 + t - (a.taps - 1) + j, ch);
            ax = fmaf(a.conv_w[ch * a.taps + j], x.x, ax);
            ay = fmaf(a.conv_w[(ch + 1) * a.taps + j], x.y, ay);
          }
        emit(t, ax, ay);
      }
    }
  }
  // cumulative log decays, a channel per thread; channels beyond dk are neutral and empty
  const float ea = expf(a.A_log[h]) * kLog2e;
  for (int c = tid; c < DK; c += kPT) {
    float L = 0.f;
    const bool ok = c < a.dk;
    const float db = ok ? a.dt_bias[(int64_t)h * a.dk + c] : 0.f;
    float x[C];
#pragma unroll
    for (int t = 0; t < C; ++t) x[t] = ok && t < m ? a.dec[(int64_t)(row0 + c0 + t) * a.ldd + (int64_t)h * a.dk + c] : 0.f;
#pragma unroll
    for (int t = 0; t < C; ++t) {
      if (ok && t < m) L -= ea * softplus_s(x[t] + db);
      sL[t * LD + c] = L;
    }
    if (!ok)
      for (int t = 0; t < C; ++t) { sq[t * LD + c] = 0.f; sk[t * LD + c] = 0.f; }
  }
  if (tid < C) beta[tid] = tid < m ? sigmoid_x(a.gates[(int64_t)(row0 + c0 + tid) * a.ldg + h]) : 0.f;
  __syncthreads();
  for (int t = warp; t < C; t += kPT / 32) {
    float q2 = 0.f, k2 = 0.f;
#pragma unroll
    for (int c = lane; c < DK; c += 32) { q2 = fmaf(sq[t * LD + c], sq[t * LD + c], q2); k2 = fmaf(sk[t * LD + c], sk[t * LD + c], k2); }
    q2 = warp_sum(q2); k2 = warp_sum(k2);
    if (lane == 0) { rq[t] = 1.f / (sqrtf(q2 + 1e-6f) * sqrtf((float)a.dk)); rk[t] = 1.f / sqrtf(k2 + 1e-6f); }
  }
  __syncthreads();
  // operand rows; sq / sk become the unit vectors
  for (int e = tid; e < C * (DK / 2); e += kPT) {
    const int t = e / (DK / 2), c = (e % (DK / 2)) * 2;
    const float qx = sq[t * LD + c] * rq[t], qy = sq[t * LD + c + 1] * rq[t], kx = sk[t * LD + c] * rk[t], ky = sk[t * LD + c + 1] * rk[t];
    sq[t * LD + c] = qx; sq[t * LD + c + 1] = qy; sk[t * LD + c] = kx; sk[t * LD + c + 1] = ky;
    const float Lx = sL[t * LD + c], Ly = sL[t * LD + c + 1];
    const float gx = ex2(Lx), gy = ex2(Ly);
    put2(im + I::xh + t * I::P + c, im + I::xl + t * I::P + c, kx * gx, ky * gy);
    put2(im + I::xh + (C + t) * I::P + c, im + I::xl + (C + t) * I::P + c, qx * gx, qy * gy);
    put2(im + I::kh + t * I::P + c, im + I::kl + t * I::P + c, kx * ex2(sL[(C - 1) * LD + c] - Lx), ky * ex2(sL[(C - 1) * LD + c + 1] - Ly));
  }
  for (int c = tid; c < DK; c += kPT) reinterpret_cast<float*>(im + I::g)[c] = ex2(sL[(C - 1) * LD + c]);
  __syncthreads();
  // pairwise products: a warp takes tokens t = warp, 7 - warp, 8 + warp, 15 - warp (equal numbers of pairs)
#pragma unroll 1
  for (int i = 0; i < 4; ++i) {
    const int t = i == 0 ? warp : (i == 1 ? 7 - warp : (i == 2 ? 8 + warp : 15 - warp));
    float kt[DK / 32], qt[DK / 32], Lt[DK / 32];
#pragma unroll
    for (int j = 0; j < DK / 32; ++j) { kt[j] = sk[t * LD + lane + 32 * j]; qt[j] = sq[t * LD + lane + 32 * j]; Lt[j] = sL[t * LD + lane + 32 * j]; }
#pragma unroll 1
    for (int s = 0; s <= t; s += 2) {                            // two tokens s: four sums share the reduction tree
      float pa[2] = {0.f, 0.f}, pb[2] = {0.f, 0.f};
#pragma unroll
      for (int u = 0; u < 2; ++u) {                              // s + 1 may be t + 1 <= 15 (discarded; its factor is cut off at 1)
#pragma unroll
        for (int j = 0; j < DK / 32; ++j) {
          const float x = sk[(s + u) * LD + lane + 32 * j] * ex2(fminf(Lt[j] - sL[(s + u) * LD + lane + 32 * j], 0.f));
          pa[u] = fmaf(kt[j], x, pa[u]);
          pb[u] = fmaf(qt[j], x, pb[u]);
        }
      }
      // halves of the warp keep s / s + 1, quarters keep A / B
      const bool hi = lane & 16, hq = lane & 8;
      float ka = hi ? pa[1] : pa[0], kb = hi ? pb[1] : pb[0];
      ka += __shfl_xor_sync(0xffffffffu, hi ? pa[0] : pa[1], 16);
      kb += __shfl_xor_sync(0xffffffffu, hi ? pb[0] : pb[1], 16);
      float k = hq ? kb : ka;
      k += __shfl_xor_sync(0xffffffffu, hq ? ka : kb, 8);
      k += __shfl_xor_sync(0xffffffffu, k, 4);
      k += __shfl_xor_sync(0xffffffffu, k, 2);
      k += __shfl_xor_sync(0xffffffffu, k, 1);
      const int su = s + (hi ? 1 : 0);
      if ((lane & 7) == 0 && su <= t) {
        if (hq) put1(im + I::bh + t * 24 + su, im + I::bl + t * 24 + su, k);
        else sA[t][su] = k * beta[t];
      }
    }
    if (lane > t && lane < C) put1(im + I::bh + t * 24 + lane, im + I::bl + t * 24 + lane, 0.f);
  }
  __syncthreads();
  // T = (I + diag(beta) A)^-1 diag(beta): one column per thread
  if (tid < C) {
    float x[C];
#pragma unroll
    for (int t = 0; t < C; ++t) {
      float s = t == tid ? beta[t] : 0.f;
#pragma unroll
      for (int u = 0; u < t; ++u) s = fmaf(-sA[t][u], x[u], s);
      x[t] = s;
      put1(im + I::th + t * 24 + tid, im + I::tl + t * 24 + tid, s);
    }
  }
}

// ---- prep: mLSTM -------------------------------------------------------------------------------
// Log gates and the running maximum, one block per (head, segment): m_t = max(F_t + m_0, M_t) with (F, M) the prefix of
// the pairs (f, i) under (F, M) o (f, i) = (F + f, max(M + f, i)); the segment's last m becomes the slot's.
constexpr int kGT = 512;
__global__ void __launch_bounds__(kGT) chunk_gates_mlstm_kernel(const ChunkArgs ca) {
  const LinrecArgs& a = ca.r;
  __shared__ float wF[kGT / 32], wM[kGT / 32], m_s;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x, seg = blockIdx.y;
  griddep_launch();
  griddep_wait();
  const int row0 = a.seg_row[seg], n = a.seg_row[seg + 1] - row0, slot = a.seg_slot[seg];
  if (slot < 0 || n < 1) return;
  float m0 = a.m[(int64_t)slot * a.H + h];
  const float bi = a.gate_b[h], bf = a.gate_b[a.H + h];
  for (int t0 = 0; t0 < n; t0 += kGT) {
    const int t = t0 + tid;
    const int64_t row = row0 + t;
    float ig = -INFINITY, fg = 0.f;
    if (t < n) {
      ig = a.cap * tanhf((a.gates[row * a.ldg + h] + bi) / a.cap);
      fg = -softplus_x(-a.cap * tanhf((a.gates[row * a.ldg + a.H + h] + bf) / a.cap));
    }
    float F = fg, M = ig;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float Fp = __shfl_up_sync(0xffffffffu, F, o), Mp = __shfl_up_sync(0xffffffffu, M, o);
      if (lane >= o) { M = fmaxf(Mp + F, M); F += Fp; }
    }
    if (lane == 31) { wF[warp] = F; wM[warp] = M; }
    __syncthreads();
    float mw = m0;                                               // m before this warp's tokens
    for (int w = 0; w < warp; ++w) mw = fmaxf(wF[w] + mw, wM[w]);
    const float mt = fmaxf(F + mw, M);
    float mb = __shfl_up_sync(0xffffffffu, mt, 1);
    if (lane == 0) mb = mw;
    if (t < n) {
      const int64_t i = row * a.H + h;
      ca.gi[i] = ig; ca.gf[i] = fg; ca.gm[i] = mt; ca.gb[i] = mb;
    }
    if (t == min(n, t0 + kGT) - 1) m_s = mt;
    __syncthreads();
    m0 = m_s;
    __syncthreads();
  }
  if (tid == 0) a.m[(int64_t)slot * a.H + h] = m0;
}

template <int DK>
__global__ void __launch_bounds__(64) chunk_prep_mlstm_kernel(const ChunkArgs ca) {
  using I = Image<LINREC_MLSTM, DK>;
  constexpr int P = I::P;
  const LinrecArgs& a = ca.r;
  extern __shared__ __align__(16) unsigned char smem[];
  bf16* sq = reinterpret_cast<bf16*>(smem);            // [C][P]
  bf16* sk = sq + C * P;
  __shared__ float F[C], ii[C], mm[C], m_start;
  const int tid = threadIdx.x, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
  const int h = blockIdx.y, seg = blockIdx.z;
  griddep_launch();
  griddep_wait();
  const int row0 = a.seg_row[seg], n = a.seg_row[seg + 1] - row0, slot = a.seg_slot[seg];
  const int c0 = blockIdx.x * C;
  if (c0 >= n || slot < 0) return;
  const int m = min(C, n - c0);
  const bf16* proj = reinterpret_cast<const bf16*>(a.proj) + (int64_t)(row0 + c0) * a.ldp + (int64_t)h * a.dk;
  bf16* im = reinterpret_cast<bf16*>(ca.image + (block_index(row0, seg, blockIdx.x) * a.H + h) * I::bytes);
  for (int e = tid; e < C * (DK / 8); e += 64) {
    const int t = e / (DK / 8), c = (e % (DK / 8)) * 8;
    const bool ok = t < m && c < a.dk;
    const uint4 z = make_uint4(0, 0, 0, 0);
    *reinterpret_cast<uint4*>(sq + t * P + c) = ok ? *reinterpret_cast<const uint4*>(proj + (int64_t)t * a.ldp + c) : z;
    *reinterpret_cast<uint4*>(sk + t * P + c) = ok ? *reinterpret_cast<const uint4*>(proj + (int64_t)t * a.ldp + a.k_col + c) : z;
  }
  if (tid < 32) {
    const int64_t i = (int64_t)(row0 + c0 + lane) * a.H + h;
    const bool ok = lane < m;
    float f = ok ? ca.gf[i] : 0.f;
#pragma unroll
    for (int o = 1; o < C; o <<= 1) {
      const float p = __shfl_up_sync(0xffffffffu, f, o);
      if (lane >= o) f += p;
    }
    if (lane < C) {
      const int64_t il = (int64_t)(row0 + c0 + m - 1) * a.H + h;
      F[lane] = f;
      ii[lane] = ok ? ca.gi[i] : -INFINITY;
      mm[lane] = ca.gm[ok ? i : il];
    }
    if (lane == 0) m_start = ca.gb[i];
  }
  __syncthreads();
  const float rs = 1.f / sqrtf((float)a.dk), FC = F[C - 1], mC = mm[C - 1];
  for (int e = tid; e < C * (DK / 2); e += 64) {
    const int t = e / (DK / 2), c = (e % (DK / 2)) * 2;
    const float2 q = ld2(sq + t * P + c), k = ld2(sk + t * P + c);
    const float wq = t < m ? rs * expf(F[t] + m_start - mm[t]) : 0.f, wk = t < m ? expf(FC - F[t] + ii[t] - mC) : 0.f;
    put2(im + I::xh + t * P + c, im + I::xl + t * P + c, q.x * wq, q.y * wq);
    put2(im + I::kh + t * P + c, im + I::kl + t * P + c, k.x * wk, k.y * wk);
  }
  const float G = expf(FC + m_start - mC);
  for (int c = tid; c < DK; c += 64) reinterpret_cast<float*>(im + I::g)[c] = G;
  if (tid < 32) {                                                // B = (q k^T) * weights: bf16 operands as they are
    float s[2][4] = {};
#pragma unroll
    for (int k = 0; k < DK / 16; ++k) {
      uint32_t qa[4], b[4];
      ldsm4(qa, sq + (lane & 15) * P + k * 16 + (lane >> 4) * 8);
      ldsm4(b, sk + ((lane & 7) + ((lane >> 4) << 3)) * P + k * 16 + ((lane >> 3) & 1) * 8);
      mma(s[0], qa, b[0], b[1]);
      mma(s[1], qa, b[2], b[3]);
    }
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = g4 + (e >> 1) * 8, u = i * 8 + t4 * 2 + (e & 1);
        const float w = u <= t && t < m ? rs * expf(F[t] - F[u] + ii[u] - mm[t]) : 0.f;
        put1(im + I::bh + t * 24 + u, im + I::bl + t * 24 + u, s[i][e] * w);
      }
  }
}

// ---- prep: gated --------------------------------------------------------------------------------
// Decays below 2^-60 a token are cut off there: the state is an average of values, so what they would leave is far below its
// rounding, and cumulative logarithms stay short enough to subtract.
template <int DK>
__global__ void __launch_bounds__(kPT, 7) chunk_prep_gated_kernel(const ChunkArgs ca) {
  using I = Image<LINREC_GATED, DK>;
  constexpr int LD = DK + 4;
  const LinrecArgs& a = ca.r;
  extern __shared__ __align__(16) float sm[];
  float* sq = sm;                    // [C][LD]
  float* sk = sq + C * LD;
  float* sL = sk + C * LD;           // cumulative log2 decays, inclusive
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.y, seg = blockIdx.z;
  griddep_launch();
  griddep_wait();
  const int row0 = a.seg_row[seg], n = a.seg_row[seg + 1] - row0, slot = a.seg_slot[seg];
  const int c0 = blockIdx.x * C;
  if (c0 >= n || slot < 0) return;
  const int m = min(C, n - c0);
  const bf16* proj = reinterpret_cast<const bf16*>(a.proj) + (int64_t)(row0 + c0) * a.ldp + (int64_t)h * a.dk;
  const float* gates = a.gates + (int64_t)(row0 + c0) * a.ldg + (int64_t)h * a.dk;
  bf16* im = reinterpret_cast<bf16*>(ca.image + (block_index(row0, seg, blockIdx.x) * a.H + h) * I::bytes);
  // a channel per thread; channels beyond dk and tokens beyond the segment are neutral and empty
  for (int c = tid; c < DK; c += kPT) {
    const bool ok = c < a.dk;
    const float low = ok ? a.lower[(int64_t)h * a.dk + c] : 0.f, bias = ok ? a.gate_b[(int64_t)h * a.dk + c] : 0.f;
    float z[C], q[C], L = 0.f;
#pragma unroll
    for (int t = 0; t < C; ++t) {
      z[t] = ok && t < m ? gates[(int64_t)t * a.ldg + c] : 0.f;
      q[t] = ok && t < m ? __bfloat162float(proj[(int64_t)t * a.ldp + c]) : 0.f;
    }
#pragma unroll
    for (int t = 0; t < C; ++t) {
      float in = 0.f;
      if (ok && t < m) L += fmaxf(log2f(forget(z[t] + bias, low, &in)), -60.f);
      sq[t * LD + c] = silu_s(q[t]);
      sk[t * LD + c] = in;
      sL[t * LD + c] = L;
    }
    reinterpret_cast<float*>(im + I::g)[c] = ex2(L);
  }
  __syncthreads();
  for (int e = tid; e < C * (DK / 2); e += kPT) {
    const int t = e / (DK / 2), c = (e % (DK / 2)) * 2, i = t * LD + c, l = (C - 1) * LD + c;
    put2(im + I::xh + t * I::P + c, im + I::xl + t * I::P + c, sq[i] * ex2(sL[i]), sq[i + 1] * ex2(sL[i + 1]));
    put2(im + I::kh + t * I::P + c, im + I::kl + t * I::P + c, sk[i] * ex2(sL[l] - sL[i]), sk[i + 1] * ex2(sL[l + 1] - sL[i + 1]));
  }
  // pairwise products: a warp takes tokens t = warp, 7 - warp, 8 + warp, 15 - warp (equal numbers of pairs)
#pragma unroll 1
  for (int i = 0; i < 4; ++i) {
    const int t = i == 0 ? warp : (i == 1 ? 7 - warp : (i == 2 ? 8 + warp : 15 - warp));
    float qt[DK / 32], Lt[DK / 32];
#pragma unroll
    for (int j = 0; j < DK / 32; ++j) { qt[j] = sq[t * LD + lane + 32 * j]; Lt[j] = sL[t * LD + lane + 32 * j]; }
#pragma unroll 1
    for (int s = 0; s <= t; s += 4) {                            // four tokens s share the reduction tree; those after t are discarded
      float p[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int u = 0; u < 4; ++u)
#pragma unroll
        for (int j = 0; j < DK / 32; ++j) {
          const int at = (s + u) * LD + lane + 32 * j;
          p[u] = fmaf(qt[j], sk[at] * ex2(fminf(Lt[j] - sL[at], 0.f)), p[u]);
        }
      const bool hi = lane & 16, hq = lane & 8;                  // halves of the warp keep tokens 0, 1 / 2, 3, quarters one of them
      float x = hi ? p[2] : p[0], y = hi ? p[3] : p[1];
      x += __shfl_xor_sync(0xffffffffu, hi ? p[0] : p[2], 16);
      y += __shfl_xor_sync(0xffffffffu, hi ? p[1] : p[3], 16);
      float k = hq ? y : x;
      k += __shfl_xor_sync(0xffffffffu, hq ? x : y, 8);
      k += __shfl_xor_sync(0xffffffffu, k, 4);
      k += __shfl_xor_sync(0xffffffffu, k, 2);
      k += __shfl_xor_sync(0xffffffffu, k, 1);
      const int su = s + (hi ? 2 : 0) + (hq ? 1 : 0);
      if ((lane & 7) == 0 && su <= t) put1(im + I::bh + t * 24 + su, im + I::bl + t * 24 + su, k);
    }
    if (lane > t && lane < C) put1(im + I::bh + t * 24 + lane, im + I::bl + t * 24 + lane, 0.f);
  }
}

// ---- scan ---------------------------------------------------------------------------------------
// A CTA owns 32 value columns of a head: two column groups of 16, each shared by two warps that hold half of the key
// channels.  The halves' partial read-outs meet in shared memory once per chunk; both then know u and update their half
// of the state.
constexpr int kST = 128;
// bf16 values of a chunk, staged as [token][32 columns] with pitch kVP: the fragments (columns x tokens) of column group cg
constexpr int kVP = 40;
__device__ __forceinline__ void value_frags(uint32_t* u, const bf16* vs, int cg, int lane) {
  ldsm4t(u, vs + ((lane & 7) + ((lane >> 4) << 3)) * kVP + cg * 16 + ((lane >> 3) & 1) * 8);
}
// Gated: what a block of chunks leaves (all but the last of a segment), the same rows and columns per thread as in the scan.
template <int DK, int STAGES>
__global__ void __launch_bounds__(kST) chunk_states_kernel(const ChunkArgs ca, int slices) {
  using I = Image<LINREC_GATED, DK>;
  constexpr int P = I::P, NT = DK / 16, KB = 2 * C * P * 2;      // bytes of K^ head and remainder
  constexpr int VB = C * kVP * 2, SB = KB + DK * 4 + VB;
  const LinrecArgs& a = ca.r;
  extern __shared__ __align__(16) unsigned char smem[];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, cg = warp >> 1, half = warp & 1, g4 = lane >> 2, t4 = lane & 3;
  const int h = blockIdx.y, seg = blockIdx.z, kc = half * (DK / 2), slice = blockIdx.x % slices, blk = blockIdx.x / slices;
  griddep_launch();
  griddep_wait();
  const int row0 = a.seg_row[seg], n = a.seg_row[seg + 1] - row0, slot = a.seg_slot[seg];
  const int chunks = (n + C - 1) / C, c_lo = blk * ca.per, c_hi = c_lo + ca.per;
  if (slot < 0 || n < 1 || c_hi >= chunks) return;               // the last block's state is the scan's
  const int va = (slice * 2 + cg) * 16 + g4, vb = va + 8;
  const int64_t entry = entry_index(row0, seg, ca.per) + blk;
  float4* out = ca.part + ((entry * a.H + h) * slices + slice) * (kST * NT) + tid;
  const int64_t ostep = (int64_t)a.H * slices * (kST * NT);      // next entry
  const unsigned char* img = ca.image + (block_index(row0, seg, c_lo) * a.H + h) * I::bytes + tid * 16;
  const size_t istep = (size_t)a.H * I::bytes;
  const uint32_t sb = (uint32_t)__cvta_generic_to_shared(smem) + tid * 16;
  const int vt = tid / 4, vc = slice * 32 + (tid % 4) * 8;       // token and first column this thread copies
  const bool vok = vc < a.dv;
  const bf16* vsrc = vok ? reinterpret_cast<const bf16*>(a.proj) + (int64_t)(row0 + c_lo * C + vt) * a.ldp + a.v_col + (int64_t)h * a.dv + vc
                         : reinterpret_cast<const bf16*>(a.proj);
  const int64_t vstep = vok ? C * a.ldp : 0;
  const int vbytes = vok ? 16 : 0;
  const uint32_t vdst = (uint32_t)__cvta_generic_to_shared(smem) + KB + DK * 4 + vt * kVP * 2 + (tid % 4) * 16;
  auto load = [&](int ch, int stage) {                           // chunk of the block; every chunk of it is whole
    const unsigned char* src = img + (size_t)ch * istep;
    const uint32_t dst = sb + stage * SB;
    constexpr int full = KB / 16 / kST, rest = KB / 16 % kST;
#pragma unroll
    for (int i = 0; i < full; ++i)
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + i * kST * 16), "l"(src + I::kh * 2 + i * kST * 16) : "memory");
    if (tid < rest)
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + full * kST * 16), "l"(src + I::kh * 2 + full * kST * 16) : "memory");
    if (tid < DK / 4) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + KB), "l"(src + I::g * 2) : "memory");
    if (vt < C)
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(vdst + stage * SB), "l"(vsrc + ch * vstep), "r"(vbytes) : "memory");
  };
#pragma unroll
  for (int s = 0; s < STAGES - 1; ++s) {
    if (s < ca.per) load(s, s);
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  float S[NT][4], keep[NT][2];
  const bool keeps = slice == 0 && cg == 0;                      // the decays are the same for every column
  const float* Sg = a.S + ((int64_t)slot * a.H + h) * a.dk * a.dv;
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    keep[i][0] = keep[i][1] = 1.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = kc + i * 8 + t4 * 2 + (e & 1), v = e >> 1 ? vb : va;
      S[i][e] = blk == 0 && c < a.dk && v < a.dv ? Sg[(int64_t)c * a.dv + v] : 0.f;
    }
    if (blk == 0) out[i * kST] = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
  }
  int stage = 0;
  for (int ch = 0; ch < ca.per; ++ch) {
    asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");
    __syncthreads();
    if (ch + STAGES - 1 < ca.per) load(ch + STAGES - 1, stage == 0 ? STAGES - 1 : stage - 1);
    asm volatile("cp.async.commit_group;" ::: "memory");
    const unsigned char* st = smem + stage * SB;
    const bf16* kh = reinterpret_cast<const bf16*>(st) + (lane & 15) * P + kc + (lane >> 4) * 8;
    const float* G = reinterpret_cast<const float*>(st + KB) + kc + t4 * 2;
    stage = stage + 1 == STAGES ? 0 : stage + 1;
    uint32_t u[4];
    value_frags(u, reinterpret_cast<const bf16*>(st + KB + DK * 4), cg, lane);
#pragma unroll
    for (int k = 0; k < NT / 2; ++k) {
      uint32_t bh[4], bl[4];
      ldsm4t(bh, kh + k * 16);
      ldsm4t(bl, kh + C * P + k * 16);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float2 gg = *reinterpret_cast<const float2*>(G + (2 * k + i) * 8);
        float* s = S[2 * k + i];
        s[0] *= gg.x; s[1] *= gg.y; s[2] *= gg.x; s[3] *= gg.y;
        if (keeps) { keep[2 * k + i][0] *= gg.x; keep[2 * k + i][1] *= gg.y; }
        mma(s, u, bh[2 * i], bh[2 * i + 1]);
        mma(s, u, bl[2 * i], bl[2 * i + 1]);
      }
    }
  }
  out += ostep;
#pragma unroll
  for (int i = 0; i < NT; ++i) out[i * kST] = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
  if (keeps && g4 == 0) {
    float* kp = ca.keep + ((entry + 1) * a.H + h) * DK + kc + t4 * 2;
#pragma unroll
    for (int i = 0; i < NT; ++i) *reinterpret_cast<float2*>(kp + i * 8) = make_float2(keep[i][0], keep[i][1]);
  }
}

template <int KIND, int DK, int STAGES>
__global__ void __launch_bounds__(kST) chunk_scan_kernel(const ChunkArgs ca, int slices) {
  using I = Image<KIND, DK>;
  constexpr int P = I::P, NT = DK / 16, NR = I::NX / 8;         // NT: n-tiles (8 channels) of this warp's half
  const LinrecArgs& a = ca.r;
  extern __shared__ __align__(16) unsigned char smem[];
  __shared__ float xch[4][NR * 4][32];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, cg = warp >> 1, half = warp & 1, g4 = lane >> 2, t4 = lane & 3;
  constexpr bool GAT = KIND == LINREC_GATED;
  const int h = blockIdx.y, seg = blockIdx.z, kc = half * (DK / 2);      // first channel of the half
  const int slice = GAT ? (int)blockIdx.x % slices : (int)blockIdx.x, blk = GAT ? (int)blockIdx.x / slices : 0;
  griddep_launch();
  griddep_wait();
  const int row0 = a.seg_row[seg], n = a.seg_row[seg + 1] - row0, slot = a.seg_slot[seg];
  if (slot < 0 || n < 1) return;
  const int all = (n + C - 1) / C, per = GAT && ca.per ? ca.per : all, first = blk * per, chunks = min(all, first + per) - first;
  if (GAT && chunks < 1) return;
  const bool cut = GAT && per < all, last = !cut || first + per >= all;
  // mLSTM: the slice after the value columns carries the normaliser as one column whose value is 1
  const bool nrm = KIND == LINREC_MLSTM && blockIdx.x == gridDim.x - 1;
  const int v0 = nrm ? 0 : (slice * 2 + cg) * 16;
  const int vlim = nrm ? (cg == 0 ? 1 : 0) : a.dv;               // columns that exist
  const int va = v0 + g4, vb = va + 8;
  const bool oka = va < vlim, okb = vb < vlim;
  const int64_t sstride = nrm ? 1 : a.dv;
  float* Sg = nrm ? a.n + ((int64_t)slot * a.H + h) * a.dk : a.S + ((int64_t)slot * a.H + h) * a.dk * a.dv;
  float S[NT][4];
  if (!cut) {
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int c = kc + i * 8 + t4 * 2 + (e & 1), v = e >> 1 ? vb : va;
        S[i][e] = c < a.dk && v < vlim ? Sg[(int64_t)c * sstride + v] : 0.f;
      }
  }
  const unsigned char* img = ca.image + (block_index(row0, seg, first) * a.H + h) * I::bytes + tid * 16;
  const size_t istep = (size_t)a.H * I::bytes;
  const uint32_t sbase = (uint32_t)__cvta_generic_to_shared(smem) + tid * 16;
  auto load = [&](int ch, int stage) {
    const unsigned char* src = img + (size_t)ch * istep;
    const uint32_t dst = sbase + stage * (uint32_t)I::bytes;
    constexpr int full = (int)(I::bytes / 16) / kST, rest = (int)(I::bytes / 16) % kST;
#pragma unroll
    for (int i = 0; i < full; ++i)
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + i * kST * 16), "l"(src + i * kST * 16) : "memory");
    if (tid < rest)
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + full * kST * 16), "l"(src + full * kST * 16) : "memory");
  };
  // values of a chunk go through the same ring: [token][32 columns], pitch chosen against bank conflicts
  constexpr int VE = KIND == LINREC_DELTA ? 4 : 2, VP = KIND == LINREC_DELTA ? 36 : kVP, VB = C * VP * VE, VPER = 32 * VE / 16;   // 16-byte pieces a row
  const int64_t ldv = KIND == LINREC_DELTA ? (int64_t)a.H * a.dv : a.ldp;
  const int vt = tid / VPER, vc = slice * 32 + (tid % VPER) * (16 / VE);          // token and first column this thread copies
  const char* vsrc = KIND == LINREC_DELTA
                         ? reinterpret_cast<const char*>(ca.v + (int64_t)(row0 + vt) * ldv + (int64_t)h * a.dv + vc)
                         : reinterpret_cast<const char*>(reinterpret_cast<const bf16*>(a.proj) + (int64_t)(row0 + first * C + vt) * ldv + a.v_col +
                                                         (int64_t)h * a.dv + vc);
  const uint32_t vdst = (uint32_t)__cvta_generic_to_shared(smem) + STAGES * (uint32_t)I::bytes + vt * VP * VE + (tid % VPER) * 16;
  auto load_v = [&](int ch, int stage) {
    if (nrm || vt >= C) return;
    const bool ok = (first + ch) * C + vt < n && vc < a.dv;                // 16-byte pieces never straddle dv (a multiple of 8)
    const char* src = ok ? vsrc + (int64_t)ch * C * ldv * VE : reinterpret_cast<const char*>(a.proj);
    const int bytes = ok ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(vdst + stage * VB), "l"(src), "r"(bytes) : "memory");
  };
  float* op = nrm ? ca.nq + (int64_t)(row0 + half * 8 + t4 * 2) * a.H + h : ca.o + (int64_t)(row0 + first * C + half * 8 + t4 * 2) * ca.ldo_ + (int64_t)h * a.dv + va;
  const int64_t ostep = nrm ? a.H : ca.ldo_;
#pragma unroll
  for (int s = 0; s < STAGES - 1; ++s) {
    if (s < chunks) { load(s, s); load_v(s, s); }
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  if (cut) {                                                     // the state at the block's start, from the blocks before it
    const int64_t e0 = entry_index(row0, seg, per), pstep = (int64_t)a.H * slices * (kST * NT);
    const float4* pp = ca.part + ((e0 * a.H + h) * slices + slice) * (kST * NT) + tid + (blk ? pstep : 0);
    const float* kp = ca.keep + ((e0 + 1) * a.H + h) * DK + kc + t4 * 2;
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const float4 f = pp[i * kST];
      S[i][0] = f.x; S[i][1] = f.y; S[i][2] = f.z; S[i][3] = f.w;
    }
#pragma unroll 1
    for (int j = 1; j < blk; ++j) {
      pp += pstep;
      kp += (int64_t)a.H * DK;
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        const float4 f = pp[i * kST];
        const float2 g = *reinterpret_cast<const float2*>(kp + i * 8);
        S[i][0] = fmaf(g.x, S[i][0], f.x); S[i][1] = fmaf(g.y, S[i][1], f.y);
        S[i][2] = fmaf(g.x, S[i][2], f.z); S[i][3] = fmaf(g.y, S[i][3], f.w);
      }
    }
  }
  int stage = 0;
  for (int ch = 0; ch < chunks; ++ch) {
    asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");
    __syncthreads();
    if (ch + STAGES - 1 < chunks) {
      const int fs = stage == 0 ? STAGES - 1 : stage - 1;
      load(ch + STAGES - 1, fs);
      load_v(ch + STAGES - 1, fs);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    float v[2][4];                                               // [token tile][row lo / hi, token 2t, 2t + 1]
    uint32_t vf[4];                                              // the same packed (gated)
    const unsigned char* vs = smem + STAGES * I::bytes + stage * VB;
    if (GAT) {
      value_frags(vf, reinterpret_cast<const bf16*>(vs), cg, lane);
    } else {
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int idx = (i * 8 + t4 * 2 + (e & 1)) * VP + cg * 16 + g4 + (e >> 1) * 8;
          if (nrm) v[i][e] = cg == 0 && g4 == 0 && e < 2 ? 1.f : 0.f;
          else if (KIND == LINREC_DELTA) v[i][e] = reinterpret_cast<const float*>(vs)[idx];
          else v[i][e] = __bfloat162float(reinterpret_cast<const bf16*>(vs)[idx]);
        }
    }
    const bf16* im = reinterpret_cast<const bf16*>(smem + stage * I::bytes);
    const float* G = reinterpret_cast<const float*>(im + I::g) + kc;
    stage = stage + 1 == STAGES ? 0 : stage + 1;
    // R^T = S^T X^T over this half's channels; the cross terms have accumulators of their own (shorter chains)
    float R[NR][4], R2[NR][4];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      R[i][0] = R[i][1] = R[i][2] = R[i][3] = 0.f;
      R2[i][0] = R2[i][1] = R2[i][2] = R2[i][3] = 0.f;
    }
    const int xr = ((lane & 7) + ((lane >> 4) << 3)) * P + ((lane >> 3) & 1) * 8 + kc;
#pragma unroll
    for (int k = 0; k < NT / 2; ++k) {
      uint32_t ah[4], al[4];
#pragma unroll
      for (int q = 0; q < 4; ++q) {                              // a0: row lo, k; a1: row hi, k; a2 / a3: k + 8
        float x = S[2 * k + (q >> 1)][(q & 1) * 2], y = S[2 * k + (q >> 1)][(q & 1) * 2 + 1];
        ah[q] = split_head(x, y);
        al[q] = pack_bf162(x, y);
      }
#pragma unroll
      for (int j = 0; j < NR / 2; ++j) {
        uint32_t bh[4], bl[4];
        ldsm4(bh, im + I::xh + j * 16 * P + xr + k * 16);
        ldsm4(bl, im + I::xl + j * 16 * P + xr + k * 16);
        mma(R[2 * j], ah, bh[0], bh[1]);
        mma(R[2 * j + 1], ah, bh[2], bh[3]);
        mma(R2[2 * j], al, bh[0], bh[1]);
        mma(R2[2 * j + 1], al, bh[2], bh[3]);
        mma(R2[2 * j], ah, bl[0], bl[1]);
        mma(R2[2 * j + 1], ah, bl[2], bl[3]);
      }
    }
#pragma unroll
    for (int i = 0; i < NR * 4; ++i) {
      R[i >> 2][i & 3] += R2[i >> 2][i & 3];
      xch[warp][i][lane] = R[i >> 2][i & 3];
    }
    asm volatile("bar.sync %0, 64;" ::"r"(1 + cg) : "memory");
#pragma unroll
    for (int i = 0; i < NR * 4; ++i) R[i >> 2][i & 3] += xch[warp ^ 1][i][lane];
    const int mr = ((lane & 7) + ((lane >> 4) << 3)) * 24 + ((lane >> 3) & 1) * 8;
    uint32_t uh[4], ul[4];
    if (KIND == LINREC_DELTA) {
      uint32_t dh[4], dl[4], bh[4], bl[4];
      ldsm4(bh, im + I::th + mr);
      ldsm4(bl, im + I::tl + mr);
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        float x = v[q >> 1][(q & 1) * 2] - R[q >> 1][(q & 1) * 2], y = v[q >> 1][(q & 1) * 2 + 1] - R[q >> 1][(q & 1) * 2 + 1];
        dh[q] = split_head(x, y);
        dl[q] = pack_bf162(x, y);
      }
      float U[2][4] = {}, U2[2][4] = {};
      mma(U[0], dh, bh[0], bh[1]); mma(U[1], dh, bh[2], bh[3]);
      mma(U2[0], dl, bh[0], bh[1]); mma(U2[1], dl, bh[2], bh[3]);
      mma(U[0], dh, bl[0], bl[1]); mma(U[1], dh, bl[2], bl[3]);
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        float x = U[q >> 1][(q & 1) * 2] + U2[q >> 1][(q & 1) * 2], y = U[q >> 1][(q & 1) * 2 + 1] + U2[q >> 1][(q & 1) * 2 + 1];
        uh[q] = split_head(x, y);
        ul[q] = pack_bf162(x, y);
      }
    } else {
#pragma unroll
      for (int q = 0; q < 4; ++q) {                              // values are bf16: no remainder
        uh[q] = GAT ? vf[q] : pack_bf162(v[q >> 1][(q & 1) * 2], v[q >> 1][(q & 1) * 2 + 1]);
        ul[q] = 0;
      }
    }
    // S^T <- G S^T + U^T K^
#pragma unroll
    for (int k = 0; k < NT / 2; ++k) {
      uint32_t bh[4], bl[4];
      const int off = (lane & 15) * P + kc + k * 16 + (lane >> 4) * 8;
      ldsm4t(bh, im + I::kh + off);
      ldsm4t(bl, im + I::kl + off);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float2 gg = *reinterpret_cast<const float2*>(G + (2 * k + i) * 8 + t4 * 2);
        float* s = S[2 * k + i];
        s[0] *= gg.x; s[1] *= gg.y; s[2] *= gg.x; s[3] *= gg.y;
        mma(s, uh, bh[2 * i], bh[2 * i + 1]);
        mma(s, uh, bl[2 * i], bl[2 * i + 1]);
        if (KIND == LINREC_DELTA) mma(s, ul, bh[2 * i], bh[2 * i + 1]);
      }
    }
    // read-outs of this half's eight tokens
    {
      uint32_t bh[4], bl[4];
      ldsm4(bh, im + I::bh + mr);
      ldsm4(bl, im + I::bl + mr);
      const uint32_t b0 = half ? bh[2] : bh[0], b1 = half ? bh[3] : bh[1], l0 = half ? bl[2] : bl[0], l1 = half ? bl[3] : bl[1];
      float O[4], O2[4] = {};
#pragma unroll
      for (int e = 0; e < 4; ++e) O[e] = half ? R[NR - 1][e] : R[NR - 2][e];
      mma(O, uh, b0, b1);
      mma(O2, uh, l0, l1);
      if (KIND == LINREC_DELTA) mma(O2, ul, b0, b1);
      const int left = n - (first + ch) * C - half * 8 - t4 * 2;
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if ((e & 1) < left && (e >> 1 ? okb : oka)) op[(e & 1) * ostep + (e >> 1) * 8] = O[e] + O2[e];
      op += C * ostep;
    }
  }
  if (!last) return;
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = kc + i * 8 + t4 * 2 + (e & 1), v = e >> 1 ? vb : va;
      if (c < a.dk && v < vlim) Sg[(int64_t)c * sstride + v] = S[i][e];
    }
}

// ---- finish -------------------------------------------------------------------------------------
constexpr int kVMax = 16;
template <int KIND>
__global__ void __launch_bounds__(128) chunk_finish_kernel(const ChunkArgs ca, int rows) {
  const LinrecArgs& a = ca.r;
  const int64_t w = (int64_t)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  griddep_launch();
  griddep_wait();
  if (w >= (int64_t)rows * a.H) return;
  const int64_t row = w / a.H;
  const int h = (int)(w % a.H);
  const float* o = ca.o + row * ca.ldo_ + (int64_t)h * a.dv;
  const bf16* og = KIND == LINREC_GATED ? nullptr : reinterpret_cast<const bf16*>(a.og) + row * a.ldo + (int64_t)h * a.dv;
  const float* nw = a.norm_w + (KIND == LINREC_MLSTM ? (int64_t)h * a.dv : 0);
  float inv = 1.f;
  if (KIND == LINREC_MLSTM) inv = 1.f / (fmaxf(fabsf(ca.nq[row * a.H + h]), expf(-ca.gm[row * a.H + h])) + 1e-6f);
  float4 x[kVMax / 4];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < kVMax / 4; ++i) {
    const int c = 4 * (lane + 32 * i);
    x[i] = c < a.dv ? *reinterpret_cast<const float4*>(o + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    x[i].x *= inv; x[i].y *= inv; x[i].z *= inv; x[i].w *= inv;
    ss = fmaf(x[i].x, x[i].x, fmaf(x[i].y, x[i].y, fmaf(x[i].z, x[i].z, fmaf(x[i].w, x[i].w, ss))));
  }
  const float r = 1.f / sqrtf(warp_sum(ss) / (float)a.dv + a.eps);
  bf16* out = reinterpret_cast<bf16*>(a.act) + row * a.lda + (int64_t)h * a.dv;
#pragma unroll
  for (int i = 0; i < kVMax / 4; ++i) {
    const int c = 4 * (lane + 32 * i);
    if (c < a.dv) {
      const float4 w4 = *reinterpret_cast<const float4*>(nw + c);
      if (KIND == LINREC_GATED) {
        act_store4(out + c, make_float4(x[i].x * r * w4.x, x[i].y * r * w4.y, x[i].z * r * w4.z, x[i].w * r * w4.w));
        continue;
      }
      const float4 gt = act_load4(og + c);
      act_store4(out + c, make_float4(x[i].x * r * w4.x * sigmoid_s(gt.x), x[i].y * r * w4.y * sigmoid_s(gt.y),
                                      x[i].z * r * w4.z * sigmoid_s(gt.z), x[i].w * r * w4.w * sigmoid_s(gt.w)));
    }
  }
}

constexpr int kMinBlock = 8;           // chunks of a block of the gated scan, at least
template <int KIND, int DK>
int run_chunks(const ChunkArgs& ca, int max_rows, int rows, cudaStream_t st) {
  using I = Image<KIND, DK>;
  const LinrecArgs& a = ca.r;
  const int chunks = (max_rows + C - 1) / C;
  cudaError_t e;
  if (KIND == LINREC_DELTA) {
    const size_t smem = sizeof(float) * 3 * C * (DK + 4);
    const dim3 grid((unsigned)chunks, (unsigned)a.H, (unsigned)ca.segs);
#define CB_PREP(N)                                                                                                         \
  {                                                                                                                        \
    auto kern = chunk_prep_delta_kernel<DK, N>;                                                                            \
    if (smem > 40 * 1024 && (e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)) != cudaSuccess) \
      return (int)e;                                                                                                       \
    e = cb_launch(kern, grid, dim3(kPT), smem, st, ca);                                                                    \
  }
    if (a.taps == 4) CB_PREP(4) else CB_PREP(0)
#undef CB_PREP
    if (e != cudaSuccess) return (int)e;
  } else if (KIND == LINREC_GATED) {
    const size_t smem = sizeof(float) * 3 * C * (DK + 4);
    auto kern = chunk_prep_gated_kernel<DK>;
    if (smem > 40 * 1024 && (e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)) != cudaSuccess) return (int)e;
    e = cb_launch(kern, dim3((unsigned)chunks, (unsigned)a.H, (unsigned)ca.segs), dim3(kPT), smem, st, ca);
    if (e != cudaSuccess) return (int)e;
  } else {
    e = cb_launch(chunk_gates_mlstm_kernel, dim3((unsigned)a.H, (unsigned)ca.segs), dim3(kGT), 0, st, ca);
    if (e != cudaSuccess) return (int)e;
    const size_t smem = sizeof(bf16) * 2 * C * I::P;
    e = cb_launch(chunk_prep_mlstm_kernel<DK>, dim3((unsigned)chunks, (unsigned)a.H, (unsigned)ca.segs), dim3(64), smem, st, ca);
    if (e != cudaSuccess) return (int)e;
  }
  constexpr int STAGES = KIND == LINREC_GATED ? 3 : (DK <= 128 ? 4 : 3);
  auto scan = chunk_scan_kernel<KIND, DK, STAGES>;
  const size_t smem = STAGES * (I::bytes + C * (KIND == LINREC_DELTA ? 36 * 4 : kVP * 2));
  e = cudaFuncSetAttribute(scan, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  const int slices = (a.dv + 31) / 32 + (KIND == LINREC_MLSTM ? 1 : 0);
  int blocks = 1;
  ChunkArgs cb = ca;
  if constexpr (KIND == LINREC_GATED) {
    const int resident = 148 * (DK <= 128 ? 3 : 1), base = slices * a.H * ca.segs;
    const int want = resident / base < chunks / kMinBlock ? resident / base : chunks / kMinBlock;
    if (want > 1) {
      cb.per = (chunks + want - 1) / want;
      blocks = (chunks + cb.per - 1) / cb.per;
      constexpr int SS = 4;
      auto states = chunk_states_kernel<DK, SS>;
      const size_t sm = SS * (2 * C * I::P * 2 + DK * 4 + C * kVP * 2);
      e = cudaFuncSetAttribute(states, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm);
      if (e != cudaSuccess) return (int)e;
      if (blocks > 1) e = cb_launch(states, dim3((unsigned)(slices * (blocks - 1)), (unsigned)a.H, (unsigned)ca.segs), dim3(kST), sm, st, cb, slices);
      if (e != cudaSuccess) return (int)e;
    }
  }
  e = cb_launch(scan, dim3((unsigned)(slices * blocks), (unsigned)a.H, (unsigned)ca.segs), dim3(kST), smem, st, cb, slices);
  if (e != cudaSuccess) return (int)e;
  return (int)cb_launch(chunk_finish_kernel<KIND>, dim3((unsigned)(((int64_t)rows * a.H + 3) / 4)), dim3(128), 0, st, ca, rows);
}

int padded_dk(int64_t dk) { return dk <= 32 ? 32 : (dk <= 64 ? 64 : (dk <= 128 ? 128 : 256)); }
int64_t image_bytes(int64_t kind, int64_t dk) {
  const int d = padded_dk(dk);
  if (kind == LINREC_DELTA)
    return d == 32 ? Image<LINREC_DELTA, 32>::bytes : (d == 64 ? Image<LINREC_DELTA, 64>::bytes : (d == 128 ? Image<LINREC_DELTA, 128>::bytes : Image<LINREC_DELTA, 256>::bytes));
  return d == 32 ? Image<LINREC_MLSTM, 32>::bytes : (d == 64 ? Image<LINREC_MLSTM, 64>::bytes : (d == 128 ? Image<LINREC_MLSTM, 128>::bytes : Image<LINREC_MLSTM, 256>::bytes));
}
int64_t al(int64_t x) { return (x + 255) & ~(int64_t)255; }
// entries of the gated scan's blocks, whatever their size
int64_t part_entries(int64_t rows, int64_t segs) { return rows / (C * kMinBlock) + 2 * segs + 2; }
int64_t part_bytes(int64_t kind, int64_t rows, int64_t segs, int64_t H, int64_t dk, int64_t dv) {
  return kind == LINREC_GATED ? al(part_entries(rows, segs) * H * ((dv + 31) / 32) * 32 * padded_dk(dk) * 4) : 0;
}
int64_t keep_bytes(int64_t kind, int64_t rows, int64_t segs, int64_t H, int64_t dk) {
  return kind == LINREC_GATED ? al(part_entries(rows, segs) * H * padded_dk(dk) * 4) : 0;
}

}  // namespace

// Whether the chunked kernels take a head of this size (16-byte rows, state columns in registers).
CB_EXPORT int cb_linrec_chunk_ok(int64_t dk, int64_t dv) { return dk % 8 == 0 && dv % 8 == 0 && dk <= 256 && dv <= 32 * kVMax; }

// Scratch bytes of a call over `rows` rows in `segs` segments.
CB_EXPORT int64_t cb_linrec_chunk_scratch(int64_t kind, int64_t rows, int64_t segs, int64_t H, int64_t dk, int64_t dv) {
  const int64_t blocks = rows / C + segs + 2;
  return al(blocks * H * image_bytes(kind, dk)) + 2 * al(rows * H * dv * 4) + 5 * al(rows * H * 4) +
         part_bytes(kind, rows, segs, H, dk, dv) + keep_bytes(kind, rows, segs, H, dk);
}

// `segs` segments of the recurrence `kind`, rows [0, rows) of the projection; bf16 projection rows and activations,
// decay and output-gate pre-activations given.  The convolution ring is only read (cb_linrec_ring afterwards).
CB_EXPORT int cb_linrec_chunk(const void* args, int64_t kind, int64_t segs, int64_t max_rows, int64_t rows, void* scratch,
                              int64_t scratch_bytes, void* stream) {
  if (!args || !scratch || segs < 1 || segs > 65535 || rows < 1 || max_rows < 1) return CB_ERR_ARG;
  ChunkArgs ca;
  ca.r = *(const LinrecArgs*)args;
  const LinrecArgs& a = ca.r;
  if (!a.proj || !a.gates || !a.act || (!a.og && kind != LINREC_GATED) || !a.seg_row || !a.seg_pos || !a.seg_slot || !a.S || a.H < 1 || a.G < 1 || a.H % a.G)
    return CB_ERR_ARG;
  if (!cb_linrec_chunk_ok(a.dk, a.dv) || a.ldp % 8 || a.k_col % 8 || a.v_col % 8 || a.lda % 4 || a.ldo % 4) return CB_ERR_SHAPE;
  if (kind == LINREC_DELTA && (!a.dec || !a.ring || a.taps < 1 || a.taps > a.ring_mask + 1)) return CB_ERR_ARG;
  if (kind == LINREC_MLSTM && (!a.n || !a.m || !(a.cap > 0.f))) return CB_ERR_ARG;
  if (kind == LINREC_GATED && (!a.gate_b || !a.lower || !a.norm_w || a.G != a.H)) return CB_ERR_ARG;
  if (scratch_bytes < cb_linrec_chunk_scratch(kind, rows, segs, a.H, a.dk, a.dv)) return CB_ERR_ARG;
  unsigned char* p = (unsigned char*)scratch;
  ca.image = p; p += al((rows / C + segs + 2) * a.H * image_bytes(kind, a.dk));
  ca.v = (float*)p; p += al(rows * a.H * (int64_t)a.dv * 4);
  ca.o = (float*)p; p += al(rows * a.H * (int64_t)a.dv * 4);
  ca.ldo_ = (int64_t)a.H * a.dv;
  float** g[5] = {&ca.gi, &ca.gf, &ca.gm, &ca.gb, &ca.nq};
  for (int i = 0; i < 5; ++i) { *g[i] = (float*)p; p += al(rows * a.H * 4); }
  ca.part = (float4*)p; p += part_bytes(kind, rows, segs, a.H, a.dk, a.dv);
  ca.keep = (float*)p;
  ca.per = 0;
  ca.segs = (int)segs;
  cudaStream_t st = (cudaStream_t)stream;
  const int d = padded_dk(a.dk);
#define CB_RUN(K)                                                        \
  switch (d) {                                                           \
    case 32: return run_chunks<K, 32>(ca, (int)max_rows, (int)rows, st); \
    case 64: return run_chunks<K, 64>(ca, (int)max_rows, (int)rows, st); \
    case 128: return run_chunks<K, 128>(ca, (int)max_rows, (int)rows, st); \
    default: return run_chunks<K, 256>(ca, (int)max_rows, (int)rows, st); \
  }
  if (kind == LINREC_DELTA) { CB_RUN(LINREC_DELTA) }
  if (kind == LINREC_MLSTM) { CB_RUN(LINREC_MLSTM) }
  if (kind == LINREC_GATED) { CB_RUN(LINREC_GATED) }
#undef CB_RUN
  return CB_ERR_ARG;
}
