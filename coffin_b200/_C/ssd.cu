// Selective state spaces with a scalar decay per head and token (Mamba-2) over prompts, and the gated norm behind them.
//
//     S_t = exp(A dt_t) S_(t-1) + dt_t B_t x_t^T,    y_t = S_t^T C_t + D x_t        (A = -exp(A_log) per head)
//
// B and C are shared by the heads of a group, so nothing per head is prepared: `conv` leaves the convolved rows
// [C | B | x] once (bf16, what the tensor cores read) with the per-head step sizes and the decays cumulated within chunks of
// 64 tokens; `scan` (one CTA per head and 32 value columns) walks the chunks,
//
//     y = ((C B^T) * M) x + diag(e^a) C S_0 + D x,   M_ts = e^(a_t - a_s) dt_s  (s <= t)
//     S <- e^(a_Q) S_0 + (diag(dt e^(a_Q - a)) B)^T x
//
// a is the cumulated log decay, only differences that are <= 0 are exponentiated.  The 32-bit factors (the state, the
// decayed scores, the weighted values) enter the products as bf16 head + remainder, sums and state are fp32.
// `step` goes token by token (decoding, 32-bit mode, odd sizes): one CTA per sequence and up to four heads of a group, which
// convolves their channels and streams their state through registers once per token.
#include "linrec.cuh"

namespace {

constexpr int Q = 64, VS = 32, VP = VS + 8, kST = 256;
constexpr float kLog2e = 1.4426950408889634f;

struct SsdArgs {
  LinrecArgs r;
  bf16* xc;                  // convolved rows [rows, conv_w columns of the projection: C | B | x]
  float* a; float* dt;       // [rows, H]: cumulated log2 decay within the chunk, step size
  float* y;                  // [rows, ldy_]
};

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void cp16(void* s, const void* g, bool ok) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(s);
  const int n = ok ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(a), "l"(g), "r"(n) : "memory");
}
__device__ __forceinline__ void cp4(void* s, const void* g, bool ok) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(s);
  const int n = ok ? 4 : 0;
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(a), "l"(g), "r"(n) : "memory");
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
__device__ __forceinline__ float2 unpack2(uint32_t v) { return make_float2(__uint_as_float(v << 16), __uint_as_float(v & 0xffff0000u)); }

// ---- conv --------------------------------------------------------------------------------------
// 16 tokens x 512 channels (two per thread) per CTA; the last blocks of x do the decays: 64 tokens x 256 heads each.
constexpr int kCT = 256, CC = 16;
template <int TAPS>
__global__ void __launch_bounds__(kCT) ssd_conv_kernel(const SsdArgs s, int cblocks) {
  const LinrecArgs& a = s.r;
  const int tid = threadIdx.x, seg = blockIdx.z;
  griddep_launch();
  griddep_wait();
  const int row0 = a.seg_row[seg], n = a.seg_row[seg + 1] - row0, slot = a.seg_slot[seg], pos0 = a.seg_pos[seg];
  if (slot < 0) return;
  if ((int)blockIdx.x >= cblocks) {
    const int h = ((int)blockIdx.x - cblocks) * kCT + tid, c0 = blockIdx.y * Q;
    if (h >= a.H) return;
    const float ea = -expf(a.A_log[h]) * kLog2e, db = a.dt_bias[h];
    float cum = 0.f;
    for (int t0 = c0; t0 < min(n, c0 + Q); t0 += 8) {
      float g[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) g[i] = t0 + i < n ? a.gates[(int64_t)(row0 + t0 + i) * a.ldg + h] : 0.f;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        if (t0 + i >= n) break;
        const float dt = softplus_s(g[i] + db);
        cum = fmaf(ea, dt, cum);
        const int64_t e = (int64_t)(row0 + t0 + i) * a.H + h;
        s.a[e] = cum;
        s.dt[e] = dt;
      }
    }
    return;
  }
  const int64_t ch = ((int64_t)blockIdx.x * kCT + tid) * 2;
  if (ch >= a.ring_w) return;
  const bf16* proj = reinterpret_cast<const bf16*>(a.proj);
  const bf16* ring = reinterpret_cast<const bf16*>(a.ring) + (int64_t)slot * (a.ring_mask + 1) * a.ring_w;
  auto raw = [&](int rel) -> float2 {                            // token of the segment, possibly before it
    if (rel >= 0) return unpack2(*reinterpret_cast<const uint32_t*>(proj + (int64_t)(row0 + rel) * a.ldp + ch));
    const int p = pos0 + rel;
    if (p < 0) return make_float2(0.f, 0.f);
    return unpack2(*reinterpret_cast<const uint32_t*>(ring + (int64_t)(p & a.ring_mask) * a.ring_w + ch));
  };
  const float bx = a.conv_b ? a.conv_b[ch] : 0.f, by = a.conv_b ? a.conv_b[ch + 1] : 0.f;
  for (int c0 = blockIdx.y * Q; c0 < min(n, (int)(blockIdx.y + 1) * Q); c0 += CC) {
    const int m = min(CC, n - c0);
    auto emit = [&](int t, float x, float y) {
      if (t < m) *reinterpret_cast<uint32_t*>(s.xc + (int64_t)(row0 + c0 + t) * a.ring_w + ch) = pack_bf162(silu_s(x), silu_s(y));
    };
    if (TAPS > 0) {
      constexpr int N = TAPS > 0 ? TAPS : 1;
      float wx[N], wy[N];
      float2 x[CC + N - 1];
#pragma unroll
      for (int j = 0; j < N; ++j) { wx[j] = a.conv_w[ch * N + j]; wy[j] = a.conv_w[(ch + 1) * N + j]; }
#pragma unroll
      for (int i = 0; i < CC + N - 1; ++i) x[i] = i - (N - 1) < m ? raw(c0 + i - (N - 1)) : make_float2(0.f, 0.f);
#pragma unroll
      for (int t = 0; t < CC; ++t) {
        float ax = bx, ay = by;
#pragma unroll
        for (int j = 0; j < N; ++j) { ax = fmaf(wx[j], x[t + j].x, ax); ay = fmaf(wy[j], x[t + j].y, ay); }
        emit(t, ax, ay);
      }
    } else {
      for (int t = 0; t < m; ++t) {
        float ax = bx, ay = by;
        for (int j = 0; j < a.taps; ++j) {
          const float2 x = raw(c0 + t - (a.taps - 1) + j);
          ax = fmaf(a.conv_w[ch * a.taps + j], x.x, ax);
          ay = fmaf(a.conv_w[(ch + 1) * a.taps + j], x.y, ay);
        }
        emit(t, ax, ay);
      }
    }
  }
}

// ---- step --------------------------------------------------------------------------------------
constexpr int kNT = 256, kHPC = 4, kRB = 8;
// V: state columns per thread (4: dv is a multiple of 4)
template <typename TP, typename TA, int V>
__global__ void __launch_bounds__(kNT, 2) ssd_step_kernel(const SsdArgs s, int hpc) {
  const LinrecArgs& a = s.r;
  extern __shared__ __align__(16) float sm[];
  const int tid = threadIdx.x, seg = blockIdx.y, dk = a.dk, dv = a.dv;
  const int hpg = a.H / a.G, cpg = (hpg + hpc - 1) / hpc, g = blockIdx.x / cpg, h0 = g * hpg + (blockIdx.x % cpg) * hpc;
  const int nh = min(hpc, (g + 1) * hpg - h0);
  const int CQ = min(dv / V, kNT), RG = kNT / CQ, q = tid % CQ, rg = tid / CQ;         // column unit and row group of this thread
  float* sc = sm;                                      // [dk]
  float* sb = sc + dk;                                 // [dk]
  float* sx = sb + dk;                                 // [hpc][dv]
  float* part = sx + hpc * dv;                         // [hpc][RG][dv]
  __shared__ float dt_s[kHPC], de_s[kHPC];
  const int nch = 2 * dk + nh * dv;
  auto channel = [&](int e) {                          // C, B, then the values of the heads
    return e < dk ? (int64_t)g * dk + e : (e < 2 * dk ? a.k_col + (int64_t)g * dk + e - dk : a.v_col + (int64_t)h0 * dv + e - 2 * dk);
  };
  const bool taps4 = a.taps == 4;
  float4 pw[2];
  float pb[2];
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    const bool ok = tid + u * kNT < nch;
    pw[u] = ok && taps4 ? *reinterpret_cast<const float4*>(a.conv_w + channel(tid + u * kNT) * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    pb[u] = ok && a.conv_b ? a.conv_b[channel(tid + u * kNT)] : 0.f;
  }
  const float p_dt = tid < nh ? a.dt_bias[h0 + tid] : 0.f, p_ea = tid < nh ? expf(a.A_log[h0 + tid]) : 0.f;
  griddep_launch();
  griddep_wait();
  const int row0 = a.seg_row ? a.seg_row[seg] : seg;
  const int nrow = a.seg_row ? a.seg_row[seg + 1] - row0 : 1;
  const int slot = a.seg_slot[seg], pos0 = a.seg_pos[seg];
  if (slot < 0 || nrow < 1 || pos0 < 0) return;
  float* Sg = a.S + ((int64_t)slot * a.H + h0) * dk * dv;
  const TA* ring = reinterpret_cast<const TA*>(a.ring) + (int64_t)slot * (a.ring_mask + 1) * a.ring_w;
  const TP* prow0 = reinterpret_cast<const TP*>(a.proj) + (int64_t)row0 * a.ldp;
  const int per = (dk + RG - 1) / RG, nb = (per + kRB - 1) / kRB, items = nh * nb;      // blocks of kRB rows per head and thread
  for (int cb = 0; cb * CQ * V < dv; ++cb) {           // more than kNT column units: one round after the other
    const int c = (cb * CQ + q) * V;
    const bool act = rg < RG && c < dv;
    auto load = [&](int it, float (*f)[V]) {
      const float* p = Sg + (int64_t)(it / nb) * dk * dv + c;
#pragma unroll
      for (int i = 0; i < kRB; ++i) {
        const int r = rg + ((it % nb) * kRB + i) * RG;
        if (V == 4) {
          const float4 x = act && r < dk ? *reinterpret_cast<const float4*>(p + (int64_t)r * dv) : make_float4(0.f, 0.f, 0.f, 0.f);
          f[i][0] = x.x; f[i][1 % V] = x.y; f[i][2 % V] = x.z; f[i][3 % V] = x.w;
        } else {
          f[i][0] = act && r < dk ? p[(int64_t)r * dv] : 0.f;
        }
      }
    };
    for (int t = 0; t < nrow; ++t) {
      const int64_t row = row0 + t;
      float nx[kRB][V];
      load(0, nx);                                     // in flight during the convolution
      const float gate = tid < nh ? a.gates[row * a.ldg + h0 + tid] : 0.f;
      auto tap = [&](int64_t ch, int j) {
        const int src = t - (a.taps - 1) + j, p = pos0 + src;
        float x = 0.f;
        if (src >= 0) x = act_round<TA>(act_load(prow0 + (int64_t)src * a.ldp + ch));
        else if (p >= 0) x = act_load(ring + (int64_t)(p & a.ring_mask) * a.ring_w + ch);
        return x;
      };
      if (taps4) {
        float x[2][4];
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
          for (int j = 0; j < 4; ++j) x[u][j] = tid + u * kNT < nch ? tap(channel(tid + u * kNT), j) : 0.f;
#pragma unroll
        for (int u = 0; u < 2; ++u)
          if (tid + u * kNT < nch)                     // sc, sb and sx are adjacent
            sm[tid + u * kNT] = silu_s(fmaf(pw[u].w, x[u][3], fmaf(pw[u].z, x[u][2], fmaf(pw[u].y, x[u][1], fmaf(pw[u].x, x[u][0], pb[u])))));
      }
#pragma unroll 1
      for (int e = tid + (taps4 ? 2 * kNT : 0); e < nch; e += kNT) {
        const int64_t ch = channel(e);
        float acc = a.conv_b ? a.conv_b[ch] : 0.f;
#pragma unroll 1
        for (int j = 0; j < a.taps; ++j) acc = fmaf(a.conv_w[ch * a.taps + j], tap(ch, j), acc);
        sm[e] = silu_s(acc);
      }
      if (tid < nh) {
        const float dt = softplus_s(gate + p_dt);
        dt_s[tid] = dt;
        de_s[tid] = __expf(-p_ea * dt);
      }
      __syncthreads();
      float acc[V];
#pragma unroll 1
      for (int it = 0; it < items; ++it) {
        float cur[kRB][V];
#pragma unroll
        for (int i = 0; i < kRB; ++i)
#pragma unroll
          for (int v = 0; v < V; ++v) cur[i][v] = nx[i][v];
        if (it + 1 < items) load(it + 1, nx);
        const int hi = it / nb, b = it % nb;
        const float de = de_s[hi], dt = dt_s[hi];
        float xv[V];
#pragma unroll
        for (int v = 0; v < V; ++v) {
          xv[v] = act ? dt * sx[hi * dv + c + v] : 0.f;
          if (b == 0) acc[v] = 0.f;
        }
        float* p = Sg + (int64_t)hi * dk * dv + c;
#pragma unroll
        for (int i = 0; i < kRB; ++i) {
          const int r = rg + (b * kRB + i) * RG;
          if (act && r < dk) {
            const float k = sb[r], cc = sc[r];
#pragma unroll
            for (int v = 0; v < V; ++v) {
              cur[i][v] = fmaf(de, cur[i][v], k * xv[v]);
              acc[v] = fmaf(cc, cur[i][v], acc[v]);
            }
            if (V == 4) *reinterpret_cast<float4*>(p + (int64_t)r * dv) = make_float4(cur[i][0], cur[i][1 % V], cur[i][2 % V], cur[i][3 % V]);
            else p[(int64_t)r * dv] = cur[i][0];
          }
        }
        if (act && b == nb - 1)
#pragma unroll
          for (int v = 0; v < V; ++v) part[(hi * RG + rg) * dv + c + v] = acc[v];
      }
      __syncthreads();
      for (int e = tid; e < nh * CQ * V; e += kNT) {
        const int hi = e / (CQ * V), col = cb * CQ * V + e % (CQ * V);
        if (col >= dv) continue;
        float y = a.D[h0 + hi] * sx[hi * dv + col];
        for (int r = 0; r < RG; ++r) y += part[(hi * RG + r) * dv + col];
        s.y[row * a.lda + (int64_t)(h0 + hi) * dv + col] = y;
      }
      __syncthreads();
    }
  }
  if (nrow == 1) {
    // one token: its raw rows enter the ring here (no reader of this step looks at that entry); longer segments
    // leave it to cb_linrec_ring, which runs after every reader
    TA* w = reinterpret_cast<TA*>(a.ring) + ((int64_t)slot * (a.ring_mask + 1) + (pos0 & a.ring_mask)) * a.ring_w;
    for (int e = tid + (h0 == g * hpg ? 0 : 2 * dk); e < nch; e += kNT) {
      const int64_t ch = channel(e);
      act_store(w + ch, act_load(prow0 + ch));
    }
  }
}

template <typename TP, typename TA>
int launch_step(const SsdArgs& s, int segs, cudaStream_t st) {
  const LinrecArgs& a = s.r;
  const int hpg = a.H / a.G;
  int hpc = kHPC;
  while (hpc > 1 && (int64_t)a.G * ((hpg + hpc - 1) / hpc) * segs < 200) hpc >>= 1;      // few sequences: one head per CTA
  const bool v4 = a.dv % 4 == 0;
  const int V = v4 ? 4 : 1, CQ = a.dv / V < kNT ? a.dv / V : kNT, RG = kNT / CQ;
  const size_t smem = sizeof(float) * ((size_t)2 * a.dk + (size_t)hpc * a.dv * (1 + RG));
  if (smem > 200 * 1024) return CB_ERR_SHAPE;
  auto kern = v4 ? ssd_step_kernel<TP, TA, 4> : ssd_step_kernel<TP, TA, 1>;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return (int)cb_launch(kern, dim3((unsigned)(a.G * ((hpg + hpc - 1) / hpc)), (unsigned)segs), dim3(kNT), smem, st, s, hpc);
}

// ---- scan --------------------------------------------------------------------------------------
template <int NP>
struct Plan {
  static constexpr int P = NP + 8, MTN = NP / 16;
  static constexpr int MPW = MTN > 8 ? MTN / 8 : 1;              // state row tiles (16 channels) per warp
  static constexpr int SH = MTN < 8 ? 8 / MTN : 1;               // warps that share a row tile
  static constexpr int NTW = 4 / SH;                             // column tiles (8) per warp
  static constexpr int TILE = 2 * Q * P + Q * VP;                // one stage: C, B, x (bf16)
  static constexpr bool XOWN = 16 * P * 2 < 2048;                // sixteen C rows do not hold a pair's exchange
  static constexpr size_t bytes = sizeof(bf16) * (2 * TILE + 2 * Q * VP + 2 * NP * VP) + sizeof(float) * 4 * Q + (XOWN ? 4 * 2048 : 0);
};

// Read-outs of token rows 16 RG .. 16 RG + 15 by two warps: each takes half of the earlier tokens (scores, decays, values)
// and half of the old state's channels over all columns; the partial sums meet in `xch` (the pair's own rows of the C tile,
// which nobody else reads, where those are large enough), and each warp finishes 16 columns.
template <int NP, int RG, int HALF>
__device__ __forceinline__ void read_out(const bf16* ct, float4* xch, const bf16* bt, const bf16* xt, const bf16* st, const float* av, const float* dtv,
                                         int lane, int m, int nv, float Dh, float* y, int64_t ldy) {
  constexpr int P = NP + 8, J0 = HALF ? (RG + 2) / 2 : 0, J1 = HALF ? RG + 1 : (RG + 2) / 2, NJ = J1 - J0, KH = NP / 32;
  const int g4 = lane >> 2, t4 = lane & 3;
  float G[NJ > 0 ? 2 * NJ : 1][4], Y[4][4];
#pragma unroll
  for (int i = 0; i < 2 * NJ; ++i) G[i][0] = G[i][1] = G[i][2] = G[i][3] = 0.f;
#pragma unroll
  for (int i = 0; i < 4; ++i) Y[i][0] = Y[i][1] = Y[i][2] = Y[i][3] = 0.f;
  const bf16* cr = ct + (RG * 16 + (lane & 15)) * P + (lane >> 4) * 8;
  const bf16* sr = st + (lane & 15) * VP + (lane >> 4) * 8;
  const bf16* br = bt + (J0 * 16 + (lane & 7) + ((lane >> 4) << 3)) * P + ((lane >> 3) & 1) * 8;
#pragma unroll
  for (int k = 0; k < NP / 16; ++k) {
    const bool mine = k / KH == HALF;                            // compile time
    if (NJ == 0 && !mine) continue;
    uint32_t ca[4];
    ldsm4(ca, cr + k * 16);
    if (mine) {
      uint32_t s0[4], s1[4];
      ldsm4t(s0, sr + k * 16 * VP);
      ldsm4t(s1, sr + k * 16 * VP + 16);
      mma(Y[0], ca, s0[0], s0[1]); mma(Y[1], ca, s0[2], s0[3]);
      mma(Y[2], ca, s1[0], s1[1]); mma(Y[3], ca, s1[2], s1[3]);
      ldsm4t(s0, sr + (NP + k * 16) * VP);
      ldsm4t(s1, sr + (NP + k * 16) * VP + 16);
      mma(Y[0], ca, s0[0], s0[1]); mma(Y[1], ca, s0[2], s0[3]);
      mma(Y[2], ca, s1[0], s1[1]); mma(Y[3], ca, s1[2], s1[3]);
    }
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      uint32_t b[4];
      ldsm4(b, br + j * 16 * P + k * 16);
      mma(G[2 * j], ca, b[0], b[1]);
      mma(G[2 * j + 1], ca, b[2], b[3]);
    }
  }
  const int tl = RG * 16 + g4, th = tl + 8;
  const float al = av[tl], ah = av[th], el = ex2(al), eh = ex2(ah);
#pragma unroll
  for (int i = 0; i < 4; ++i) { Y[i][0] *= el; Y[i][1] *= el; Y[i][2] *= eh; Y[i][3] *= eh; }
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    uint32_t mh[4], ml[4], b0[4], b1[4];
    ldsm4t(b0, xt + ((J0 + j) * 16 + (lane & 15)) * VP + (lane >> 4) * 8);
    ldsm4t(b1, xt + ((J0 + j) * 16 + (lane & 15)) * VP + 16 + (lane >> 4) * 8);
#pragma unroll
    for (int p = 0; p < 2; ++p) {                                // tokens u, u + 1 of rows lo, then hi
      const int u = (J0 + j) * 16 + p * 8 + t4 * 2;
      const float2 au = *reinterpret_cast<const float2*>(av + u), du = *reinterpret_cast<const float2*>(dtv + u);
      const float* gg = G[2 * j + p];
      float x = gg[0] * (du.x * ex2(fminf(al - au.x, 0.f))), z = gg[1] * (du.y * ex2(fminf(al - au.y, 0.f)));
      float v = gg[2] * (du.x * ex2(fminf(ah - au.x, 0.f))), w = gg[3] * (du.y * ex2(fminf(ah - au.y, 0.f)));
      if (J0 + j == RG) {
        if (u > tl) x = 0.f;
        if (u + 1 > tl) z = 0.f;
        if (u > th) v = 0.f;
        if (u + 1 > th) w = 0.f;
      }
      mh[2 * p] = split_head(x, z); ml[2 * p] = pack_bf162(x, z);          // a0 / a2: row lo; a1 / a3: row hi
      mh[2 * p + 1] = split_head(v, w); ml[2 * p + 1] = pack_bf162(v, w);
    }
    mma(Y[0], mh, b0[0], b0[1]); mma(Y[1], mh, b0[2], b0[3]);
    mma(Y[2], mh, b1[0], b1[1]); mma(Y[3], mh, b1[2], b1[3]);
    mma(Y[0], ml, b0[0], b0[1]); mma(Y[1], ml, b0[2], b0[3]);
    mma(Y[2], ml, b1[0], b1[1]); mma(Y[3], ml, b1[2], b1[3]);
  }
  asm volatile("bar.sync %0, 64;" ::"r"(1 + RG) : "memory");     // both warps are done with the C rows
#pragma unroll
  for (int i = 0; i < 2; ++i) {                                  // [half that wrote][2][lane]
    const float* o = Y[(HALF ? 0 : 2) + i];
    xch[(HALF * 2 + i) * 32 + lane] = make_float4(o[0], o[1], o[2], o[3]);
  }
  asm volatile("bar.sync %0, 64;" ::"r"(1 + RG) : "memory");
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const float4 o = xch[((1 - HALF) * 2 + i) * 32 + lane];
    const float* q = Y[HALF * 2 + i];
    const float r[4] = {q[0] + o.x, q[1] + o.y, q[2] + o.z, q[3] + o.w};
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = e ? th : tl, c = HALF * 16 + i * 8 + t4 * 2;
      if (t < m && c < nv) {
        const float2 x = unpack2(*reinterpret_cast<const uint32_t*>(xt + t * VP + c));
        *reinterpret_cast<float2*>(y + t * ldy + c) = make_float2(fmaf(Dh, x.x, r[2 * e]), fmaf(Dh, x.y, r[2 * e + 1]));
      }
    }
  }
}

template <int NP>
__global__ void __launch_bounds__(kST, NP <= 128 ? 2 : 1) ssd_scan_kernel(const SsdArgs s) {
  using L = Plan<NP>;
  constexpr int P = L::P, MPW = L::MPW, NTW = L::NTW;
  const LinrecArgs& a = s.r;
  extern __shared__ __align__(16) unsigned char smem[];
  bf16* tiles = reinterpret_cast<bf16*>(smem);                   // [2][C | B | x]
  bf16* xw = tiles + 2 * L::TILE;                                // weighted values: head, remainder
  bf16* st = xw + 2 * Q * VP;                                    // state at the chunk's start: head, remainder
  float* sa = reinterpret_cast<float*>(st + 2 * NP * VP);        // [2][Q] cumulated decays, [2][Q] step sizes
  float* sdt = sa + 2 * Q;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g4 = lane >> 2, t4 = lane & 3;
  const int h = blockIdx.y, seg = blockIdx.z, v0 = blockIdx.x * VS;
  const float Dh = a.D[h];
  griddep_launch();
  griddep_wait();
  const int row0 = a.seg_row[seg], n = a.seg_row[seg + 1] - row0, slot = a.seg_slot[seg];
  if (slot < 0 || n < 1) return;
  const int chunks = (n + Q - 1) / Q, N = a.dk, nv = min(VS, a.dv - v0);
  const int64_t qb = (int64_t)(h / (a.H / a.G)) * N, xb = a.v_col + (int64_t)h * a.dv + v0;
  auto load = [&](int ch) {
    bf16* t = tiles + (ch & 1) * L::TILE;
    const int left = n - ch * Q;
    const bf16* src = s.xc + (int64_t)(row0 + ch * Q) * a.ring_w;
#pragma unroll 1
    for (int e = tid; e < Q * (NP / 8); e += kST) {
      const int r = e / (NP / 8), c = (e % (NP / 8)) * 8;
      const bool ok = r < left && c < N;
      const bf16* p = ok ? src + (int64_t)r * a.ring_w + qb + c : s.xc;
      cp16(t + r * P + c, p, ok);
      cp16(t + Q * P + r * P + c, ok ? p + a.k_col : s.xc, ok);
    }
    {
      const int r = tid / (VS / 8), c = (tid % (VS / 8)) * 8;
      const bool ok = r < left && c < nv;
      if (r < Q) cp16(t + 2 * Q * P + r * VP + c, ok ? src + (int64_t)r * a.ring_w + xb + c : s.xc, ok);
    }
    if (tid < 2 * Q) {
      const int r = tid % Q;
      const float* p = tid < Q ? s.a : s.dt;
      cp4((tid < Q ? sa : sdt) + (ch & 1) * Q + r, r < left ? p + (int64_t)(row0 + ch * Q + r) * a.H + h : p, r < left);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load(0);
  // this warp's part of the state: row tiles (warp / SH) * MPW .., column tiles (warp % SH) * NTW ..
  float S[MPW][NTW][4];
  const int rt0 = warp / L::SH * MPW, ct0 = warp % L::SH * NTW;
  float* Sg = a.S + ((int64_t)slot * a.H + h) * N * a.dv + v0;
  auto state_out = [&]() {                                       // registers -> head / remainder in shared memory
#pragma unroll
    for (int m = 0; m < MPW; ++m)
#pragma unroll
      for (int j = 0; j < NTW; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int k = (rt0 + m) * 16 + g4 + 8 * e, c = (ct0 + j) * 8 + t4 * 2;
          float x = S[m][j][2 * e], y = S[m][j][2 * e + 1];
          *reinterpret_cast<uint32_t*>(st + k * VP + c) = split_head(x, y);
          *reinterpret_cast<uint32_t*>(st + (NP + k) * VP + c) = pack_bf162(x, y);
        }
  };
#pragma unroll
  for (int m = 0; m < MPW; ++m)
#pragma unroll
    for (int j = 0; j < NTW; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int k = (rt0 + m) * 16 + g4 + 8 * (e >> 1), c = (ct0 + j) * 8 + t4 * 2 + (e & 1);
        S[m][j][e] = k < N && c < nv ? Sg[(int64_t)k * a.dv + c] : 0.f;
      }
  state_out();
  const int half = warp >> 2, rg = half ? 3 - (warp & 3) : warp & 3;      // token tile; long and short ones share a scheduler
  for (int ch = 0; ch < chunks; ++ch) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                             // tiles, decays and state of this chunk are in place
    if (ch + 1 < chunks) load(ch + 1);
    bf16* ct = tiles + (ch & 1) * L::TILE;
    const bf16* bt = ct + Q * P;
    const bf16* xt = bt + Q * P;
    const float* av = sa + (ch & 1) * Q;
    const float* dtv = sdt + (ch & 1) * Q;
    const int m = min(Q, n - ch * Q);
    const float aq = av[m - 1];
    {                                                            // weighted values: token and eight columns per thread
      const int t = tid >> 2, c = (tid & 3) * 8;
      const float w = dtv[t] * ex2(fminf(aq - av[t], 0.f));      // padding tokens: step size 0
      const uint4 v = *reinterpret_cast<const uint4*>(xt + t * VP + c);
      float f[8];
      bf16x8_to_float(v, f);
      uint32_t hd[4], rm[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        float x = f[2 * i] * w, y = f[2 * i + 1] * w;
        hd[i] = split_head(x, y);
        rm[i] = pack_bf162(x, y);
      }
      *reinterpret_cast<uint4*>(xw + t * VP + c) = make_uint4(hd[0], hd[1], hd[2], hd[3]);
      *reinterpret_cast<uint4*>(xw + Q * VP + t * VP + c) = make_uint4(rm[0], rm[1], rm[2], rm[3]);
    }
    if (rg * 16 < m) {
      float4* xch = L::XOWN ? reinterpret_cast<float4*>(sdt + 2 * Q) + rg * 128 : reinterpret_cast<float4*>(ct + rg * 16 * P);
      float* y = s.y + (int64_t)(row0 + ch * Q) * a.lda + (int64_t)h * a.dv + v0;
#define CB_READ(R)                                                                                   \
  if (rg == R) {                                                                                     \
    if (half) read_out<NP, R, 1>(ct, xch, bt, xt, st, av, dtv, lane, m, nv, Dh, y, a.lda);                \
    else read_out<NP, R, 0>(ct, xch, bt, xt, st, av, dtv, lane, m, nv, Dh, y, a.lda);                     \
  }
      CB_READ(0) CB_READ(1) CB_READ(2) CB_READ(3)
#undef CB_READ
    }
    __syncthreads();                                             // weighted values in place, the old state has been read
    const float ge = ex2(aq);
#pragma unroll
    for (int i = 0; i < MPW; ++i) {
#pragma unroll
      for (int j = 0; j < NTW; ++j) { S[i][j][0] *= ge; S[i][j][1] *= ge; S[i][j][2] *= ge; S[i][j][3] *= ge; }
#pragma unroll
      for (int k = 0; k < Q / 16; ++k) {                         // padding tokens weigh nothing
        uint32_t ba[4];
        ldsm4t(ba, bt + (k * 16 + (lane & 7) + ((lane >> 4) << 3)) * P + (rt0 + i) * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int rem = 0; rem < 2; ++rem) {
          const bf16* w = xw + rem * Q * VP + (k * 16 + (lane & 15)) * VP;
          if (NTW >= 2) {
#pragma unroll
            for (int j = 0; j < NTW / 2; ++j) {
              uint32_t b[4];
              ldsm4t(b, w + (ct0 + 2 * j) * 8 + (lane >> 4) * 8);
              mma(S[i][(2 * j) % NTW], ba, b[0], b[1]);
              mma(S[i][(2 * j + 1) % NTW], ba, b[2], b[3]);
            }
          } else {
            uint32_t b[4];
            ldsm4t(b, w + (ct0 & ~1) * 8 + (lane >> 4) * 8);
            mma(S[i][0], ba, ct0 & 1 ? b[2] : b[0], ct0 & 1 ? b[3] : b[1]);
          }
        }
      }
    }
    state_out();
  }
#pragma unroll
  for (int i = 0; i < MPW; ++i)
#pragma unroll
    for (int j = 0; j < NTW; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int k = (rt0 + i) * 16 + g4 + 8 * (e >> 1), c = (ct0 + j) * 8 + t4 * 2 + (e & 1);
        if (k < N && c < nv) Sg[(int64_t)k * a.dv + c] = S[i][j][e];
      }
}

// ---- gated norm --------------------------------------------------------------------------------
// act = rmsnorm(y * silu(z)) * w, the row cut into equal parts with a root mean square each; one CTA per (part, row)
constexpr int kGT = 512;
template <typename TZ, typename TA, int V>
__global__ void __launch_bounds__(kGT) gated_norm_kernel(const float* __restrict__ y, int64_t ldy, const TZ* __restrict__ z, int64_t ldz,
                                                         const float* __restrict__ w, TA* __restrict__ act, int64_t lda, int n, float eps) {
  extern __shared__ float u_s[];
  __shared__ float red[32];
  griddep_launch();
  griddep_wait();
  const int64_t row = blockIdx.y;
  const int c0 = blockIdx.x * n;
  const float* yr = y + row * ldy + c0;
  const TZ* zr = z + row * ldz + c0;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < n; i += kGT * V) {
    float u[V];
    if (V == 4) {
      const float4 f = *reinterpret_cast<const float4*>(yr + i), g = act_load4(zr + i);
      u[0] = f.x * silu_s(g.x); u[1 % V] = f.y * silu_s(g.y); u[2 % V] = f.z * silu_s(g.z); u[3 % V] = f.w * silu_s(g.w);
    } else {
      u[0] = yr[i] * silu_s(act_load(zr + i));
    }
#pragma unroll
    for (int v = 0; v < V; ++v) { u_s[i + v] = u[v]; ss = fmaf(u[v], u[v], ss); }
  }
  const float r = 1.f / sqrtf(block_sum(ss, red) / (float)n + eps);
  TA* out = act + row * lda + c0;
  for (int i = threadIdx.x * V; i < n; i += kGT * V) {
    if (V == 4) {
      const float4 g = *reinterpret_cast<const float4*>(w + c0 + i);
      act_store4(out + i, make_float4(u_s[i] * r * g.x, u_s[i + 1 % V] * r * g.y, u_s[i + 2 % V] * r * g.z, u_s[i + 3 % V] * r * g.w));
    } else {
      act_store(out + i, u_s[i] * r * w[c0 + i]);
    }
  }
}
template <typename TZ, typename TA>
int launch_gated(const float* y, int64_t ldy, const void* z, int64_t ldz, const float* w, void* act, int64_t lda, int64_t rows, int64_t groups,
                 int64_t n, float eps, cudaStream_t st) {
  const bool v4 = n % 4 == 0 && ldy % 4 == 0 && ldz % 4 == 0 && lda % 4 == 0 && !((uintptr_t)z & 15);
  auto kern = v4 ? gated_norm_kernel<TZ, TA, 4> : gated_norm_kernel<TZ, TA, 1>;
  const size_t smem = sizeof(float) * (size_t)n;
  if (smem > 200 * 1024) return CB_ERR_SHAPE;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return (int)cb_launch(kern, dim3((unsigned)groups, (unsigned)rows), dim3(kGT), smem, st, y, ldy, (const TZ*)z, ldz, w, (TA*)act, lda, (int)n, eps);
}

int64_t al(int64_t x) { return (x + 255) & ~(int64_t)255; }

template <int NP>
int launch_scan(const SsdArgs& s, int segs, cudaStream_t st) {
  auto kern = ssd_scan_kernel<NP>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Plan<NP>::bytes);
  if (e != cudaSuccess) return (int)e;
  return (int)cb_launch(kern, dim3((unsigned)((s.r.dv + VS - 1) / VS), (unsigned)s.r.H, (unsigned)segs), dim3(kST), Plan<NP>::bytes, st, s);
}

}  // namespace

// Whether the chunked kernels take heads of this size (16-byte rows).
CB_EXPORT int cb_ssd_chunk_ok(int64_t dk, int64_t dv) { return dk % 8 == 0 && dv % 8 == 0 && dk >= 8 && dk <= 256; }

CB_EXPORT int64_t cb_ssd_chunk_scratch(int64_t rows, int64_t H, int64_t conv_width) {
  return al(rows * conv_width * 2) + 2 * al(rows * H * 4);
}

// `segs` segments of at most `max_rows` rows in chunks: bf16 projection rows [C | B | x | ...] (C at column 0, B at k_col, x at
// v_col; the first ring_w columns pass the convolution), fp32 step-size pre-activations in `gates`; read-outs go to
// `act` as fp32 [rows, lda].  The convolution ring is only read (cb_linrec_ring afterwards).
CB_EXPORT int cb_ssd_chunk(const void* args, int64_t segs, int64_t max_rows, int64_t rows, void* scratch, int64_t scratch_bytes, void* stream) {
  if (!args || !scratch || segs < 1 || segs > 65535 || rows < 1 || max_rows < 1) return CB_ERR_ARG;
  SsdArgs s;
  s.r = *(const LinrecArgs*)args;
  const LinrecArgs& a = s.r;
  if (!a.proj || !a.gates || !a.act || !a.seg_row || !a.seg_pos || !a.seg_slot || !a.S || !a.ring || !a.conv_w || !a.A_log || !a.dt_bias || !a.D ||
      a.H < 1 || a.G < 1 || a.H % a.G || a.taps < 1 || a.taps > a.ring_mask + 1)
    return CB_ERR_ARG;
  if (!cb_ssd_chunk_ok(a.dk, a.dv) || a.ldp % 2 || a.ring_w % 8 || a.k_col % 8 || a.v_col % 8 || a.lda % 2 || max_rows > 64 * 65535ll) return CB_ERR_SHAPE;
  if (scratch_bytes < cb_ssd_chunk_scratch(rows, a.H, a.ring_w)) return CB_ERR_ARG;
  unsigned char* p = (unsigned char*)scratch;
  s.xc = (bf16*)p; p += al(rows * a.ring_w * 2);
  s.a = (float*)p; p += al(rows * a.H * 4);
  s.dt = (float*)p;
  s.y = (float*)a.act;
  cudaStream_t st = (cudaStream_t)stream;
  const int cblocks = (int)((a.ring_w / 2 + kCT - 1) / kCT);
  const dim3 grid((unsigned)(cblocks + (a.H + kCT - 1) / kCT), (unsigned)((max_rows + Q - 1) / Q), (unsigned)segs);
  cudaError_t e;
  if (a.taps == 4) e = cb_launch(ssd_conv_kernel<4>, grid, dim3(kCT), 0, st, s, cblocks);
  else if (a.taps == 3) e = cb_launch(ssd_conv_kernel<3>, grid, dim3(kCT), 0, st, s, cblocks);
  else if (a.taps == 2) e = cb_launch(ssd_conv_kernel<2>, grid, dim3(kCT), 0, st, s, cblocks);
  else e = cb_launch(ssd_conv_kernel<0>, grid, dim3(kCT), 0, st, s, cblocks);
  if (e != cudaSuccess) return (int)e;
  if (a.dk <= 32) return launch_scan<32>(s, (int)segs, st);
  if (a.dk <= 64) return launch_scan<64>(s, (int)segs, st);
  if (a.dk <= 128) return launch_scan<128>(s, (int)segs, st);
  return launch_scan<256>(s, (int)segs, st);
}

// `segs` segments token by token (seg_row null: one row each); p_f32: projection rows are fp32, f32: the ring is fp32 (else bf16).
CB_EXPORT int cb_ssd_step(const void* args, int64_t segs, int64_t p_f32, int64_t f32, void* stream) {
  if (!args || segs < 1 || segs > 65535) return CB_ERR_ARG;
  SsdArgs s;
  s.r = *(const LinrecArgs*)args;
  s.xc = nullptr; s.a = s.dt = nullptr; s.y = (float*)s.r.act;
  const LinrecArgs& a = s.r;
  if (!a.proj || !a.gates || !a.act || !a.seg_pos || !a.seg_slot || !a.S || !a.ring || !a.conv_w || !a.A_log || !a.dt_bias || !a.D || a.H < 1 ||
      a.G < 1 || a.H % a.G || a.dk < 1 || a.dv < 1 || a.taps < 1 || a.taps > a.ring_mask + 1)
    return CB_ERR_ARG;
  cudaStream_t st = (cudaStream_t)stream;
  if (f32) return launch_step<float, float>(s, (int)segs, st);
  return p_f32 ? launch_step<float, bf16>(s, (int)segs, st) : launch_step<bf16, bf16>(s, (int)segs, st);
}

// act[r, c] = y[r, c] silu(z[r, c]) / rms(its part of the row) * w[c]; `groups` equal parts of n columns.  y fp32; z_f32 / f32: type
// of z / of act (else bf16).
CB_EXPORT int cb_gated_norm(const void* y, int64_t ldy, const void* z, int64_t ldz, const void* w, void* act, int64_t lda, int64_t rows,
                            int64_t groups, int64_t n, float eps, int64_t z_f32, int64_t f32, void* stream) {
  if (!y || !z || !w || !act || rows < 1 || rows > 65535 || groups < 1 || n < 1) return CB_ERR_ARG;
  cudaStream_t st = (cudaStream_t)stream;
  if (f32) return launch_gated<float, float>((const float*)y, ldy, z, ldz, (const float*)w, act, lda, rows, groups, n, eps, st);
  if (z_f32) return launch_gated<float, bf16>((const float*)y, ldy, z, ldz, (const float*)w, act, lda, rows, groups, n, eps, st);
  return launch_gated<bf16, bf16>((const float*)y, ldy, z, ldz, (const float*)w, act, lda, rows, groups, n, eps, st);
}
