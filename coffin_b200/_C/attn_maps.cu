// Attention with several score maps per head over the same values: key/value append, the plain row kernel (any
// sizes, fp32 or bf16 pages) and the kernel that merges key splits, combines the maps and finishes the head.
// The tensor-core kernels for prompts and decoding are attn_maps_flash.cu.
#include "attn_maps.cuh"

namespace {

// Keys (turned) and values (mixed) of a row into its page; with `turn_q` its queries are turned in place.
template <typename TP, typename TA>
__global__ void __launch_bounds__(256) maps_append_kernel(const AttnMapsArgs a, int turn_q) {
  griddep_launch();
  griddep_wait();
  const int row = blockIdx.x, seg = a.row_seg ? a.row_seg[row] : row, pos = a.positions[row];
  if (pos < 0) return;
  const int64_t slot = (int64_t)a.tables[(int64_t)seg * a.ldbt + pos / kPage] * kPage + pos % kPage;
  TP* p = reinterpret_cast<TP*>(const_cast<void*>(a.proj)) + (int64_t)row * a.ldp;
  const int nk = a.G * a.maps * a.dim, nv = a.G * a.vdim;
  TA* kp = reinterpret_cast<TA*>(a.kpool) + slot * pool_ldk(a);
  TA* vp = reinterpret_cast<TA*>(a.vpool) + slot * pool_ldv(a);
  const float2* cs = a.cs + (int64_t)row * a.rot_half;
  const TP* w = a.v0 ? reinterpret_cast<const TP*>(a.v0) + (int64_t)row * a.ldv0 : nullptr;
  for (int c = threadIdx.x; c < nk; c += 256) act_store(kp + c, turned(p + a.k_col, c, c % a.dim, cs, a.rot_half));
  for (int c = threadIdx.x; c < nv; c += 256) act_store(vp + c, mixed(act_load(p + a.v_col + c), w ? act_load(w + c) : 0.f, a));
  if (turn_q && a.rot_half) {
    const int H = a.H * a.maps;
    for (int e = threadIdx.x; e < H * a.rot_half; e += 256) {
      const int i = e % a.rot_half;
      TP* q = p + (e / a.rot_half) * a.dim + 2 * i;
      const float2 t = cs[i];
      const float u = act_load(q), v = act_load(q + 1);
      act_store(q, u * t.x - v * t.y);
      act_store(q + 1, v * t.x + u * t.y);
    }
  }
}

// The same for bf16 rows and pages whose heads are whole 16-byte pieces.
__global__ void __launch_bounds__(256) maps_append8_kernel(const AttnMapsArgs a, int turn_q) {
  griddep_launch();
  griddep_wait();
  const int row = blockIdx.x, seg = a.row_seg ? a.row_seg[row] : row, pos = a.positions[row];
  if (pos < 0) return;
  const int64_t slot = (int64_t)a.tables[(int64_t)seg * a.ldbt + pos / kPage] * kPage + pos % kPage;
  bf16* p = reinterpret_cast<bf16*>(const_cast<void*>(a.proj)) + (int64_t)row * a.ldp;
  bf16* kp = reinterpret_cast<bf16*>(a.kpool) + slot * pool_ldk(a);
  bf16* vp = reinterpret_cast<bf16*>(a.vpool) + slot * pool_ldv(a);
  const float2* cs = a.cs + (int64_t)row * a.rot_half;
  const bf16* w = a.v0 ? reinterpret_cast<const bf16*>(a.v0) + (int64_t)row * a.ldv0 : nullptr;
  const int nk = a.G * a.maps * a.dim / 8, nv = a.G * a.vdim / 8, nq = turn_q && a.rot_half ? a.H * a.maps * a.dim / 8 : 0;
  for (int e = threadIdx.x; e < nk + nq + nv; e += 256) {
    float f[8];
    if (e < nk + nq) {
      const int c = (e < nk ? e : e - nk) * 8, i0 = c % a.dim / 2;
      bf16* src = p + (e < nk ? a.k_col : 0) + c;
      bf16x8_to_float(*reinterpret_cast<const uint4*>(src), f);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        if (i0 + i < a.rot_half) {
          const float2 t = cs[i0 + i];
          const float u = f[2 * i], v = f[2 * i + 1];
          f[2 * i] = u * t.x - v * t.y;
          f[2 * i + 1] = v * t.x + u * t.y;
        }
      }
      *reinterpret_cast<uint4*>(e < nk ? kp + c : src) = float_to_bf16x8(f);
    } else {
      const int c = (e - nk - nq) * 8;
      bf16x8_to_float(*reinterpret_cast<const uint4*>(p + a.v_col + c), f);
      if (w) {
        float g[8];
        bf16x8_to_float(*reinterpret_cast<const uint4*>(w + c), g);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] = mixed(f[i], g[i], a);
      }
      *reinterpret_cast<uint4*>(vp + c) = float_to_bf16x8(f);
    }
  }
}

// The extended form: heads are normed, then turned; values may turn; keys that are their own values stay as projected, with their
// factor beside them.  2^sh threads per head; V columns per access (8: bf16, a head is one access of its threads and stays in
// registers).
template <typename T, int V>
__device__ __forceinline__ void load_cols(const T* p, int n, float* f) {
  if (V == 8) {
    bf16x8_to_float(*reinterpret_cast<const uint4*>(p), f);
  } else {
    f[0] = act_load(p);
    f[1] = n > 1 ? act_load(p + 1) : 0.f;
  }
}
template <typename T, int V>
__device__ __forceinline__ void store_cols(T* p, int n, const float* f) {
  if (V == 8) {
    *reinterpret_cast<uint4*>(p) = float_to_bf16x8(f);
  } else {
    act_store(p, f[0]);
    if (n > 1) act_store(p + 1, f[1]);
  }
}
// w[c ..] (n columns left) times r
template <int V>
__device__ __forceinline__ void weigh(float* f, const float* w, int n, float r) {
  if (V == 8) {
    const float4 a = *reinterpret_cast<const float4*>(w), b = *reinterpret_cast<const float4*>(w + 4);
    const float g[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] *= r * g[i];
  } else {
    f[0] *= r * w[0];
    if (n > 1) f[1] *= r * w[1];
  }
}
template <int V>
__device__ __forceinline__ void turn_cols(float* f, const float2* t, int pairs) {
  if (V == 8 && pairs >= 4 && !((uintptr_t)t & 15)) {
    const float4 a = *reinterpret_cast<const float4*>(t), b = *reinterpret_cast<const float4*>(t + 2);
    const float c[4] = {a.x, a.z, b.x, b.z}, s[4] = {a.y, a.w, b.y, b.w};
#pragma unroll
    for (int i = 0; i < V / 2; ++i) {
      const float x = f[2 * i], y = f[2 * i + 1];
      f[2 * i] = x * c[i & 3] - y * s[i & 3];
      f[2 * i + 1] = y * c[i & 3] + x * s[i & 3];
    }
    return;
  }
#pragma unroll
  for (int i = 0; i < V / 2; ++i)
    if (i < pairs) {
      const float2 c = t[i];
      const float x = f[2 * i], y = f[2 * i + 1];
      f[2 * i] = x * c.x - y * c.y;
      f[2 * i + 1] = y * c.x + x * c.y;
    }
}
template <typename TP, typename TA, int V>
__global__ void __launch_bounds__(512) maps_prep_kernel(const AttnMapsArgs a, int turn_q, int sh) {
  griddep_launch();
  griddep_wait();
  const int row = blockIdx.x, seg = a.row_seg ? a.row_seg[row] : row, pos = a.positions[row];
  if (pos < 0) return;
  const int64_t block = a.tables[(int64_t)seg * a.ldbt + pos / kPage], slot = block * kPage + pos % kPage;
  TP* p = reinterpret_cast<TP*>(const_cast<void*>(a.proj)) + (int64_t)row * a.ldp;
  const int nk = a.G * a.maps, nq = turn_q ? a.H * a.maps : 0, nv = a.kr ? 0 : a.G, total = nk + nq + nv;
  const int per = blockDim.x >> sh, l = threadIdx.x & ((1 << sh) - 1), stride = V << sh;
  for (int u0 = 0; u0 < total; u0 += per) {
    const int u = u0 + (threadIdx.x >> sh);
    const bool ok = u < total, key = u < nk, val = u >= nk + nq;
    const int n = val ? a.vdim : a.dim, hd = key ? u : (val ? u - nk - nq : u - nk);      // columns of the head, its number
    TP* src = p + (key ? a.k_col : (val ? a.v_col : 0)) + hd * n;
    float f[V], rstd = 1.f;
    if (V == 8 && ok && l * V < n) load_cols<TP, V>(src + l * V, n, f);        // this thread's only columns
    if (a.norm) {
      float ss = 0.f;
      if (ok && !val)
        for (int c = l * V; c < n; c += stride) {
          if (V != 8) load_cols<TP, V>(src + c, n - c, f);
#pragma unroll
          for (int i = 0; i < V; ++i) ss = fmaf(f[i], f[i], ss);
        }
      for (int o = 1 << sh >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      rstd = 1.f / sqrtf(ss / (float)n + a.eps);
    }
    if (!ok) continue;                                           // the last pass
    const bool as_is = key && a.kr;
    if (as_is && l == 0) a.kr[factor_at(a, block, hd) + pos % kPage] = rstd;
    const float* nw = val ? nullptr : (key ? a.kn : a.qn);
    const float2* turn = val ? a.vcs + (int64_t)row * (a.vdim / 2) : a.cs + (int64_t)row * a.rot_half;
    const int half = val ? (a.vcs ? a.vdim / 2 : 0) : a.rot_half;
    for (int c = l * V; c < n; c += stride) {
      if (V != 8) load_cols<TP, V>(src + c, n - c, f);
      if (val && a.v0) {
        float g[V];
        load_cols<TP, V>(reinterpret_cast<const TP*>(a.v0) + (int64_t)row * a.ldv0 + hd * n + c, n - c, g);
#pragma unroll
        for (int i = 0; i < V; ++i) f[i] = mixed(f[i], g[i], a);
      }
      if (!as_is) {
        if (nw) {
          weigh<V>(f, nw + c, n - c, rstd);
        } else if (!val) {
#pragma unroll
          for (int i = 0; i < V; ++i) f[i] *= rstd;
        }
        turn_cols<V>(f, turn + c / 2, half - c / 2);
      }
      if (key) store_cols<TA, V>(reinterpret_cast<TA*>(a.kpool) + slot * pool_ldk(a) + hd * n + c, n - c, f);
      else if (val) store_cols<TA, V>(reinterpret_cast<TA*>(a.vpool) + slot * pool_ldv(a) + hd * n + c, n - c, f);
      else store_cols<TP, V>(src + c, n - c, f);
    }
  }
}
template <typename TP, typename TA, int V>
int launch_prep(const AttnMapsArgs& a, int rows, int turn_q, cudaStream_t st) {
  const int most = ((a.kr || a.dim > a.vdim ? a.dim : a.vdim) + V - 1) / V, total = (turn_q ? a.H + a.G : a.G) * a.maps + (a.kr ? 0 : a.G);
  int sh = 0;
  while (sh < 5 && 1 << sh < most) ++sh;
  const int passes = ((total << sh) + 511) / 512, per = (total + passes - 1) / passes;     // as few threads as the passes need
  int threads = ((per << sh) + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  return (int)cb_launch(maps_prep_kernel<TP, TA, V>, dim3((unsigned)rows), dim3((unsigned)threads), 0, st, a, turn_q, sh);
}

// One CTA per (query row, head, map): 128 keys at a time, scores by thread, running softmax, values by column.
constexpr int kRT = 128;
template <typename TP, typename TA>
__global__ void __launch_bounds__(kRT) maps_row_kernel(const AttnMapsArgs a) {
  extern __shared__ float sm[];
  __shared__ float red[32];
  float* q = sm;                 // [dim]
  float* pr = q + a.dim;         // [kRT]
  float* o = pr + kRT;           // [vdim]
  const int tid = threadIdx.x, vh = blockIdx.x, row = blockIdx.y;
  griddep_launch();
  griddep_wait();
  const int seg = a.row_seg ? a.row_seg[row] : row, pos = a.positions[row];
  const int h = vh / a.maps, map = vh % a.maps, g = h / (a.H / a.G);
  float* po = a.part_o + ((int64_t)row * a.H * a.maps + vh) * a.nsplit * a.vdim;
  float* pm = a.part_ml + ((int64_t)row * a.H * a.maps + vh) * a.nsplit * 2;
  if (pos < 0) return;
  const float f = a.scale * query_temp(a, pos), inv_cap = a.cap > 0.f ? 1.f / a.cap : 0.f;
  const TP* qr = reinterpret_cast<const TP*>(a.proj) + (int64_t)row * a.ldp + (int64_t)vh * a.dim;
  for (int c = tid; c < a.dim; c += kRT) q[c] = act_round<TA>(act_load(qr + c)) * f;
  for (int c = tid; c < a.vdim; c += kRT) o[c] = 0.f;
  __syncthreads();
  const int64_t ldk = pool_ldk(a), ldv = a.kr ? ldk : pool_ldv(a);
  const TA* K = reinterpret_cast<const TA*>(a.kpool) + (int64_t)(g * a.maps + map) * a.dim;
  const TA* V = a.kr ? K : reinterpret_cast<const TA*>(a.vpool) + (int64_t)g * a.vdim;
  const int* bt = a.tables + (int64_t)seg * a.ldbt;
  const float r1 = a.r1 ? a.r1[h] : 0.f, r2 = a.r1 ? a.r2[h] : 0.f;
  float m = -INFINITY, l = 0.f;
  for (int k0 = first_key(a, pos); k0 <= pos; k0 += kRT) {
    const int n = min(kRT, pos + 1 - k0), j = k0 + tid;
    float s = -INFINITY;
    if (tid < n) {
      const TA* kr = K + ((int64_t)bt[j / kPage] * kPage + j % kPage) * ldk;
      float d = 0.f;
      for (int c = 0; c < a.dim; ++c) d = fmaf(q[c], act_load(kr + c), d);
      if (a.kr) d *= a.kr[factor_at(a, bt[j / kPage], g) + j % kPage];
      s = a.cap > 0.f ? a.cap * tanhf(d * inv_cap) : d;
      if (a.r1) s -= r1 * log1pf(r2 * (float)(pos - j));
    }
    const float mn = fmaxf(m, block_max(s, red));
    const float p = tid < n ? expf(s - mn) : 0.f, w = expf(m - mn);
    pr[tid] = p;
    l = l * w + block_sum(p, red);
    m = mn;
    __syncthreads();
    for (int c = tid; c < a.vdim; c += kRT) {
      float acc = o[c] * w;
      for (int i = 0; i < n; ++i) {
        const int jj = k0 + i;
        acc = fmaf(pr[i], act_load(V + ((int64_t)bt[jj / kPage] * kPage + jj % kPage) * ldv + c), acc);
      }
      o[c] = acc;
    }
    __syncthreads();
  }
  for (int c = tid; c < a.vdim; c += kRT) po[c] = o[c];
  for (int s = 1; s < a.nsplit; ++s)
    for (int c = tid; c < a.vdim; c += kRT) po[(int64_t)s * a.vdim + c] = 0.f;
  for (int s = tid; s < a.nsplit; s += kRT) { pm[2 * s] = s ? -INFINITY : m; pm[2 * s + 1] = s ? 0.f : l; }
}

// One warp per (row, head): merge the key splits of every map (and its sink), o = a_0 - lambda a_1 (two maps), RMS norm
// over the head's values without weight (two maps), times post_scale, times sigmoid(gate) per head and per element.
struct ElemGate { const void* p; int64_t ld; int f32; };        // pre-activations [rows, H * vdim]
__device__ __forceinline__ float elem_gate(const ElemGate& g, int64_t row, int c) {
  return sigmoid_x(g.f32 ? reinterpret_cast<const float*>(g.p)[row * g.ld + c]
                         : __bfloat162float(reinterpret_cast<const bf16*>(g.p)[row * g.ld + c]));
}
constexpr int kVMax = 16;      // values per lane: vdim <= 512; at most 64 splits (4 in the warp form)
template <typename TA>
__global__ void __launch_bounds__(128) maps_finish_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                                          const float* __restrict__ gates, int64_t ldg, TA* __restrict__ act,
                                                          int64_t lda, const int* __restrict__ positions, int rows, int H,
                                                          int maps, int vdim, int nsplit, float lambda, float post_scale, float eps,
                                                          const float* __restrict__ sink, const ElemGate eg, const float2* __restrict__ vcs) {
  griddep_launch();
  griddep_wait();
  const int64_t w = (int64_t)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (w >= (int64_t)rows * H) return;
  const int64_t row = w / H;
  const int h = (int)(w % H);
  if (positions[row] < 0) return;
  const bool v4 = vdim % 4 == 0;
  float o[kVMax];
#pragma unroll
  for (int i = 0; i < kVMax; ++i) o[i] = 0.f;
  if (nsplit == 1 && v4 && maps == 2 && !sink) {                // prompts: everything a lane needs in one round of loads
    const int64_t vh = (row * H + h) * 2;
    const float d0 = part_ml[vh * 2 + 1], d1 = part_ml[vh * 2 + 3];
    const float* po = part_o + vh * vdim;
    float4 p0[kVMax / 4], p1[kVMax / 4];
#pragma unroll
    for (int i = 0; i < kVMax / 4; ++i) {
      const int v = 4 * (lane + 32 * i);
      p0[i] = v < vdim ? *reinterpret_cast<const float4*>(po + v) : make_float4(0.f, 0.f, 0.f, 0.f);
      p1[i] = v < vdim ? *reinterpret_cast<const float4*>(po + vdim + v) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const float f0 = 1.f / d0, f1 = -lambda / d1;
#pragma unroll
    for (int i = 0; i < kVMax / 4; ++i) {
      o[4 * i] = fmaf(f1, p1[i].x, f0 * p0[i].x); o[4 * i + 1] = fmaf(f1, p1[i].y, f0 * p0[i].y);
      o[4 * i + 2] = fmaf(f1, p1[i].z, f0 * p0[i].z); o[4 * i + 3] = fmaf(f1, p1[i].w, f0 * p0[i].w);
    }
  } else
  for (int mp = 0; mp < maps; ++mp) {
    const int64_t vh = (row * H + h) * maps + mp;
    const float* ml = part_ml + vh * nsplit * 2;
    const float* po = part_o + vh * nsplit * vdim;
    float M = -INFINITY;
    if (lane < nsplit) M = ml[2 * lane];
    M = warp_max(M);
    const float sk = sink ? sink[h * maps + mp] : -INFINITY;
    M = fmaxf(M, sk);
    // splits are filled from the front: each lane weighs its own, the sums walk the filled ones
    float fac = 0.f, den = 0.f;
    if (lane < nsplit && ml[2 * lane] != -INFINITY) { fac = expf(ml[2 * lane] - M); den = fac * ml[2 * lane + 1]; }
    den = warp_sum(den);
    if (sink) den += expf(sk - M);
    fac *= (mp == 0 ? 1.f : -lambda) / den;
    const int used = __popc(__ballot_sync(0xffffffffu, lane < nsplit && ml[2 * lane] != -INFINITY));
    for (int s = 0; s < used; ++s) {
      const float f = __shfl_sync(0xffffffffu, fac, s);
#pragma unroll
      for (int i = 0; i < kVMax / 4; ++i) {                      // columns of a lane: 4 (lane + 32 i) .. + 3
        const int v = 4 * (lane + 32 * i);
        if (v + 3 < vdim && v4) {
          const float4 p = *reinterpret_cast<const float4*>(po + (int64_t)s * vdim + v);
          o[4 * i] = fmaf(f, p.x, o[4 * i]); o[4 * i + 1] = fmaf(f, p.y, o[4 * i + 1]);
          o[4 * i + 2] = fmaf(f, p.z, o[4 * i + 2]); o[4 * i + 3] = fmaf(f, p.w, o[4 * i + 3]);
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (v + e < vdim) o[4 * i + e] = fmaf(f, po[(int64_t)s * vdim + v + e], o[4 * i + e]);
        }
      }
    }
  }
  float r = post_scale;
  if (maps > 1) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < kVMax; ++i) ss = fmaf(o[i], o[i], ss);
    r *= 1.f / sqrtf(warp_sum(ss) / (float)vdim + eps);
  }
  if (gates) r *= sigmoid_x(gates[row * ldg + h]);
  TA* out = act + row * lda + (int64_t)h * vdim;
#pragma unroll
  for (int i = 0; i < kVMax / 4; ++i) {
    const int v = 4 * (lane + 32 * i);
    if (vcs)
#pragma unroll
      for (int e = 0; e < 4; e += 2)
        if (v + e + 1 < vdim) turn_back(o[4 * i + e], o[4 * i + e + 1], vcs[row * (vdim / 2) + (v + e) / 2]);
    if (eg.p)
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (v + e < vdim) o[4 * i + e] *= elem_gate(eg, row, h * vdim + v + e);
    if (v + 3 < vdim && v4 && lda % 4 == 0) {
      act_store4(out + v, make_float4(o[4 * i] * r, o[4 * i + 1] * r, o[4 * i + 2] * r, o[4 * i + 3] * r));
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (v + e < vdim) act_store(out + v + e, o[4 * i + e] * r);
    }
  }
}

// The same for rows with many key splits (decode): one CTA per (row, head), its warps share the (map, split) sums.
constexpr int kWT = 256;
template <typename TA>
__global__ void __launch_bounds__(kWT) maps_finish_wide_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                                               const float* __restrict__ gates, int64_t ldg, TA* __restrict__ act,
                                                               int64_t lda, const int* __restrict__ positions, int H, int maps,
                                                               int vdim, int nsplit, float lambda, float post_scale, float eps,
                                                               const float* __restrict__ sink, const ElemGate eg, const float2* __restrict__ vcs) {
  extern __shared__ float sm[];                        // [warps][vdim]
  __shared__ float red[32];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int64_t row = blockIdx.y;
  const int h = blockIdx.x;
  griddep_launch();
  griddep_wait();
  if (positions[row] < 0) return;
  float o[kVMax];
#pragma unroll
  for (int i = 0; i < kVMax; ++i) o[i] = 0.f;
  for (int mp = 0; mp < maps; ++mp) {
    const int64_t vh = (row * H + h) * maps + mp;
    const float* ml = part_ml + vh * nsplit * 2;
    const float* po = part_o + vh * nsplit * vdim;
    float2 v[2];                                       // splits lane and lane + 32
#pragma unroll
    for (int k = 0; k < 2; ++k)
      v[k] = lane + 32 * k < nsplit ? *reinterpret_cast<const float2*>(ml + 2 * (lane + 32 * k)) : make_float2(-INFINITY, 0.f);
    const float sk = sink ? sink[h * maps + mp] : -INFINITY, M = fmaxf(sk, warp_max(fmaxf(v[0].x, v[1].x)));
    float fac[2];
#pragma unroll
    for (int k = 0; k < 2; ++k) fac[k] = v[k].x == -INFINITY ? 0.f : expf(v[k].x - M);
    const float den = warp_sum(fac[0] * v[0].y + fac[1] * v[1].y) + (sink ? expf(sk - M) : 0.f), c = (mp == 0 ? 1.f : -lambda) / den;
    const int used = __popc(__ballot_sync(0xffffffffu, v[0].x != -INFINITY)) + __popc(__ballot_sync(0xffffffffu, v[1].x != -INFINITY));
#pragma unroll 4
    for (int s = warp; s < used; s += kWT / 32) {
      const float f = c * __shfl_sync(0xffffffffu, s < 32 ? fac[0] : fac[1], s & 31);
#pragma unroll
      for (int i = 0; i < kVMax; ++i) {
        const int v_ = lane + 32 * i;
        if (v_ < vdim) o[i] = fmaf(f, po[(int64_t)s * vdim + v_], o[i]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < kVMax; ++i)
    if (lane + 32 * i < vdim) sm[warp * vdim + lane + 32 * i] = o[i];
  __syncthreads();
  float x[2] = {0.f, 0.f}, ss = 0.f;
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const int c = tid + kWT * k;
    if (c < vdim)
#pragma unroll
      for (int w = 0; w < kWT / 32; ++w) x[k] += sm[w * vdim + c];
    ss = fmaf(x[k], x[k], ss);
    if (vcs) {                                                   // the other entry of a pair is the neighbouring thread's
      const float y = __shfl_xor_sync(0xffffffffu, x[k], 1);
      if ((c | 1) < vdim) {
        const float2 t = vcs[row * (vdim / 2) + c / 2];
        x[k] = c & 1 ? x[k] * t.x - y * t.y : x[k] * t.x + y * t.y;
      }
    }
  }
  float r = post_scale;
  if (maps > 1) r *= 1.f / sqrtf(block_sum(ss, red) / (float)vdim + eps);
  if (gates) r *= sigmoid_x(gates[row * ldg + h]);
#pragma unroll
  for (int k = 0; k < 2; ++k)
    if (tid + kWT * k < vdim) {
      const int c = h * vdim + tid + kWT * k;
      act_store(act + row * lda + c, x[k] * r * (eg.p ? elem_gate(eg, row, c) : 1.f));
    }
}

bool maps_args_ok(const AttnMapsArgs& a) {
  return a.proj && a.kpool && a.vpool && a.tables && a.positions && a.H > 0 && a.G > 0 && a.H % a.G == 0 && a.maps >= 1 && a.dim > 0 &&
         a.vdim > 0 && 2 * a.rot_half <= a.dim && (!a.rot_half || a.cs) && !a.r1 == !a.r2 && (!a.kr || (a.maps == 1 && a.dim == a.vdim && !a.vcs));
}

}  // namespace

CB_EXPORT int cb_attn_maps_args_size() { return (int)sizeof(AttnMapsArgs); }

// Keys and values of `rows` projection rows into the pages; turn_q: their queries are turned in place.
CB_EXPORT int cb_attn_maps_append(const void* args, int64_t rows, int64_t turn_q, int64_t p_f32, int64_t f32, void* stream) {
  if (!args || rows < 1) return CB_ERR_ARG;
  const AttnMapsArgs& a = *(const AttnMapsArgs*)args;
  if (!maps_args_ok(a)) return CB_ERR_ARG;
  cudaStream_t st = (cudaStream_t)stream;
  const dim3 grid((unsigned)rows), block(256);
  const int tq = (int)turn_q;
  if (extended(a)) {
    if (f32) return launch_prep<float, float, 2>(a, (int)rows, tq, st);
    if (p_f32) return launch_prep<float, bf16, 2>(a, (int)rows, tq, st);
    const bool odd = a.dim % 8 || a.vdim % 8 || a.dim > 256 || a.vdim > 256 || (((uintptr_t)a.qn | (uintptr_t)a.kn) & 15) || a.ldp % 8 || a.k_col % 8 || a.v_col % 8 || pool_ldk(a) % 8 || pool_ldv(a) % 8 || a.ldv0 % 8 ||
                     (((uintptr_t)a.proj | (uintptr_t)a.v0 | (uintptr_t)a.kpool | (uintptr_t)a.vpool) & 15);
    if (odd) return launch_prep<bf16, bf16, 2>(a, (int)rows, tq, st);
    return launch_prep<bf16, bf16, 8>(a, (int)rows, tq, st);
  }
  if (f32) return (int)cb_launch(maps_append_kernel<float, float>, grid, block, 0, st, a, tq);
  if (p_f32) return (int)cb_launch(maps_append_kernel<float, bf16>, grid, block, 0, st, a, tq);
  const bool wide = !(a.dim % 8 || a.vdim % 8 || a.ldp % 8 || a.k_col % 8 || a.v_col % 8 || pool_ldk(a) % 8 || pool_ldv(a) % 8 ||
                      a.ldv0 % 8 || (((uintptr_t)a.proj | (uintptr_t)a.v0 | (uintptr_t)a.kpool | (uintptr_t)a.vpool) & 15));
  if (wide) return (int)cb_launch(maps_append8_kernel, grid, block, 0, st, a, tq);
  return (int)cb_launch(maps_append_kernel<bf16, bf16>, grid, block, 0, st, a, tq);
}

// The plain kernel: every row against the pages (its own key included, so append first).
CB_EXPORT int cb_attn_maps_rows(const void* args, int64_t rows, int64_t p_f32, int64_t f32, void* stream) {
  if (!args || rows < 1 || rows > 65535) return CB_ERR_ARG;
  const AttnMapsArgs& a = *(const AttnMapsArgs*)args;
  if (!maps_args_ok(a) || !a.part_o || !a.part_ml || a.nsplit < 1) return CB_ERR_ARG;
  const size_t smem = sizeof(float) * (size_t)(a.dim + kRT + a.vdim);
  if (smem > 40 * 1024) return CB_ERR_SHAPE;
  cudaStream_t st = (cudaStream_t)stream;
  const dim3 grid((unsigned)(a.H * a.maps), (unsigned)rows), block(kRT);
  if (f32) return (int)cb_launch(maps_row_kernel<float, float>, grid, block, smem, st, a);
  if (p_f32) return (int)cb_launch(maps_row_kernel<float, bf16>, grid, block, smem, st, a);
  return (int)cb_launch(maps_row_kernel<bf16, bf16>, grid, block, smem, st, a);
}

CB_EXPORT int cb_attn_maps_finish(const void* part_o, const void* part_ml, const void* gates, int64_t ldg, void* act, int64_t lda,
                                  const void* positions, int64_t rows, int64_t H, int64_t maps, int64_t vdim, int64_t nsplit,
                                  float lambda, float post_scale, float eps, const void* sink, const void* egate, int64_t lde,
                                  int64_t e_f32, const void* turns, int64_t f32, void* stream) {
  if (!part_o || !part_ml || !act || !positions || rows < 1 || maps < 1 || maps > 2 || nsplit < 1) return CB_ERR_ARG;
  const float* sk = (const float*)sink;
  const ElemGate eg = {egate, lde, (int)e_f32};
  const float2* vcs = (const float2*)turns;
  if (vcs && (maps != 1 || vdim % 2)) return CB_ERR_SHAPE;
  if (vdim > 32 * kVMax || nsplit > 64) return CB_ERR_SHAPE;
  cudaStream_t st = (cudaStream_t)stream;
  // a CTA per head, where there are many splits to walk or few heads to fill the machine with
  if (nsplit > 4 || (nsplit > 1 && maps == 1 && rows * H <= 512)) {
    if (rows > 65535) return CB_ERR_SHAPE;
    const size_t smem = sizeof(float) * (size_t)(kWT / 32) * vdim;
    const dim3 wide((unsigned)H, (unsigned)rows);
    if (f32)
      return (int)cb_launch(maps_finish_wide_kernel<float>, wide, dim3(kWT), smem, st, (const float*)part_o, (const float*)part_ml,
                            (const float*)gates, ldg, (float*)act, lda, (const int*)positions, (int)H, (int)maps, (int)vdim,
                            (int)nsplit, lambda, post_scale, eps, sk, eg, vcs);
    return (int)cb_launch(maps_finish_wide_kernel<bf16>, wide, dim3(kWT), smem, st, (const float*)part_o, (const float*)part_ml,
                          (const float*)gates, ldg, (bf16*)act, lda, (const int*)positions, (int)H, (int)maps, (int)vdim, (int)nsplit,
                          lambda, post_scale, eps, sk, eg, vcs);
  }
  const dim3 grid((unsigned)((rows * H + 3) / 4)), block(128);
  if (f32)
    return (int)cb_launch(maps_finish_kernel<float>, grid, block, 0, st, (const float*)part_o, (const float*)part_ml,
                          (const float*)gates, ldg, (float*)act, lda, (const int*)positions, (int)rows, (int)H, (int)maps,
                          (int)vdim, (int)nsplit, lambda, post_scale, eps, sk, eg, vcs);
  return (int)cb_launch(maps_finish_kernel<bf16>, grid, block, 0, st, (const float*)part_o, (const float*)part_ml,
                        (const float*)gates, ldg, (bf16*)act, lda, (const int*)positions, (int)rows, (int)H, (int)maps, (int)vdim,
                        (int)nsplit, lambda, post_scale, eps, sk, eg, vcs);
}
