// Tensor-core prompt kernel and split-key decode kernel of the multi-map attention (attn_maps.cuh), bf16 pages.
//
// Prompt: one CTA per (128 consecutive query rows of a segment, head, map); keys and values come page by page through
// a two-stage cp.async ring.  Scores, cap, query temperature and softmax are fp32.  The weights stay fp32 across the
// second product: P is split into a bf16 head and a bf16 remainder (16 mantissa bits) and multiplied twice - with two
// maps the result is a difference of two averages, which would amplify a rounded P.
// Decode: one CTA per (key split, key/value head, row) walks its pages with every query head and map of the group, so
// a page is read once; the CTA that owns the newest page appends the token's key and value first.
// Both leave unnormalised sums and (max, denominator) for maps_finish_kernel.
#include "attn_maps.cuh"

namespace {

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
// (x, y) -> packed bf16 head; the remainders replace x and y
__device__ __forceinline__ uint32_t split_head(float& x, float& y) {
  const uint32_t h = pack_bf162(x, y);
  x -= __uint_as_float(h << 16);
  y -= __uint_as_float(h & 0xffff0000u);
  return h;
}

constexpr int kBM = 128, kBN = 64, kFT = 256;
constexpr float kLog2e = 1.4426950408889634f;

// Modes: scores as they are, capped scores, keys that are their own values (one staged page serves both products).
enum FlashMode : int { PLAIN = 0, CAPPED = 1, SHARED = 2 };
template <int DK, int DV, int MODE>
constexpr size_t flash_smem() {
  return sizeof(bf16) * ((size_t)kBM * (DK + 8) + 2 * (size_t)kBN * (DK + 8 + (MODE == SHARED ? 0 : DV + 8))) + (MODE == SHARED ? 2 * kBN * 4 : 0);
}

template <int DK, int DV, int MODE>
__global__ void __launch_bounds__(kFT, 1) maps_flash_kernel(const AttnMapsArgs a) {
  constexpr bool CAP = MODE == CAPPED, KV = MODE == SHARED;
  static_assert(!KV || DK == DV, "values are the keys");
  constexpr int LK = DK + 8, LV = DV + 8, NK = DK / 16, NV = DV / 8;
  constexpr bool QREG = DK <= 128;
  extern __shared__ __align__(128) unsigned char smem[];
  bf16* qs = reinterpret_cast<bf16*>(smem);            // [kBM][LK]
  bf16* ks = qs + kBM * LK;                            // [2][kBN][LK]
  bf16* vs = KV ? ks : ks + 2 * kBN * LK;              // [2][kBN][LV]
  float* fs = reinterpret_cast<float*>(ks + 2 * kBN * LK);       // [2][kBN] factors of the keys (SHARED)
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g4 = lane >> 2, t4 = lane & 3;
  const int vh = blockIdx.y, seg = blockIdx.z;
  griddep_launch();
  griddep_wait();
  const int row0 = a.seg_row[seg], n = a.seg_row[seg + 1] - row0, pos0 = a.seg_pos[seg];
  const int tile = (int)gridDim.x - 1 - (int)blockIdx.x;         // long tiles first
  const int t0 = tile * kBM;
  if (t0 >= n) return;
  const int h = vh / a.maps, map = vh % a.maps, g = h / (a.H / a.G);
  const int64_t ldk = pool_ldk(a), ldv = pool_ldv(a);
  const bf16* K = reinterpret_cast<const bf16*>(a.kpool) + (int64_t)(g * a.maps + map) * a.dim;
  const bf16* V = reinterpret_cast<const bf16*>(a.vpool) + (int64_t)g * a.vdim;
  const int* bt = a.tables + (int64_t)seg * a.ldbt;
  const bf16* Q = reinterpret_cast<const bf16*>(a.proj) + (int64_t)(row0 + t0) * a.ldp + (int64_t)vh * a.dim;
  const int rows = min(kBM, n - t0);
  for (int e = tid; e < kBM * (DK / 8); e += kFT) {
    const int r = e / (DK / 8), c = (e % (DK / 8)) * 8;
    const bool ok = r < rows && c < a.dim;
    cp16(qs + r * LK + c, ok ? Q + (int64_t)r * a.ldp + c : Q, ok);
  }
  const int last = pos0 + t0 + rows - 1, pages = last / kPage + 1, page0 = first_key(a, pos0 + t0) / kPage;
  auto load = [&](int pg) {
    const int64_t base = (int64_t)bt[pg] * kPage;
    bf16* kd = ks + (pg & 1) * kBN * LK;
    bf16* vd = vs + (pg & 1) * kBN * LV;
    for (int e = tid; e < kBN * (DK / 8); e += kFT) {
      const int r = e / (DK / 8), c = (e % (DK / 8)) * 8;
      const bool ok = c < a.dim && pg * kPage + r <= last;
      cp16(kd + r * LK + c, ok ? K + (base + r) * ldk + c : K, ok);
    }
    if (KV) {
      if (tid < kBN / 4) cp16(fs + (pg & 1) * kBN + tid * 4, a.kr + factor_at(a, bt[pg], g) + tid * 4, true);
    } else {
      for (int e = tid; e < kBN * (DV / 8); e += kFT) {
        const int r = e / (DV / 8), c = (e % (DV / 8)) * 8;
        const bool ok = c < a.vdim && pg * kPage + r <= last;
        cp16(vd + r * LV + c, ok ? V + (base + r) * ldv + c : V, ok);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load(page0);
  float o[NV][4];
#pragma unroll
  for (int i = 0; i < NV; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float mx[2] = {kNoKey, kNoKey}, den[2] = {0.f, 0.f};       // finite: with a window a page may hold no key of a row
  const int rlo = warp * 16 + g4;                                // tile rows of this lane: rlo, rlo + 8
  const int plo = pos0 + t0 + rlo, phi = plo + 8, klo = first_key(a, plo), khi = first_key(a, phi);   // positions, first keys
  const float inv_cap = CAP ? 1.f / a.cap : 0.f;
  float f[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    f[i] = a.scale * query_temp(a, i ? phi : plo);
    f[i] *= CAP ? 2.f * kLog2e * inv_cap : kLog2e;               // CAP: exponent of exp(2 s / cap); else log2 units
  }
  const float r1 = KV && a.r1 ? a.r1[h] : 0.f, r2 = KV && a.r1 ? a.r2[h] : 0.f;
  const float cap2 = a.cap * kLog2e;
  uint32_t qf[QREG ? NK : 1][4];
  const int warp_last = pos0 + t0 + warp * 16 + 15, warp_first = first_key(a, pos0 + t0 + warp * 16), warp_full = first_key(a, warp_last);
  for (int pg = page0; pg < pages; ++pg) {
    if (pg + 1 < pages) {
      load(pg + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    if (QREG && pg == page0) {
#pragma unroll
      for (int k = 0; k < NK; ++k) ldsm4(qf[QREG ? k : 0], qs + (warp * 16 + (lane & 15)) * LK + k * 16 + (lane >> 4) * 8);
    }
    if (pg * kPage <= warp_last && pg * kPage + kPage > warp_first) {
      const bf16* kt = ks + (pg & 1) * kBN * LK;
      const bf16* vt = vs + (pg & 1) * kBN * LV;
      float s[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
#pragma unroll
      for (int k = 0; k < NK; ++k) {
        uint32_t qq[4];
        if (!QREG) ldsm4(qq, qs + (warp * 16 + (lane & 15)) * LK + k * 16 + (lane >> 4) * 8);
        const uint32_t* qa = QREG ? qf[QREG ? k : 0] : qq;
#pragma unroll
        for (int j = 0; j < 4; ++j) {                            // 16 keys per load: two n-tiles
          uint32_t b[4];
          ldsm4(b, kt + (j * 16 + (lane & 7) + ((lane >> 4) << 3)) * LK + k * 16 + ((lane >> 3) & 1) * 8);
          mma(s[2 * j], qa, b[0], b[1]);
          mma(s[2 * j + 1], qa, b[2], b[3]);
        }
      }
      // some key of the page is after some row, or before some row's window
      const bool edge = pg * kPage + kPage - 1 > pos0 + t0 + warp * 16 || pg * kPage < warp_full;
      float nm[2] = {mx[0], mx[1]};
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          float x = s[i][e] * f[e >> 1];
          if (KV) {
            const int key = i * 8 + t4 * 2 + (e & 1);
            x *= fs[(pg & 1) * kBN + key];
            if (a.r1) x = fmaf(-r1, lg2(fmaf(r2, (float)((e >> 1 ? phi : plo) - pg * kPage - key), 1.f)), x);      // NaN past the diagonal: masked below
          }
          if (CAP) x = cap2 - __fdividef(2.f * cap2, ex2(x) + 1.f);        // log2(e) * cap * tanh(score / cap)
          if (edge) {
            const int key = pg * kPage + i * 8 + t4 * 2 + (e & 1);
            if (key > (e >> 1 ? phi : plo) || key < (e >> 1 ? khi : klo)) x = -INFINITY;
          }
          s[i][e] = x;
          nm[e >> 1] = fmaxf(nm[e >> 1], x);
        }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        nm[i] = fmaxf(nm[i], __shfl_xor_sync(0xffffffffu, nm[i], 1));
        nm[i] = fmaxf(nm[i], __shfl_xor_sync(0xffffffffu, nm[i], 2));
        const float w = ex2(mx[i] - nm[i]);
        if (nm[i] > mx[i]) {
#pragma unroll
          for (int v = 0; v < NV; ++v) { o[v][2 * i] *= w; o[v][2 * i + 1] *= w; }
          den[i] *= w;
        }
        mx[i] = nm[i];
      }
      // P: bf16 head and remainder, already in A-fragment order
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int q = 0; q < 4; ++q) {                            // a0: row lo, keys 2t..; a1: row hi; a2 / a3: keys + 8
          const int i = 2 * k + (q >> 1), e = (q & 1) * 2;
          float x = ex2(s[i][e] - nm[q & 1]), y = ex2(s[i][e + 1] - nm[q & 1]);
          den[q & 1] += x + y;
          ph[q] = split_head(x, y);
          pl[q] = pack_bf162(x, y);
        }
#pragma unroll
        for (int v = 0; v < NV; v += 2) {
          uint32_t b[4];
          ldsm4t(b, vt + (k * 16 + (lane & 15)) * LV + v * 8 + (lane >> 4) * 8);
          mma(o[v], ph, b[0], b[1]);
          mma(o[v + 1], ph, b[2], b[3]);
          mma(o[v], pl, b[0], b[1]);
          mma(o[v + 1], pl, b[2], b[3]);
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    den[i] += __shfl_xor_sync(0xffffffffu, den[i], 1);
    den[i] += __shfl_xor_sync(0xffffffffu, den[i], 2);
    const int r = rlo + 8 * i;
    if (r >= rows) continue;
    if (a.act) {                                                 // one map: the head is finished here
      const int64_t row = row0 + t0 + r;
      if (a.sink) den[i] += ex2(a.sink[h] * kLog2e - mx[i]);
      const float s = a.oscale * (a.gates ? sigmoid_x(a.gates[row * a.ldg + h]) : 1.f) / den[i];
      const float2* vcs = a.vcs ? a.vcs + row * (a.vdim / 2) : nullptr;
      bf16* out = reinterpret_cast<bf16*>(a.act) + row * a.lda + (int64_t)h * a.vdim;
      const bf16* eg = a.egate ? reinterpret_cast<const bf16*>(a.egate) + row * a.lde + (int64_t)h * a.vdim : nullptr;
#pragma unroll
      for (int v = 0; v < NV; ++v) {
        const int c = v * 8 + t4 * 2;
        if (c >= a.vdim) continue;
        float x = o[v][2 * i] * s, y = o[v][2 * i + 1] * s;
        if (vcs) turn_back(x, y, vcs[c / 2]);
        if (eg) {
          const uint32_t g = *reinterpret_cast<const uint32_t*>(eg + c);
          x *= sigmoid_x(__uint_as_float(g << 16));
          y *= sigmoid_x(__uint_as_float(g & 0xffff0000u));
        }
        *reinterpret_cast<uint32_t*>(out + c) = pack_bf162(x, y);
      }
      continue;
    }
    const int64_t idx = ((int64_t)(row0 + t0 + r) * a.H * a.maps + vh) * a.nsplit;
    float* po = a.part_o + idx * a.vdim;
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int c = v * 8 + t4 * 2;
      if (c < a.vdim) *reinterpret_cast<float2*>(po + c) = make_float2(o[v][2 * i], o[v][2 * i + 1]);
    }
    if (t4 == 0) {
      a.part_ml[idx * 2] = mx[i] * (1.f / kLog2e);
      a.part_ml[idx * 2 + 1] = den[i];
      for (int sp = 1; sp < a.nsplit; ++sp) a.part_ml[(idx + sp) * 2] = -INFINITY;
    }
  }
}

template <int DK, int DV, int MODE>
int flash_launch(const AttnMapsArgs& a, int tiles, int segs, cudaStream_t st) {
  auto kern = maps_flash_kernel<DK, DV, MODE>;
  constexpr size_t smem = flash_smem<DK, DV, MODE>();
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  return (int)cb_launch(kern, dim3((unsigned)tiles, (unsigned)(a.H * a.maps), (unsigned)segs), dim3(kFT), smem, st, a);
}
template <int DK>
int flash_dv(const AttnMapsArgs& a, int tiles, int segs, cudaStream_t st) {
  const bool cap = a.cap > 0.f;
  if (a.kr) return cap ? CB_ERR_SHAPE : flash_launch<DK, DK, SHARED>(a, tiles, segs, st);
#define CB_DV(N) \
  if (a.vdim <= N) return cap ? flash_launch<DK, N, CAPPED>(a, tiles, segs, st) : flash_launch<DK, N, PLAIN>(a, tiles, segs, st)
  CB_DV(32); CB_DV(64); CB_DV(128); CB_DV(256);
#undef CB_DV
  return CB_ERR_SHAPE;
}

// ---- decode -------------------------------------------------------------------------------------
// One CTA per (key split, up to 8 / maps heads of a group, row).  Pages go through a two-stage cp.async ring; scores and
// weighted sums are mma products with the query vectors as rows: eight of the sixteen rows are enough, so the second
// product takes the bf16 heads of the weights in rows 0-7 and their remainders in rows 8-15.
constexpr int kDT = 256;
constexpr int decode_ctas(int dk, int dv, int maps) { return maps == 1 && dk <= 128 && dv <= 128 ? 2 : 1; }    // per SM
// Forms: as described, with norms, turned values and distance penalties (one map), and the same with keys that are their own values.
// _FIXED: bounded scores (AttnMapsArgs.bound); a warp exponentiates its own scores, no maximum crosses the block.
enum DecodeForm : int { BASIC = 0, NORMED = 1, KEYS_ONLY = 2, NORMED_FIXED = 3, KEYS_FIXED = 4 };
constexpr bool keys_only(int form) { return form == KEYS_ONLY || form == KEYS_FIXED; }
constexpr bool fixed_ref(int form) { return form == NORMED_FIXED || form == KEYS_FIXED; }
// staged pages: keys alone leave room for more
constexpr int decode_ring(int form, int dk, int dv) { return keys_only(form) ? 4 : (fixed_ref(form) && dk + dv <= 256 ? 3 : 2); }
template <int DK, int DV, int MAPS, int FORM>
constexpr size_t decode_smem() {
  return sizeof(bf16) * (decode_ring(FORM, DK, DV) * (size_t)kPage * (MAPS * (DK + 8) + (keys_only(FORM) ? 0 : DV + 8)) + MAPS * 8 * (DK + 8) +
                         (fixed_ref(FORM) ? 2 : 1) * 16 * (kPage + 8)) +
         sizeof(float) * ((fixed_ref(FORM) ? 0 : 8 * kPage) + (keys_only(FORM) ? decode_ring(FORM, DK, DV) * kPage : 0));
}
template <int DK, int DV, int MAPS, typename TP, int FORM>
__global__ void __launch_bounds__(kDT, decode_ctas(DK, DV, MAPS)) maps_decode_kernel(const AttnMapsArgs a, int hpc) {
  constexpr bool KV = keys_only(FORM), FIX = fixed_ref(FORM);
  static_assert(FORM == BASIC || MAPS == 1, "one map");
  static_assert(!KV || DK == DV, "values are the keys");
  constexpr int LK = DK + 8, LV = DV + 8, KPAGE = MAPS * kPage * LK, VPAGE = kPage * LV, NP = DV / 16, NPW = (NP + 7) / 8;
  constexpr int ST = decode_ring(FORM, DK, DV), PA = 16 * (kPage + 8);
  extern __shared__ __align__(128) unsigned char smem[];
  bf16* ks = reinterpret_cast<bf16*>(smem);            // [ST][MAPS][kPage][LK]
  bf16* vs = KV ? ks : ks + ST * KPAGE;                // [ST][kPage][LV]
  bf16* qs = KV ? ks + ST * KPAGE : vs + ST * VPAGE;   // [MAPS][8][LK]
  bf16* pa = qs + MAPS * 8 * LK;                       // [16][kPage + 8]: heads, remainders (FIXED: two of them)
  float* ps = reinterpret_cast<float*>(pa + (FIX ? 2 : 1) * PA);   // [8][kPage] scores (not FIXED)
  float* fs = ps + (FIX ? 0 : 8 * kPage);              // [ST][kPage] factors of the keys (KEYS_ONLY)
  __shared__ float w_s[8], own_s, l_s[FIX ? kDT / 32 : 1][8];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g4 = lane >> 2, t4 = lane & 3;
  const int split = blockIdx.x, row = blockIdx.z;
  const int R = a.H / a.G, cpg = (R + hpc - 1) / hpc, g = blockIdx.y / cpg, r0 = (blockIdx.y % cpg) * hpc, nh = min(hpc, R - r0);
  const int nq = nh * MAPS;                            // vector i: head i / MAPS of the CTA, map i % MAPS
  griddep_launch();
  griddep_wait();
  const int pos = a.positions[row], seg = a.row_seg ? a.row_seg[row] : row;
  if (pos < 0) return;
  const int64_t vh0 = (int64_t)row * a.H * MAPS + (int64_t)(g * R + r0) * MAPS;
  const int lo = first_key(a, pos), page0 = lo / kPage, pages = pos / kPage + 1, per = (pages - page0 + a.nsplit - 1) / a.nsplit;
  const int pg0 = page0 + split * per, pg1 = min(pages, pg0 + per);
  if (pg0 >= pages) {
    if (tid < nq) a.part_ml[((vh0 + tid) * a.nsplit + split) * 2] = -INFINITY;
    return;
  }
  const int* bt = a.tables + (int64_t)seg * a.ldbt;
  const int64_t ldk = pool_ldk(a), ldv = pool_ldv(a);
  bf16* K = reinterpret_cast<bf16*>(a.kpool) + (int64_t)g * MAPS * a.dim;
  bf16* V = reinterpret_cast<bf16*>(a.vpool) + (int64_t)g * a.vdim;
  const TP* pr = reinterpret_cast<const TP*>(a.proj) + (int64_t)row * a.ldp;
  const float2* cs = a.cs + (int64_t)row * a.rot_half;
  const TP* v0 = a.v0 ? reinterpret_cast<const TP*>(a.v0) + (int64_t)row * a.ldv0 : nullptr;
  auto load = [&](int pg) {
    const int64_t base = (int64_t)bt[pg] * kPage;
    const int n = pos + 1 - pg * kPage;                // keys of the page that exist
    bf16* kd = ks + (pg % ST) * KPAGE;
    bf16* vd = vs + (pg % ST) * VPAGE;
    for (int e = tid; e < MAPS * kPage * (DK / 8); e += kDT) {
      const int r = e / (MAPS * DK / 8), m = (e / (DK / 8)) % MAPS, c = (e % (DK / 8)) * 8;
      const bool ok = r < n && c < a.dim;
      cp16(kd + (m * kPage + r) * LK + c, ok ? K + (base + r) * ldk + m * a.dim + c : K, ok);
    }
    if (KV) {
      if (tid < kPage / 4) cp16(fs + (pg % ST) * kPage + tid * 4, a.kr + factor_at(a, bt[pg], g) + tid * 4, true);
    } else {
      for (int e = tid; e < kPage * (DV / 8); e += kDT) {
        const int r = e / (DV / 8), c = (e % (DV / 8)) * 8;
        const bool ok = r < n && c < a.vdim;
        cp16(vd + r * LV + c, ok ? V + (base + r) * ldv + c : V, ok);
      }
    }
  };
#pragma unroll
  for (int i = 0; i < ST - 1; ++i) {
    if (pg0 + i < pg1) load(pg0 + i);
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  const bool cap = a.cap > 0.f;
  const float f = a.scale * query_temp(a, pos) * (cap ? 2.f * kLog2e / a.cap : kLog2e), cap2 = a.cap * kLog2e;
  if (FORM == BASIC) {
    for (int e = tid; e < MAPS * 8 * LK; e += kDT) {
      const int m = e / (8 * LK), i = (e / LK) % 8, c = e % LK;
      const bool ok = i < nh && c < a.dim;
      qs[e] = ok ? __float2bfloat16(turned(pr, ((g * R + r0 + i) * MAPS + m) * a.dim + c, c, cs, a.rot_half)) : __float2bfloat16(0.f);
    }
  } else {
    // a warp per query vector, a pair of columns per lane and step; then the norm of the token's own key by the last warp
    auto inverse_rms = [&](const TP* x) {
      float ss = 0.f;
      for (int c = lane * 2; c < a.dim; c += 64) {
        const float u = act_load(x + c), v = act_load(x + c + 1);
        ss = fmaf(u, u, fmaf(v, v, ss));
      }
      return a.norm ? 1.f / sqrtf(warp_sum(ss) / (float)a.dim + a.eps) : 1.f;
    };
    const TP* q = pr + (int64_t)(g * R + r0 + warp) * a.dim;
    const float rq = warp < nh ? inverse_rms(q) : 0.f;
    for (int c = lane * 2; c < LK; c += 64) {
      float x = 0.f, y = 0.f;
      if (warp < nh && c < a.dim) {
        x = act_load(q + c) * rq;
        y = act_load(q + c + 1) * rq;
        if (a.qn) { x *= a.qn[c]; y *= a.qn[c + 1]; }
        if (c >> 1 < a.rot_half) {
          const float2 t = cs[c >> 1];
          const float u = x;
          x = u * t.x - y * t.y;
          y = y * t.x + u * t.y;
        }
      }
      *reinterpret_cast<uint32_t*>(qs + warp * LK + c) = pack_bf162(x, y);
    }
    if (warp == kDT / 32 - 1 && pg1 == pages) {
      const float rk = inverse_rms(pr + a.k_col + (int64_t)g * a.dim);
      if (lane == 0) own_s = rk;
    }
  }
  const float r1 = FORM != BASIC && a.r1 && g4 < nh ? a.r1[g * R + r0 + g4] : 0.f, r2 = FORM != BASIC && a.r1 && g4 < nh ? a.r2[g * R + r0 + g4] : 0.f;
  for (int e = tid; e < (FIX ? 2 : 1) * PA; e += kDT) pa[e] = __float2bfloat16(0.f);
  float o[NPW][2][4];
#pragma unroll
  for (int i = 0; i < NPW; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j) o[i][j][0] = o[i][j][1] = o[i][j][2] = o[i][j][3] = 0.f;
  const float ref = FIX ? a.bound * kLog2e : 0.f;
  float m_run = FIX ? ref : -INFINITY, l_run = 0.f;    // of vector `warp` (FIXED: this lane's part of vector g4)
  for (int pg = pg0; pg < pg1; ++pg) {
    if (FIX) {                                         // one barrier ends the page before and starts this one
      asm volatile("cp.async.wait_group %0;" ::"n"(ST - 2) : "memory");
      __syncthreads();
      if (pg + ST - 1 < pg1) load(pg + ST - 1);
      asm volatile("cp.async.commit_group;" ::: "memory");
    } else {
      if (pg + ST - 1 < pg1) load(pg + ST - 1);
      asm volatile("cp.async.commit_group;" ::: "memory");
      asm volatile("cp.async.wait_group %0;" ::"n"(ST - 1) : "memory");
      __syncthreads();
    }
    bf16* kt = ks + (pg % ST) * KPAGE;
    bf16* vt = vs + (pg % ST) * VPAGE;
    if (pg == pages - 1) {
      // the token's own key and value: into the staged page, and into the pool (CTAs of other heads of the group store
      // the same values)
      const int r = pos % kPage;
      const int64_t slot = (int64_t)bt[pg] * kPage + r;
      if (FORM == BASIC) {
        for (int c = tid; c < MAPS * a.dim; c += kDT) {
          const bf16 x = __float2bfloat16(turned(pr + a.k_col, g * MAPS * a.dim + c, c % a.dim, cs, a.rot_half));
          kt[((c / a.dim) * kPage + r) * LK + c % a.dim] = x;
          K[slot * ldk + c] = x;
        }
        for (int c = tid; c < a.vdim; c += kDT) {
          const int64_t vc = (int64_t)g * a.vdim + c;
          const bf16 x = __float2bfloat16(mixed(act_load(pr + a.v_col + vc), v0 ? act_load(v0 + vc) : 0.f, a));
          vt[r * LV + c] = x;
          V[slot * ldv + c] = x;
        }
      } else {
        const TP* k = pr + a.k_col + (int64_t)g * a.dim;
        const float rk = KV ? 1.f : own_s;
        for (int c = tid * 2; c < a.dim; c += 2 * kDT) {
          float x = act_load(k + c) * rk, y = act_load(k + c + 1) * rk;
          if (!KV && a.kn) { x *= a.kn[c]; y *= a.kn[c + 1]; }
          if (!KV && c >> 1 < a.rot_half) {
            const float2 t = cs[c >> 1];
            const float u = x;
            x = u * t.x - y * t.y;
            y = y * t.x + u * t.y;
          }
          const uint32_t xy = pack_bf162(x, y);
          *reinterpret_cast<uint32_t*>(kt + r * LK + c) = xy;
          *reinterpret_cast<uint32_t*>(K + slot * ldk + c) = xy;
        }
        if (KV) {
          if (tid == 0) fs[(pg % ST) * kPage + r] = a.kr[factor_at(a, bt[pg], g) + r] = own_s;
        } else {
          const float2* vcs = a.vcs + (int64_t)row * (a.vdim / 2);
          for (int c = (kDT - 1 - tid) * 2; c < a.vdim; c += 2 * kDT) {      // first the threads that had no key columns
            const int64_t vc = (int64_t)g * a.vdim + c;
            float x = mixed(act_load(pr + a.v_col + vc), v0 ? act_load(v0 + vc) : 0.f, a);
            float y = mixed(act_load(pr + a.v_col + vc + 1), v0 ? act_load(v0 + vc + 1) : 0.f, a);
            if (a.vcs) {
              const float2 t = vcs[c >> 1];
              const float u = x;
              x = u * t.x - y * t.y;
              y = y * t.x + u * t.y;
            }
            const uint32_t xy = pack_bf162(x, y);
            *reinterpret_cast<uint32_t*>(vt + r * LV + c) = xy;
            *reinterpret_cast<uint32_t*>(V + slot * ldv + c) = xy;
          }
        }
      }
      __syncthreads();
    }
    // scores of keys 8 warp .. 8 warp + 7
#pragma unroll
    for (int m = 0; m < MAPS; ++m) {
      float s[4] = {0.f, 0.f, 0.f, 0.f}, s2[4] = {0.f, 0.f, 0.f, 0.f};
      const bf16* qr = qs + (m * 8 + g4) * LK + t4 * 2;
      const bf16* kr = kt + (m * kPage + warp * 8 + (lane & 7)) * LK + (lane >> 3) * 8;
#pragma unroll
      for (int k = 0; k < DK / 32; ++k) {
        uint32_t b[4];
        ldsm4(b, kr + k * 32);
        const uint32_t a0[4] = {*reinterpret_cast<const uint32_t*>(qr + k * 32), 0u, *reinterpret_cast<const uint32_t*>(qr + k * 32 + 8), 0u};
        const uint32_t a1[4] = {*reinterpret_cast<const uint32_t*>(qr + k * 32 + 16), 0u, *reinterpret_cast<const uint32_t*>(qr + k * 32 + 24), 0u};
        mma(s, a0, b[0], b[1]);
        mma(s2, a1, b[2], b[3]);
      }
      if (FIX) {
        float p[2];
        const int key = warp * 8 + t4 * 2, left = pos - pg * kPage - key;      // distance of the first key
        float2 kf = make_float2(1.f, 1.f);
        if (KV) kf = *reinterpret_cast<const float2*>(fs + (pg % ST) * kPage + key);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float x = fmaf((s[e] + s2[e]) * f, e ? kf.y : kf.x, -ref);
          if (a.r1) x = fmaf(-r1, lg2(fmaf(r2, (float)(left - e), 1.f)), x);
          p[e] = left - e >= 0 && pg * kPage + key + e >= lo ? ex2(x) : 0.f;
        }
        if (g4 < nh) {
          l_run += p[0] + p[1];
          bf16* pw = pa + (pg & 1) * PA + g4 * (kPage + 8) + key;
          *reinterpret_cast<uint32_t*>(pw) = split_head(p[0], p[1]);
          *reinterpret_cast<uint32_t*>(pw + 8 * (kPage + 8)) = pack_bf162(p[0], p[1]);
        }
      } else if (g4 < nh) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float x = (s[e] + s2[e]) * f;
          const int key = warp * 8 + t4 * 2 + e;
          if (KV) x *= fs[(pg % ST) * kPage + key];
          if (cap) x = cap2 - __fdividef(2.f * cap2, ex2(x) + 1.f);
          if (FORM != BASIC && a.r1) x = fmaf(-r1, lg2(fmaf(r2, (float)(pos - pg * kPage - key), 1.f)), x);
          ps[(g4 * MAPS + m) * kPage + key] = pg * kPage + key <= pos && pg * kPage + key >= lo ? x : -INFINITY;
        }
      }
    }
    __syncthreads();
    if (!FIX && warp < nq) {
      const float2 x = *reinterpret_cast<const float2*>(ps + warp * kPage + 2 * lane);
      const float mn = fmaxf(m_run, warp_max(fmaxf(x.x, x.y)));  // finite: a walked page holds a visible key
      float e0 = ex2(x.x - mn), e1 = ex2(x.y - mn);
      const float w = ex2(m_run - mn);
      l_run = l_run * w + warp_sum(e0 + e1);
      m_run = mn;
      *reinterpret_cast<uint32_t*>(pa + warp * (kPage + 8) + 2 * lane) = split_head(e0, e1);
      *reinterpret_cast<uint32_t*>(pa + (8 + warp) * (kPage + 8) + 2 * lane) = pack_bf162(e0, e1);
      if (lane == 0) w_s[warp] = w;
    }
    if (!FIX) __syncthreads();
    const float w = FIX ? 1.f : (g4 < nq ? w_s[g4] : 0.f);
    uint32_t pf[4][4];
#pragma unroll
    for (int k = 0; k < 4; ++k) ldsm4(pf[k], pa + (FIX ? (pg & 1) * PA : 0) + (lane & 15) * (kPage + 8) + k * 16 + (lane >> 4) * 8);
#pragma unroll
    for (int i = 0; i < NPW; ++i) {
      const int cp = warp + 8 * i;
      if (cp >= NP) break;
      if (!FIX) {
#pragma unroll
        for (int j = 0; j < 2; ++j) { o[i][j][0] *= w; o[i][j][1] *= w; o[i][j][2] *= w; o[i][j][3] *= w; }
      }
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        uint32_t b[4];
        ldsm4t(b, vt + (k * 16 + (lane & 15)) * LV + cp * 16 + (lane >> 4) * 8);
        mma(o[i][0], pf[k], b[0], b[1]);
        mma(o[i][1], pf[k], b[2], b[3]);
      }
    }
    if (!FIX) __syncthreads();
  }
  if (FIX) {                                           // denominators: lanes of a vector, then warps; vector `warp` ends up in l_run
    l_run += __shfl_xor_sync(0xffffffffu, l_run, 1);
    l_run += __shfl_xor_sync(0xffffffffu, l_run, 2);
    if (t4 == 0) l_s[warp][g4] = l_run;
    __syncthreads();
    l_run = 0.f;
#pragma unroll
    for (int i = 0; i < kDT / 32; ++i) l_run += l_s[i][warp];
  }
  if (MAPS == 1 && a.act) {                            // the only split: the heads are finished here
    if (warp < nq && lane == 0) w_s[warp] = a.oscale / (l_run + (a.sink ? ex2(a.sink[g * R + r0 + warp] * kLog2e - m_run) : 0.f));
    __syncthreads();
    if (g4 >= nq) return;
    const float inv = w_s[g4];
    const int hc = (g * R + r0 + g4) * a.vdim;
    bf16* out = reinterpret_cast<bf16*>(a.act) + (int64_t)row * a.lda + hc;
    const float2* vcs = FORM != BASIC && !KV && a.vcs ? a.vcs + (int64_t)row * (a.vdim / 2) : nullptr;
    const TP* eg = a.egate ? reinterpret_cast<const TP*>(a.egate) + (int64_t)row * a.lde + hc : nullptr;
#pragma unroll
    for (int i = 0; i < NPW; ++i)
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int c = (warp + 8 * i) * 16 + j * 8 + t4 * 2;
        if (warp + 8 * i >= NP || c >= a.vdim) continue;
        float x = (o[i][j][0] + o[i][j][2]) * inv, y = (o[i][j][1] + o[i][j][3]) * inv;
        if (vcs) turn_back(x, y, vcs[c >> 1]);
        if (eg) { x *= sigmoid_x(act_load(eg + c)); y *= sigmoid_x(act_load(eg + c + 1)); }
        *reinterpret_cast<uint32_t*>(out + c) = pack_bf162(x, y);
      }
    return;
  }
#pragma unroll
  for (int i = 0; i < NPW; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int c = (warp + 8 * i) * 16 + j * 8 + t4 * 2;
      if (warp + 8 * i < NP && g4 < nq && c < a.vdim)
        *reinterpret_cast<float2*>(a.part_o + ((vh0 + g4) * a.nsplit + split) * a.vdim + c) =
            make_float2(o[i][j][0] + o[i][j][2], o[i][j][1] + o[i][j][3]);
    }
  if (warp < nq && lane == 0) {
    float* ml = a.part_ml + ((vh0 + warp) * a.nsplit + split) * 2;
    ml[0] = m_run * (1.f / kLog2e);
    ml[1] = l_run;
  }
}

template <int DK, int DV, int MAPS, typename TP, int FORM>
int decode_form(const AttnMapsArgs& a, int hpc, int rows, cudaStream_t st) {
  constexpr size_t smem = decode_smem<DK, DV, MAPS, FORM>();
  auto kern = maps_decode_kernel<DK, DV, MAPS, TP, FORM>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  const int R = a.H / a.G;
  return (int)cb_launch(kern, dim3((unsigned)a.nsplit, (unsigned)(a.G * ((R + hpc - 1) / hpc)), (unsigned)rows), dim3(kDT), smem, st, a, hpc);
}
template <int DK, int DV, int MAPS, typename TP>
int decode_launch(const AttnMapsArgs& a, int hpc, int rows, cudaStream_t st) {
  if constexpr (MAPS == 1) {
    if (extended(a) && a.bound > 0.f) return decode_form<DK, DV, 1, TP, NORMED_FIXED>(a, hpc, rows, st);
    if (extended(a)) return decode_form<DK, DV, 1, TP, NORMED>(a, hpc, rows, st);
  }
  return decode_form<DK, DV, MAPS, TP, BASIC>(a, hpc, rows, st);
}
template <int DK, int MAPS, typename TP>
int decode_dv(const AttnMapsArgs& a, int hpc, int rows, cudaStream_t st) {
  if constexpr (MAPS == 1) {
    constexpr int D = DK < 64 ? 64 : DK;
    if (a.kr && a.bound > 0.f) return decode_form<D, D, 1, TP, KEYS_FIXED>(a, hpc, rows, st);
    if (a.kr) return decode_form<D, D, 1, TP, KEYS_ONLY>(a, hpc, rows, st);
  }
  if (a.vdim <= 64) return decode_launch<DK, 64, MAPS, TP>(a, hpc, rows, st);
  if (a.vdim <= 128) return decode_launch<DK, 128, MAPS, TP>(a, hpc, rows, st);
  return decode_launch<DK, 256, MAPS, TP>(a, hpc, rows, st);
}
template <int MAPS, typename TP>
int decode_dk(const AttnMapsArgs& a, int hpc, int rows, cudaStream_t st) {
  if (a.dim <= 32) return decode_dv<32, MAPS, TP>(a, hpc, rows, st);
  if (a.dim <= 64) return decode_dv<64, MAPS, TP>(a, hpc, rows, st);
  if (a.dim <= 128) return decode_dv<128, MAPS, TP>(a, hpc, rows, st);
  return decode_dv<256, MAPS, TP>(a, hpc, rows, st);
}

}  // namespace

// Whether the prompt / decode kernels of this file take a head of these sizes (16-byte rows; values in 8-column pieces).
CB_EXPORT int cb_attn_maps_tc_ok(int64_t G, int64_t maps, int64_t dim, int64_t vdim) {
  return dim % 8 == 0 && vdim % 8 == 0 && dim <= 256 && vdim <= 256 && dim >= 8 && vdim >= 8 && maps >= 1 && maps <= 2 && G >= 1;
}

// Prompt attention: `segs` segments (seg_row, seg_pos, one block table each) of at most `max_rows` rows; bf16 projection
// rows, keys and values appended before.
CB_EXPORT int cb_attn_maps_flash(const void* args, int64_t segs, int64_t max_rows, void* stream) {
  if (!args || segs < 1 || segs > 65535 || max_rows < 1) return CB_ERR_ARG;
  const AttnMapsArgs& a = *(const AttnMapsArgs*)args;
  if (!a.proj || !a.kpool || !a.vpool || !a.tables || !a.seg_row || !a.seg_pos || a.H < 1 || a.G < 1 || a.H % a.G) return CB_ERR_ARG;
  if (a.act ? a.maps != 1 || a.lda % 2 || a.lde % 2 : !a.part_o || !a.part_ml) return CB_ERR_ARG;
  if ((a.r1 && !a.kr) || (a.kr && (a.maps != 1 || a.dim != a.vdim || a.vcs || a.sink || a.egate))) return CB_ERR_SHAPE;
  if (!cb_attn_maps_tc_ok(a.G, a.maps, a.dim, a.vdim) || a.ldp % 8 || a.k_col % 8 || a.v_col % 8 || a.ldk % 8 || a.ldv % 8) return CB_ERR_SHAPE;
  const int tiles = (int)((max_rows + kBM - 1) / kBM);
  cudaStream_t st = (cudaStream_t)stream;
  if (a.dim <= 32) return flash_dv<32>(a, tiles, (int)segs, st);
  if (a.dim <= 64) return flash_dv<64>(a, tiles, (int)segs, st);
  if (a.dim <= 128) return flash_dv<128>(a, tiles, (int)segs, st);
  return flash_dv<256>(a, tiles, (int)segs, st);
}

// Decode attention of `rows` single tokens (appends their keys and values): splits of every row into part_o / part_ml, or with
// one split of one map the finished heads into act.
CB_EXPORT int cb_attn_maps_decode(const void* args, int64_t rows, int64_t p_f32, void* stream) {
  if (!args || rows < 1 || rows > 65535) return CB_ERR_ARG;
  const AttnMapsArgs& a = *(const AttnMapsArgs*)args;
  if (a.act ? a.maps != 1 || a.nsplit != 1 || a.lda % 2 : !a.part_o || !a.part_ml) return CB_ERR_ARG;
  if (!a.proj || !a.kpool || !a.vpool || !a.tables || !a.positions || a.H < 1 || a.G < 1 || a.H % a.G ||
      a.nsplit < 1 || a.nsplit > 64 || 2 * a.rot_half > a.dim || (a.rot_half && !a.cs) || !a.r1 != !a.r2)
    return CB_ERR_ARG;
  if (a.bound > kMaxBound || (a.bound > 0.f && a.cap > 0.f)) return CB_ERR_ARG;
  if (extended(a) && (a.maps != 1 || (a.kr && (a.dim != a.vdim || a.vcs)))) return CB_ERR_SHAPE;
  if (!cb_attn_maps_tc_ok(a.G, a.maps, a.dim, a.vdim) || a.ldk % 8 || a.ldv % 8) return CB_ERR_SHAPE;
  cudaStream_t st = (cudaStream_t)stream;
  const int R = a.H / a.G;
  int hpc = 8 / a.maps;                                  // heads per CTA: at most 8 query vectors
  if (hpc > R) hpc = R;
  if (a.maps == 1) return p_f32 ? decode_dk<1, float>(a, hpc, (int)rows, st) : decode_dk<1, bf16>(a, hpc, (int)rows, st);
  return p_f32 ? decode_dk<2, float>(a, hpc, (int)rows, st) : decode_dk<2, bf16>(a, hpc, (int)rows, st);
}
