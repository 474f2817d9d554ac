// Prompt attention with several score maps per head (attn_maps.cuh) on the 5th-generation tensor cores.
//
// One CTA owns 128 consecutive query rows of one (head, map) of a segment and walks the sequence's pages (64 keys) up
// to the diagonal, with the division of labour of attn_tc.cu: a TMA warp fills rings of key and value pages, two
// threads issue S_j = Q K_j^T (Q in tensor memory) and O += P_j V_j, eight warps do the softmax, two threads per row.
// What differs: key and value sizes are independent; scores take a per-row query temperature and an optional cap
// (cap * tanh(score / cap), evaluated through one exponential); the weights keep 32-bit meaning across the second
// product, P = bf16 head + bf16 remainder, two products per page; the result leaves as unnormalised fp32 sums with
// (reference maximum, denominator), which maps_finish_kernel combines across the maps.
//
// SHARED: the keys are their own values.  One ring of pages serves both products (K-major for the scores, MN-major for the
// sums), released by the second; a key's factor comes with its page, and the penalty r1 ln(1 + r2 distance) is taken off.
//
// With a cap the scores are bounded, so the reference maximum is the cap itself (when 2^-2cap is far from underflow):
// no row maximum, no exchange between the halves of a row, no rescale.  The same where norms of queries and keys bound the
// scores (FIXED, SHARED_FIXED: a distance penalty is never negative, and a token's own key has none).  Otherwise the reference is raised lazily as in
// attn_tc.cu.  Waits are bounded by 2 s and report through the status word; TMEM is freed on every path.
#include "attn_maps.cuh"
#include "sm100.cuh"

namespace {
using namespace sm100;

constexpr int kBQ = 128, kBKV = 64, kThreads = 352;
constexpr float kLog2e = 1.4426950408889634f;
enum Mode : int { PLAIN = 0, CAP = 1, CAP_FIXED = 2, SHARED = 3, FIXED = 4, SHARED_FIXED = 5 };

__device__ __forceinline__ uint64_t now_ns() {
  uint64_t t;
  asm volatile("mov.u64 %0, %globaltimer;" : "=l"(t));
  return t;
}
__device__ __forceinline__ bool wait_bar(uint64_t* bar, uint32_t parity, volatile int* abort_flag) {
  if (mbar_try(bar, parity)) return true;
  const uint64_t t0 = now_ns();
  for (;;) {
    for (int i = 0; i < 128; ++i)
      if (mbar_try(bar, parity)) return true;
    if (*abort_flag) return false;
    if (now_ns() - t0 > 2000000000ull) return false;
  }
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// Buffers of scores and of weights.  Heads up to 128 keep one of each: two CTAs then fit an SM and cover each other's waits (a
// tile's scores are computed while the softmax of the tile before it, already in registers, goes on).
constexpr int buffers(int dk, int dv) { return dk <= 128 && dv <= 128 ? 1 : 2; }
template <int DK, int DV, int MODE, int STAGES>
__global__ void __launch_bounds__(kThreads, 3 - buffers(DK, DV))
maps_tc_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV, const AttnMapsArgs a, int* status) {
  constexpr bool KV = MODE == SHARED || MODE == SHARED_FIXED, FIX = MODE == FIXED || MODE == SHARED_FIXED;
  static_assert(!KV || DK == DV, "values are the keys");
  constexpr int NK = DK / 64, NV = DV / 64;           // 64-element (128-byte) chunks
  constexpr int K_BYTES = kBKV * DK * 2, V_BYTES = KV ? 0 : kBKV * DV * 2, P_BYTES = kBQ * kBKV * 2;
  constexpr int KC = kBKV * 128;                      // bytes of one chunk block of a page
  constexpr int NB = buffers(DK, DV);
  constexpr uint32_t TMEM_COLS = NB * kBKV + DV + DK / 2 <= 256 ? 256 : 512;
  static_assert(NB * kBKV + DV + DK / 2 <= 512 && (NB == 2 || TMEM_COLS == 256), "tensor memory");
  constexpr uint32_t IDESC_S = umma_idesc(kBQ, kBKV, 1, 1);
  constexpr uint32_t IDESC_O = umma_idesc(kBQ, DV, 1, 1) | (1u << 16);     // B operand MN-major
  extern __shared__ __align__(1024) unsigned char smem_raw[];
  unsigned char* base = reinterpret_cast<unsigned char*>(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  unsigned char* Ks = base;                           // [STAGES][K_BYTES]
  unsigned char* Vs = Ks + STAGES * K_BYTES;          // [STAGES][V_BYTES]
  unsigned char* Ps = Vs + STAGES * V_BYTES;          // [NB][head | remainder]
  __shared__ uint64_t q_full, k_full[STAGES], v_full[STAGES], k_free[STAGES], v_free[STAGES], s_full[NB], s_free[NB], p_full[NB], p_free[NB],
      o_full, pair_bar[4];
  __shared__ __align__(16) float factor_s[KV ? STAGES : 1][kBKV];
  __shared__ float xch[2][2][kBQ];                    // [tile parity][column half][row]: maxima of half rows
  __shared__ uint32_t tmem_base_s;
  __shared__ int abort_s;
  volatile int* abort_flag = &abort_s;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int qt = (int)gridDim.x - 1 - (int)blockIdx.x, vh = blockIdx.y, seg = blockIdx.z;    // long tiles first
  const int h = vh / a.maps, kh = h / (a.H / a.G), kmap = kh * a.maps + vh % a.maps;
  griddep_launch();
  griddep_wait();
  const int seg0 = a.seg_row[seg], n = a.seg_row[seg + 1] - seg0, pos0 = a.seg_pos[seg];
  const int row0 = qt * kBQ;
  if (row0 >= n) return;                              // the whole CTA, before anything is allocated
  const int page0 = first_key(a, pos0 + row0) / kBKV;             // pages before it are outside every row's window
  const int n_tiles = (pos0 + min(n, row0 + kBQ) - 1) / kBKV + 1 - page0;

  if (threadIdx.x == 0) {
    mbar_init(&q_full, 8);
    mbar_init(&o_full, 1);
    for (int i = 0; i < STAGES; ++i) {
      mbar_init(&k_full[i], 1); mbar_init(&v_full[i], 1); mbar_init(&k_free[i], 1); mbar_init(&v_free[i], 1);
    }
    for (int i = 0; i < NB; ++i) {
      mbar_init(&s_full[i], 1); mbar_init(&s_free[i], 8); mbar_init(&p_full[i], 8); mbar_init(&p_free[i], 1);
    }
    for (int i = 0; i < 4; ++i) mbar_init(&pair_bar[i], 64);
    abort_s = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
  }
  if (warp == 1) {
    tmem_alloc(&tmem_base_s, TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = tmem_base_s;
  const uint32_t tmem_o = tmem_base + NB * kBKV;      // S [NB] | O | Q
  const uint32_t tmem_q = tmem_o + DV;

  if (warp == 0) {
    // ------------------------------------ TMA producer ------------------------------------------
    if (lane == 0) {
      const int* bt = a.tables + (int64_t)seg * a.ldbt;
      for (int j = 0; j < n_tiles && !*abort_flag; ++j) {
        const int s = j % STAGES;
        const uint32_t ph = (j / STAGES) & 1;
        const int slot0 = bt[page0 + j] * kBKV;
        if (!wait_bar(&k_free[s], ph ^ 1, abort_flag)) { atomicCAS(status, 0, 81); abort_s = 1; break; }
        mbar_expect_tx(&k_full[s], K_BYTES + (KV ? kBKV * 4 : 0));
        for (int c = 0; c < NK; ++c) tma_load_2d(Ks + s * K_BYTES + c * KC, &tmK, &k_full[s], kmap * DK + c * 64, slot0);
        if (KV) {
          bulk_load(factor_s[s], a.kr + factor_at(a, bt[page0 + j], kh), kBKV * 4, &k_full[s]);
          continue;
        }
        if (!wait_bar(&v_free[s], ph ^ 1, abort_flag)) { atomicCAS(status, 0, 82); abort_s = 1; break; }
        mbar_expect_tx(&v_full[s], V_BYTES);
        for (int c = 0; c < NV; ++c) tma_load_2d(Vs + s * V_BYTES + c * KC, &tmV, &v_full[s], kh * DV + c * 64, slot0);
      }
    }
  } else if (warp == 1) {
    // ------------------------------------ MMA issuer: S_j = Q K_j^T -----------------------------
    if (lane == 0) {
      const bool ok = wait_bar(&q_full, 0, abort_flag);
      if (!ok) { atomicCAS(status, 0, 83); abort_s = 1; }
      tc_fence_after();
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int s = j % STAGES, sb = j % NB;
        if (!wait_bar(&k_full[s], (j / STAGES) & 1, abort_flag)) { atomicCAS(status, 0, 84); abort_s = 1; break; }
        if (!wait_bar(&s_free[sb], ((j / NB) & 1) ^ 1, abort_flag)) { atomicCAS(status, 0, 85); abort_s = 1; break; }
        tc_fence_after();
#pragma unroll
        for (int c = 0; c < NK; ++c) {
          const uint64_t kd = umma_desc_sw128(Ks + s * K_BYTES + c * KC);
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_f16_ta(tmem_base + sb * kBKV, tmem_q + c * 32 + k * 8, kd + 2 * k, IDESC_S, (c | k) != 0);
        }
        if (!KV) umma_commit(&k_free[s]);
        umma_commit(&s_full[sb]);
      }
    }
  } else if (warp == 10) {
    // ------------------------------------ MMA issuer: O += P_j V_j ------------------------------
    if (lane == 0) {
      bool ok = true;
      for (int j = 0; j < n_tiles; ++j) {
        const int s = j % STAGES, sb = j % NB;
        if (!wait_bar(&p_full[sb], (j / NB) & 1, abort_flag)) { atomicCAS(status, 0, 86); abort_s = 1; ok = false; break; }
        if (!wait_bar(KV ? &k_full[s] : &v_full[s], (j / STAGES) & 1, abort_flag)) { atomicCAS(status, 0, 87); abort_s = 1; ok = false; break; }
        tc_fence_after();
        const uint64_t pd = umma_desc_sw128(Ps + sb * 2 * P_BYTES), rd = umma_desc_sw128(Ps + sb * 2 * P_BYTES + P_BYTES);
        const uint64_t vd = umma_desc_mn_sw128(KV ? Ks + s * K_BYTES : Vs + s * V_BYTES, KC);
#pragma unroll
        for (int k = 0; k < 4; ++k)      // 16 keys per instruction: +32 bytes along P's rows, +16 rows of V
          umma_f16(tmem_o, pd + 2 * k, vd + (uint64_t)(k * 16 * 128 >> 4), IDESC_O, (j | k) != 0);
#pragma unroll
        for (int k = 0; k < 4; ++k) umma_f16(tmem_o, rd + 2 * k, vd + (uint64_t)(k * 16 * 128 >> 4), IDESC_O, 1);
        umma_commit(KV ? &k_free[s] : &v_free[s]);
        umma_commit(&p_free[sb]);
      }
      if (ok) umma_commit(&o_full);
    }
  } else {
    // ------------------------------------ softmax + epilogue ------------------------------------
    const int q = warp & 3, hf = (warp - 2) >> 2;      // TMEM lane quadrant, half of the row's columns
    const int r = q * 32 + lane;
    const int t = row0 + r, pos = pos0 + t;
    const uint32_t lane_base = (uint32_t)(q * 32) << 16;
    {
      const bf16* qrow = reinterpret_cast<const bf16*>(a.proj) + (int64_t)(seg0 + min(t, n - 1)) * a.ldp + (int64_t)vh * DK;
#pragma unroll 1
      for (int i = hf; i < NK; i += 2) {
        uint32_t w[32];
#pragma unroll
        for (int v = 0; v < 8; ++v) {
          const uint4 x = *reinterpret_cast<const uint4*>(qrow + i * 64 + v * 8);
          w[4 * v] = x.x; w[4 * v + 1] = x.y; w[4 * v + 2] = x.z; w[4 * v + 3] = x.w;
        }
        tmem_st32(tmem_q + lane_base + i * 32, w);
      }
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&q_full);
    }
    // score -> log2 units; with a cap first to the exponent of exp(2 score / cap)
    const float f = a.scale * query_temp(a, min(pos, pos0 + n - 1)) * (MODE == PLAIN || KV || FIX ? kLog2e : 2.f * kLog2e / a.cap);
    const float r1 = KV && a.r1 ? a.r1[h] : 0.f, r2 = KV && a.r1 ? a.r2[h] : 0.f;
    const float cap2 = a.cap * kLog2e;
    const int key_lo = first_key(a, pos), full_lo = first_key(a, pos0 + row0 + kBQ - 1);
    float m_ref = MODE == CAP_FIXED ? cap2 : (FIX ? a.bound * kLog2e : -INFINITY), l = 0.f;
    bool ok = true;
    uint32_t xph = 0;
    for (int j = 0; j < n_tiles; ++j) {
      const int sb = j % NB, xb = j & 1;
      if (!wait_bar(&s_full[sb], (j / NB) & 1, abort_flag)) { if (lane == 0) { atomicCAS(status, 0, 88); abort_s = 1; } ok = false; break; }
      tc_fence_after();
      uint32_t sv[32];
      tmem_ld32(tmem_base + lane_base + sb * kBKV + hf * 32, sv);
      tmem_ld_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&s_free[sb]);
      const int page = (page0 + j) * kBKV, key0 = page + hf * 32;
      const bool edge = page + kBKV - 1 > pos0 + row0 || page < full_lo;     // the page touches the diagonal or a window's start
      if (MODE == CAP_FIXED) {
        // 2^(log2e (cap tanh - cap)) = 2^(-2 cap log2e / (exp(2 s / cap) + 1))
#pragma unroll
        for (int c = 0; c < 32; ++c) sv[c] = __float_as_uint(ex2(-2.f * cap2 * rcp(ex2(__uint_as_float(sv[c]) * f) + 1.f)));
        if (edge) {
#pragma unroll
          for (int c = 0; c < 32; ++c)
            if (key0 + c > pos || key0 + c < key_lo) sv[c] = 0u;
        }
      } else {
        if (MODE == CAP) {
#pragma unroll
          for (int c = 0; c < 32; ++c) sv[c] = __float_as_uint(cap2 - 2.f * cap2 * rcp(ex2(__uint_as_float(sv[c]) * f) + 1.f));
        }
        if (KV) {
          // the factors of this page have landed: its scores were computed behind the same barrier
          if (!wait_bar(&k_full[j % STAGES], (j / STAGES) & 1, abort_flag)) { if (lane == 0) { atomicCAS(status, 0, 94); abort_s = 1; } ok = false; break; }
          const float4* kf = reinterpret_cast<const float4*>(factor_s[j % STAGES] + hf * 32);
          const float far = fmaf(r2, (float)(pos - key0), 1.f);
#pragma unroll
          for (int c4 = 0; c4 < 8; ++c4) {
            const float4 k4 = kf[c4];
            const float kk[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              float x = MODE == SHARED_FIXED ? fmaf(__uint_as_float(sv[c4 * 4 + e]) * f, kk[e], -m_ref) : __uint_as_float(sv[c4 * 4 + e]) * f * kk[e];
              if (a.r1) x = fmaf(-r1, lg2(fmaf(-r2, (float)(c4 * 4 + e), far)), x);      // NaN past the diagonal: masked below
              sv[c4 * 4 + e] = __float_as_uint(x);
            }
          }
        }
        if (FIX) {
#pragma unroll
          for (int c = 0; c < 32; ++c) sv[c] = __float_as_uint(ex2(KV ? __uint_as_float(sv[c]) : fmaf(__uint_as_float(sv[c]), f, -m_ref)));
          if (edge) {
#pragma unroll
            for (int c = 0; c < 32; ++c)
              if (key0 + c > pos || key0 + c < key_lo) sv[c] = 0u;
          }
        } else {
        if (edge) {
#pragma unroll
          for (int c = 0; c < 32; ++c)
            if (key0 + c > pos || key0 + c < key_lo) sv[c] = 0xff800000u;        // -inf
        }
        float mx = __uint_as_float(sv[0]);
#pragma unroll
        for (int c = 1; c < 32; ++c) mx = fmaxf(mx, __uint_as_float(sv[c]));
        if (MODE == PLAIN) mx *= f;                    // f > 0: the largest score is the largest product
        xch[xb][hf][r] = mx;
        mbar_arrive(&pair_bar[q]);
        if (!wait_bar(&pair_bar[q], xph, abort_flag)) { if (lane == 0) { atomicCAS(status, 0, 92); abort_s = 1; } ok = false; break; }
        xph ^= 1;
        mx = fmaxf(kNoKey, fmaxf(xch[xb][0][r], xch[xb][1][r]));   // finite: with a window a page may hold no key of a row
        if (j == 0) {
          m_ref = mx;
        } else if (__any_sync(0xffffffffu, mx > m_ref + 8.f)) {
          // every product that wrote O has to be complete before its rows are rescaled
          if (!wait_bar(&p_free[(j - 1) % NB], ((j - 1) / NB) & 1, abort_flag)) {
            if (lane == 0) { atomicCAS(status, 0, 89); abort_s = 1; }
            ok = false;
            break;
          }
          tc_fence_after();
          const float m_new = fmaxf(m_ref, mx), w = ex2(m_ref - m_new);
          m_ref = m_new;
          l *= w;
#pragma unroll 1
          for (int c0 = hf * (DV / 2); c0 < (hf + 1) * (DV / 2); c0 += 32) {
            uint32_t o[32];
            tmem_ld32(tmem_o + lane_base + c0, o);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * w);
            tmem_st32(tmem_o + lane_base + c0, o);
          }
          tmem_st_wait();
          tc_fence_before();
        }
#pragma unroll
        for (int c = 0; c < 32; ++c)
          sv[c] = __float_as_uint(ex2(MODE == PLAIN ? fmaf(__uint_as_float(sv[c]), f, -m_ref) : __uint_as_float(sv[c]) - m_ref));
        }
      }
      // head and remainder of the weights
      uint32_t ph[16], pr[16];
      float l0 = 0.f, l1 = 0.f;
#pragma unroll
      for (int c = 0; c < 16; ++c) {
        float x = __uint_as_float(sv[2 * c]), y = __uint_as_float(sv[2 * c + 1]);
        l0 += x; l1 += y;
        ph[c] = pack_bf162(x, y);
        x -= __uint_as_float(ph[c] << 16);
        y -= __uint_as_float(ph[c] & 0xffff0000u);
        pr[c] = pack_bf162(x, y);
      }
      l += l0 + l1;
      if (j >= NB && !wait_bar(&p_free[sb], ((j - NB) / NB) & 1, abort_flag)) {   // the product before has read this buffer
        if (lane == 0) { atomicCAS(status, 0, 90); abort_s = 1; }
        ok = false;
        break;
      }
      unsigned char* prow = Ps + sb * 2 * P_BYTES + r * 128;
#pragma unroll
      for (int c = 0; c < 4; ++c) {                    // 16-byte chunk c of row r lives at chunk c ^ (r % 8)
        const int at = ((hf * 4 + c) ^ (r & 7)) << 4;
        *reinterpret_cast<uint4*>(prow + at) = make_uint4(ph[4 * c], ph[4 * c + 1], ph[4 * c + 2], ph[4 * c + 3]);
        *reinterpret_cast<uint4*>(prow + P_BYTES + at) = make_uint4(pr[4 * c], pr[4 * c + 1], pr[4 * c + 2], pr[4 * c + 3]);
      }
      fence_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[sb]);
    }
    if (ok && !wait_bar(&o_full, 0, abort_flag)) { if (lane == 0) { atomicCAS(status, 0, 91); abort_s = 1; } ok = false; }
    if (ok) {                                          // the halves of a row add their sums through the idle P buffer
      float* lx = reinterpret_cast<float*>(Ps);
      lx[hf * kBQ + r] = l;
      mbar_arrive(&pair_bar[q]);
      if (!wait_bar(&pair_bar[q], xph, abort_flag)) { if (lane == 0) { atomicCAS(status, 0, 93); abort_s = 1; } ok = false; }
      else l = lx[r] + lx[kBQ + r];
    }
    if (ok && a.act) {                                 // one map: the head is finished here
      tc_fence_after();
      const int64_t row = seg0 + t;
      if (a.sink) l += ex2(a.sink[h] * kLog2e - m_ref);
      const float s = t < n ? a.oscale * (a.gates ? sigmoid_x(a.gates[row * a.ldg + h]) : 1.f) / l : 0.f;
      const float2* vcs = !KV && a.vcs ? a.vcs + row * (DV / 2) : nullptr;
      const bf16* eg = a.egate ? reinterpret_cast<const bf16*>(a.egate) + row * a.lde + (int64_t)h * DV : nullptr;
      bf16* op = reinterpret_cast<bf16*>(a.act) + row * a.lda + (int64_t)h * DV;
#pragma unroll 1
      for (int c0 = hf * (DV / 2); c0 < (hf + 1) * (DV / 2); c0 += 32) {
        uint32_t o[32];
        tmem_ld32(tmem_o + lane_base + c0, o);         // warp-collective: rows beyond the segment load too
        tmem_ld_wait();
        if (t < n) {
#pragma unroll
          for (int v = 0; v < 4; ++v) {
            float x[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) x[e] = __uint_as_float(o[8 * v + e]) * s;
            if (vcs) {
#pragma unroll
              for (int e = 0; e < 8; e += 4) {
                const float4 t2 = *reinterpret_cast<const float4*>(vcs + (c0 + v * 8 + e) / 2);
                turn_back(x[e], x[e + 1], make_float2(t2.x, t2.y));
                turn_back(x[e + 2], x[e + 3], make_float2(t2.z, t2.w));
              }
            }
            if (eg) {
              float g[8];
              bf16x8_to_float(*reinterpret_cast<const uint4*>(eg + c0 + v * 8), g);
#pragma unroll
              for (int e = 0; e < 8; ++e) x[e] *= sigmoid_x(g[e]);
            }
            *reinterpret_cast<uint4*>(op + c0 + v * 8) = float_to_bf16x8(x);
          }
        }
      }
    } else if (ok) {
      tc_fence_after();
      const int64_t idx = ((int64_t)(seg0 + t) * a.H * a.maps + vh) * a.nsplit;
      float* op = a.part_o + idx * DV;
#pragma unroll 1
      for (int c0 = hf * (DV / 2); c0 < (hf + 1) * (DV / 2); c0 += 32) {
        uint32_t o[32];
        tmem_ld32(tmem_o + lane_base + c0, o);         // warp-collective: rows beyond the segment load too
        tmem_ld_wait();
        if (t < n) {
#pragma unroll
          for (int v = 0; v < 8; ++v)
            *reinterpret_cast<uint4*>(op + c0 + v * 4) = make_uint4(o[4 * v], o[4 * v + 1], o[4 * v + 2], o[4 * v + 3]);
        }
      }
      if (t < n && hf == 0) {
        a.part_ml[idx * 2] = m_ref * (1.f / kLog2e);
        a.part_ml[idx * 2 + 1] = l;
        for (int s = 1; s < a.nsplit; ++s) a.part_ml[(idx + s) * 2] = -INFINITY;
      }
    }
  }
  // ------------------------------------ teardown --------------------------------------------------
  tc_fence_before();
  __syncthreads();
  if (abort_s) {  // give copies still in flight time to land before the shared memory is released
    const uint64_t t0 = now_ns();
    while (now_ns() - t0 < 2000000ull) __nanosleep(1000);
  }
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, TMEM_COLS);
  }
}

template <int DK, int DV, int MODE>
int launch_tc(const CUtensorMap& tmK, const CUtensorMap& tmV, const AttnMapsArgs& a, int tiles, int segs, int* status, cudaStream_t st) {
  constexpr int NB = buffers(DK, DV), COLS = MODE == SHARED || MODE == SHARED_FIXED ? DK : DK + DV, STAGES = COLS > (NB == 1 ? 192 : 384) ? 2 : 3;
  const size_t smem = (size_t)STAGES * kBKV * COLS * 2 + 2 * NB * (size_t)kBQ * kBKV * 2 + 1024;
  auto kern = maps_tc_kernel<DK, DV, MODE, STAGES>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  const dim3 grid((unsigned)tiles, (unsigned)(a.H * a.maps), (unsigned)segs);
  return (int)cb_launch(kern, grid, dim3(kThreads), smem, st, tmK, tmV, a, status);
}
template <int DK, int DV>
int mode_tc(const CUtensorMap& tmK, const CUtensorMap& tmV, const AttnMapsArgs& a, int tiles, int segs, int* status, cudaStream_t st) {
  if constexpr (DK == DV) {
    if (a.kr && a.bound > 0.f) return launch_tc<DK, DV, SHARED_FIXED>(tmK, tmK, a, tiles, segs, status, st);
    if (a.kr) return launch_tc<DK, DV, SHARED>(tmK, tmK, a, tiles, segs, status, st);
  }
  if (!(a.cap > 0.f) && a.bound > 0.f) return launch_tc<DK, DV, FIXED>(tmK, tmV, a, tiles, segs, status, st);
  if (!(a.cap > 0.f)) return launch_tc<DK, DV, PLAIN>(tmK, tmV, a, tiles, segs, status, st);
  // 2^(-2 cap log2e) well inside the range of fp32 and of a bf16 remainder 2^-16 below it
  if (a.cap <= 30.f) return launch_tc<DK, DV, CAP_FIXED>(tmK, tmV, a, tiles, segs, status, st);
  return launch_tc<DK, DV, CAP>(tmK, tmV, a, tiles, segs, status, st);
}

}  // namespace

// Whether cb_attn_maps_flash_tc takes these head sizes.
CB_EXPORT int cb_attn_maps_flash_tc_ok(int64_t dim, int64_t vdim) {
  return (dim == 64 || dim == 128 || dim == 192 || dim == 256) && (vdim == 64 || vdim == 128 || vdim == 256 || (vdim == 192 && dim == 192));
}

// Prompt attention of `segs` segments of at most `max_rows` rows on tcgen05; arguments as for cb_attn_maps_flash.
// `slots`: rows of the pools.
CB_EXPORT int cb_attn_maps_flash_tc(const void* args, int64_t segs, int64_t max_rows, int64_t slots, void* status, void* stream) {
  if (!args || segs < 1 || segs > 65535 || max_rows < 1 || !status) return CB_ERR_ARG;
  const AttnMapsArgs& a = *(const AttnMapsArgs*)args;
  if (!a.proj || !a.kpool || !a.vpool || !a.tables || !a.seg_row || !a.seg_pos || a.H < 1 || a.G < 1 || a.H % a.G || a.maps < 1) return CB_ERR_ARG;
  if (a.act ? a.maps != 1 || a.lda % 8 || ((uintptr_t)a.act & 15) || a.lde % 8 || ((uintptr_t)a.egate & 15) : !a.part_o || !a.part_ml)
    return CB_ERR_ARG;
  if ((a.r1 && !a.kr) || (a.kr && (a.maps != 1 || a.dim != a.vdim || a.vcs || a.sink || a.egate || a.cap > 0.f || !a.act))) return CB_ERR_SHAPE;
  if ((a.vcs && (((uintptr_t)a.vcs & 15) || !a.act)) || a.bound > kMaxBound) return CB_ERR_ARG;
  if (!cb_attn_maps_flash_tc_ok(a.dim, a.vdim) || !(a.scale > 0.f) || a.ldp % 8 || a.ldk % 8 || a.ldv % 8 || ((uintptr_t)a.proj & 15)) return CB_ERR_SHAPE;
  CUtensorMap tmK, tmV;
  const uint64_t kw = (uint64_t)a.G * a.maps * a.dim, vw = (uint64_t)a.G * a.vdim;
  int rc = cb_make_tmap_2d(&tmK, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.kpool, (uint64_t)slots, kw, (uint64_t)pool_ldk(a), kBKV, 64);
  if (rc) return rc;
  rc = a.kr ? 0 : cb_make_tmap_2d(&tmV, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.vpool, (uint64_t)slots, vw, (uint64_t)pool_ldv(a), kBKV, 64);
  if (rc) return rc;
  const int tiles = (int)((max_rows + kBQ - 1) / kBQ);
  int* st_word = (int*)status;
  cudaStream_t st = (cudaStream_t)stream;
#define CB_TC(K, V) \
  if (a.dim == K && a.vdim == V) return mode_tc<K, V>(tmK, tmV, a, tiles, (int)segs, st_word, st)
  CB_TC(64, 64); CB_TC(64, 128); CB_TC(64, 256); CB_TC(128, 64); CB_TC(128, 128); CB_TC(128, 256); CB_TC(192, 64); CB_TC(192, 128); CB_TC(192, 192); CB_TC(192, 256); CB_TC(256, 64); CB_TC(256, 128);
  CB_TC(256, 256);
#undef CB_TC
  return CB_ERR_SHAPE;
}
