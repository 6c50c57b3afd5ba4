// Prefill form of latent attention on the 5th-generation tensor cores (same arguments as latent_prefill.cu, head widths of 64
// or 128): a CTA owns 256 query rows of one head as two tiles of 128.
//
//   warps 0-3, 4-7 : softmax of one tile each; a thread owns a row (= a TMEM lane), so maxima and sums need no shuffles
//   warp 8         : TMA producer (queries once; rings of key and value tiles of 64 keys)
//   warp 9         : MMA issuer
// Tensor memory holds, per tile, two 64-column score buffers and the output accumulator; the 16-bit weights overwrite the
// scores they came from and are the A operand of the value product straight from tensor memory.  All shared-memory operands
// are K-major with the 128-byte swizzle: queries and keys as they lie in memory (the rotated key part is read from the
// gathered latent row, so it exists once and not per head), values because the expansion GEMM wrote them transposed.  While
// a tile's softmax runs, the other tile's products and the next scores occupy the tensor cores.  The accumulator is rescaled
// only when a row's maximum has grown by more than 2^8; until then the weights are taken against the older maximum (exact,
// the sums use the same reference).
#include "latent_segs.cuh"
#include "sm100.cuh"
#include "tmap.cuh"

using namespace he;
using namespace sm100;

namespace {

constexpr int QM = 128, KN = 64, STAGES = 3, NTHR = 320;
constexpr int K_SUB = KN * 128;              // bytes of a 64-key x 64-column tile
constexpr int Q_SUB = QM * 128;
constexpr float LOG2E = 1.4426950408889634f;
constexpr float LAZY = 8.f;                  // log2 growth of a maximum that is tolerated without rescaling

struct __align__(8) Bars {
  uint64_t q_full, k_full[STAGES], k_empty[STAGES], v_full[STAGES], v_empty[STAGES];
  uint64_t s_full[2][2];     // [tile][buffer] scores are in tensor memory
  uint64_t p_full[2][2];     // [tile][buffer] weights are in tensor memory (one arrive per warp).  Per buffer: a softmax may be
                             // one key tile ahead of the issuer, so one barrier could complete two phases unseen
  uint64_t o_done[2];        // the value product of the last weights has finished
  uint64_t drain;            // every product issued has finished (before tensor memory is freed)
  uint32_t tmem_base;
  int abort_flag;
};

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t pack2(float a, float b) {
  __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&h);
}

// Bounded wait that goes on after an abort.
__device__ __forceinline__ void drain(uint64_t* bar, uint32_t parity) {
  for (uint32_t i = 0; i < WAIT_LIMIT; ++i) {
    if (mbar_try_wait(bar, parity)) return;
    if (i > 64) __nanosleep(32);
  }
}

// Key tiles [lo_q, hi_q) (of 64 keys from key `lo`) that rows [first, last] see.
__device__ __forceinline__ void tile_range(const LatentSeg& g, int window, int first, int last, int& a, int& b) {
  const int k_lo = window > 0 ? max(g.lo, g.pos0 + first - window + 1) : g.lo;
  a = (k_lo - g.lo) / KN;
  b = (g.pos0 + last - g.lo) / KN + 1;
}

template <int NK, int DV>
constexpr size_t smem_bytes() {
  return (size_t)2 * NK * Q_SUB + STAGES * (size_t)(NK * K_SUB + DV * 128) + sizeof(Bars) + 1024;
}

// NK: 64-column sub-tiles of a query / key row (unrotated ones and the rotated one); DV: value width
template <int NK, int DV>
__global__ void __launch_bounds__(NTHR, 1)
latent_prefill_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                         const __grid_constant__ CUtensorMap tmR, const __grid_constant__ CUtensorMap tmV,
                         const __grid_constant__ LatentPrefillArgs a) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  uint8_t* sQ = smem;                                   // [2 tiles][NK][128 rows][128 bytes]
  uint8_t* sK = sQ + 2 * NK * Q_SUB;                    // [STAGES][NK][64 keys][128 bytes]
  uint8_t* sV = sK + STAGES * NK * K_SUB;               // [STAGES][DV rows][128 bytes = 64 keys]
  Bars* bar = reinterpret_cast<Bars*>(sV + STAGES * DV * 128);
  volatile int* abort_flag = &bar->abort_flag;
  constexpr int BM = 2 * QM;

  LatentSeg g;
  int tile;
  if (!latent_find_tile<BM>(a.seg_start, a.pos, a.n_seg, a.window, (int)gridDim.x - 1 - (int)blockIdx.x, g, tile)) return;
  const int hl = blockIdx.y, h = a.head0 + hl;
  const int t0 = tile * BM, rows = min(BM, g.T - t0);
  int lo_t[2], hi_t[2];
  tile_range(g, a.window, t0, t0 + min(rows, QM) - 1, lo_t[0], hi_t[0]);
  lo_t[1] = hi_t[1] = hi_t[0];
  if (rows > QM) tile_range(g, a.window, t0 + QM, t0 + rows - 1, lo_t[1], hi_t[1]);
  const int j_lo = lo_t[0], j_hi = max(hi_t[0], hi_t[1]);   // the second tile starts and ends no earlier than the first
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  if (threadIdx.x == 0) {
    mbar_init(&bar->q_full, 1);
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(&bar->k_full[s], 1);
      mbar_init(&bar->k_empty[s], 1);
      mbar_init(&bar->v_full[s], 1);
      mbar_init(&bar->v_empty[s], 1);
    }
    for (int t = 0; t < 2; ++t) {
      mbar_init(&bar->s_full[t][0], 1);
      mbar_init(&bar->s_full[t][1], 1);
      mbar_init(&bar->p_full[t][0], 4);
      mbar_init(&bar->p_full[t][1], 4);
      mbar_init(&bar->o_done[t], 1);
    }
    mbar_init(&bar->drain, 1);
    bar->abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 9) {
    tmem_alloc(&bar->tmem_base, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tm = bar->tmem_base;
  // columns: scores [tile][buffer] at 0, 64, 128, 192; accumulators at 256 and 384
  const auto s_col = [&](int t, int b) { return tm + (uint32_t)(t * 128 + b * 64); };
  const auto o_col = [&](int t) { return tm + (uint32_t)(256 + t * 128); };

  if (warp == 8) {
    if (elect_one()) {
      const int n_q = rows > QM ? 2 : 1;
      mbar_expect_tx(&bar->q_full, n_q * NK * Q_SUB);
      for (int t = 0; t < n_q; ++t)
        for (int k = 0; k < NK; ++k)
          tma_load_2d(sQ + (t * NK + k) * Q_SUB, &tmQ, &bar->q_full, h * a.qd + k * 64, g.row0 + t0 + t * QM);
      int n_k = 0, n_v = 0;
      for (int j = j_lo; j < j_hi; ++j) {
        const int it = j - j_lo, s = it % STAGES;
        const uint32_t ph = (it / STAGES) & 1;
        const int key = g.key0 + j * KN;
        if (!mbar_wait(&bar->k_empty[s], ph ^ 1, abort_flag, a.status, 601)) break;
        mbar_expect_tx(&bar->k_full[s], NK * K_SUB);
        for (int k = 0; k < NK - 1; ++k)
          tma_load_2d(sK + (s * NK + k) * K_SUB, &tmK, &bar->k_full[s], hl * a.dn + k * 64, key);
        tma_load_2d(sK + (s * NK + NK - 1) * K_SUB, &tmR, &bar->k_full[s], a.rank_cols, key);
        ++n_k;
        if (!mbar_wait(&bar->v_empty[s], ph ^ 1, abort_flag, a.status, 602)) break;
        mbar_expect_tx(&bar->v_full[s], DV * 128);
        tma_load_2d(sV + s * DV * 128, &tmV, &bar->v_full[s], key, hl * DV);
        ++n_v;
      }
      // no copy may still be in flight when the CTA leaves (matters only after an abort)
      drain(&bar->q_full, 0);
      for (int s = 0; s < STAGES; ++s) {
        if (s < n_k) drain(&bar->k_full[s], ((n_k - 1 - s) / STAGES) & 1);
        if (s < n_v) drain(&bar->v_full[s], ((n_v - 1 - s) / STAGES) & 1);
      }
    }
  } else if (warp == 9) {
    if (elect_one()) {
      constexpr uint32_t id_s = umma_idesc_bf16(QM, KN), id_o = umma_idesc_bf16(QM, DV);
      const auto active = [&](int t, int j) { return j >= lo_t[t] && j < hi_t[t]; };
      int n_s[2] = {0, 0}, n_o[2] = {0, 0};      // score products issued, value products issued per tile
      bool ok = mbar_wait(&bar->q_full, 0, abort_flag, a.status, 603);
      // scores of key tile j for both query tiles
      const auto scores = [&](int j) {
        const int it = j - j_lo, s = it % STAGES;
        if (!mbar_wait(&bar->k_full[s], (it / STAGES) & 1, abort_flag, a.status, 604)) return false;
        tc_fence_after();
        for (int t = 0; t < 2; ++t) {
          if (!active(t, j)) continue;
          const int b = n_s[t] & 1;
          // the buffer still holds the weights of two tiles ago until their value product is done
          if (n_s[t] >= 2 && !mbar_wait(&bar->o_done[t], n_s[t] & 1, abort_flag, a.status, 605)) return false;
          tc_fence_after();
#pragma unroll
          for (int k = 0; k < NK; ++k) {
            const uint32_t qa = smem_u32(sQ + (t * NK + k) * Q_SUB), ka = smem_u32(sK + (s * NK + k) * K_SUB);
#pragma unroll
            for (int u = 0; u < 4; ++u)
              umma_f16(s_col(t, b), umma_desc_k_sw128(qa + u * 32), umma_desc_k_sw128(ka + u * 32), id_s, (k > 0 || u > 0) ? 1u : 0u);
          }
          umma_commit(&bar->s_full[t][b]);
          ++n_s[t];
        }
        umma_commit(&bar->k_empty[s]);
        return true;
      };
      ok = ok && scores(j_lo);
      for (int j = j_lo; j < j_hi && ok; ++j) {
        if (j + 1 < j_hi && !scores(j + 1)) break;
        const int it = j - j_lo, s = it % STAGES;
        bool have_v = false;
        for (int t = 0; t < 2 && ok; ++t) {
          if (!active(t, j)) continue;
          const int i = n_o[t], b = i & 1;
          if (!mbar_wait(&bar->p_full[t][b], (i >> 1) & 1, abort_flag, a.status, 606)) { ok = false; break; }
          if (!have_v) {
            if (!mbar_wait(&bar->v_full[s], (it / STAGES) & 1, abort_flag, a.status, 607)) { ok = false; break; }
            have_v = true;
          }
          tc_fence_after();
          const uint32_t va = smem_u32(sV + s * DV * 128);
#pragma unroll
          for (int u = 0; u < 4; ++u)
            umma_f16_ts(o_col(t), s_col(t, b) + u * 8, umma_desc_k_sw128(va + u * 32), id_o, (i > 0 || u > 0) ? 1u : 0u);
          umma_commit(&bar->o_done[t]);
          ++n_o[t];
        }
        if (!ok) break;
        umma_commit(&bar->v_empty[s]);
      }
      umma_commit(&bar->drain);
      drain(&bar->drain, 0);
    }
  } else {
    // ------------------------------------------------------------ softmax of tile `t`, one row per thread
    const int t = warp >> 2, wl = warp & 3, row = wl * 32 + lane;
    const uint32_t lane_off = (uint32_t)(wl * 32) << 16;
    const int q_first = g.pos0 + t0 + t * QM + wl * 32, q_pos = q_first + lane;       // position of the warp's first row, own
    const float sc = a.scale * LOG2E;
    float m_ref = -INFINITY, l = 0.f;
    bool ok = true;
    int i = 0;
    for (int j = lo_t[t]; j < hi_t[t]; ++j, ++i) {
      const int b = i & 1;
      ok = __all_sync(0xffffffffu, mbar_wait(&bar->s_full[t][b], (i >> 1) & 1, abort_flag, a.status, 608));
      if (!ok) break;
      tc_fence_after();
      uint32_t r0[32], r1[32];
      tmem_ld_32x32(s_col(t, b) + lane_off, r0);
      tmem_ld_32x32(s_col(t, b) + lane_off + 32, r1);
      tmem_ld_wait();
      const int k0 = g.lo + j * KN;
      // masks only where the tile crosses an edge of what the warp's rows see
      if (k0 + KN - 1 > q_first || (a.window > 0 && k0 <= q_first + 31 - a.window)) {
        const int hi = q_pos - k0, lo = a.window > 0 ? hi - a.window : -1;            // visible columns: lo < c <= hi
#pragma unroll
        for (int c = 0; c < 32; ++c) {
          if (c > hi || (a.window > 0 && c <= lo)) r0[c] = 0xff800000u;
          if (c + 32 > hi || (a.window > 0 && c + 32 <= lo)) r1[c] = 0xff800000u;
        }
      }
      float mx = -INFINITY;
#pragma unroll
      for (int c = 0; c < 32; ++c) mx = fmaxf(mx, fmaxf(__uint_as_float(r0[c]), __uint_as_float(r1[c])));
      mx *= sc;                                        // the scale is positive (checked by the launcher)
      // a maximum far above the reference (or the first one): move the reference and rescale what was accumulated
      const bool grow = mx > m_ref + LAZY;
      if (__any_sync(0xffffffffu, grow)) {
        const float m_new = grow ? mx : m_ref, f = m_ref == -INFINITY ? 0.f : ex2(m_ref - m_new);
        m_ref = m_new;
        l *= f;
        if (i > 0) {
          ok = __all_sync(0xffffffffu, mbar_wait(&bar->o_done[t], (i - 1) & 1, abort_flag, a.status, 609));
          if (!ok) break;
          tc_fence_after();
#pragma unroll 1
          for (int c = 0; c < DV; c += 32) {
            uint32_t o[32];
            tmem_ld_32x32(o_col(t) + lane_off + c, o);
            tmem_ld_wait();
#pragma unroll
            for (int e = 0; e < 32; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * f);
            tmem_st_32x32(o_col(t) + lane_off + c, o);
          }
        }
      }
      const float neg = m_ref == -INFINITY ? 0.f : -m_ref;     // nothing seen yet: every weight is 2^-inf = 0
      float s0 = 0.f, s1 = 0.f;
#pragma unroll
      for (int c = 0; c < 32; c += 2) {
        const float p0 = ex2(fmaf(__uint_as_float(r0[c]), sc, neg)), p1 = ex2(fmaf(__uint_as_float(r0[c + 1]), sc, neg));
        const float p2 = ex2(fmaf(__uint_as_float(r1[c]), sc, neg)), p3 = ex2(fmaf(__uint_as_float(r1[c + 1]), sc, neg));
        s0 += p0 + p1;
        s1 += p2 + p3;
        r0[c >> 1] = pack2(p0, p1);
        r1[c >> 1] = pack2(p2, p3);
      }
      l += s0 + s1;
#pragma unroll
      for (int c = 0; c < 16; ++c) r0[16 + c] = r1[c];
      tmem_st_32x32(s_col(t, b) + lane_off, r0);
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bar->p_full[t][b]);
    }
    if (ok && i > 0) {
      // the last two value products may both be outstanding: wait for them in turn, a parity tells only neighbours apart
      if (i > 1) ok = __all_sync(0xffffffffu, mbar_wait(&bar->o_done[t], i & 1, abort_flag, a.status, 610));
      if (ok) ok = __all_sync(0xffffffffu, mbar_wait(&bar->o_done[t], (i - 1) & 1, abort_flag, a.status, 611));
      if (ok) {
        tc_fence_after();
        float f = 1.f;
        if (a.sink != nullptr) {
          const float sk = a.sink[h] * LOG2E, mn = fmaxf(m_ref, sk);
          f = ex2(m_ref - mn);
          l = l * f + ex2(sk - mn);
        }
        const float inv = l > 0.f ? f / l : 0.f;
        const bool live = t * QM + row < rows;
        __nv_bfloat16* dst = a.out + ((size_t)(g.row0 + t0 + t * QM + (live ? row : 0)) * a.H + h) * DV;
#pragma unroll 1
        for (int c = 0; c < DV; c += 32) {
          uint32_t o[32];
          tmem_ld_32x32(o_col(t) + lane_off + c, o);
          tmem_ld_wait();
          if (live) {
#pragma unroll
            for (int v = 0; v < 4; ++v) {
              uint4 pk;
              uint32_t* pw = reinterpret_cast<uint32_t*>(&pk);
#pragma unroll
              for (int e = 0; e < 4; ++e)
                pw[e] = pack2(__uint_as_float(o[v * 8 + 2 * e]) * inv, __uint_as_float(o[v * 8 + 2 * e + 1]) * inv);
              *reinterpret_cast<uint4*>(dst + c + v * 8) = pk;
            }
          }
        }
        tc_fence_before();
      }
    }
  }
  __syncthreads();
  tc_fence_after();
  if (warp == 9) tmem_dealloc(tm, 512);
}

template <int NK, int DV>
int launch(const LatentPrefillArgs& a, const CUtensorMap& q, const CUtensorMap& k, const CUtensorMap& r, const CUtensorMap& v,
           cudaStream_t stream) {
  constexpr size_t smem = smem_bytes<NK, DV>();
  cudaError_t e = cudaFuncSetAttribute(latent_prefill_tc_kernel<NK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  latent_prefill_tc_kernel<NK, DV><<<dim3(a.tiles, a.n_heads), NTHR, smem, stream>>>(q, k, r, v, a);
  HE_LAUNCH_CHECK();
  return 0;
}

}  // namespace

// Is there a tensor-memory form for this head shape?  (256 query rows per tile; values expanded transposed)
HE_API int he_latent_prefill_tc_ok(int dn, int qd, int dv) {
  return (dn == 64 || dn == 128) && (dv == 64 || dv == 128) && qd > dn && qd - dn <= 64;
}

HE_API int he_latent_prefill_tc(const LatentPrefillArgs* args, cudaStream_t stream) {
  const LatentPrefillArgs& a = *args;
  if (a.n_seg <= 0 || a.tiles <= 0 || a.n_heads <= 0) return 0;
  if (!he_latent_prefill_tc_ok(a.dn, a.qd, a.dv) || a.qd % 8 != 0 || a.rank_cols % 8 != 0 || a.W % 8 != 0 || a.head0 < 0 ||
      a.head0 + a.n_heads > a.H || a.n_heads > 65535 || a.keys <= 0 || a.keys % LATENT_SEG_ALIGN != 0 || a.rows <= 0 ||
      !(a.scale > 0.f) || a.rank_cols + a.qd - a.dn > a.W)
    return -HE_ERR_BAD_ARG;
  CUtensorMap q, k, r, v;
  int rc = make_map(&q, a.q, a.rows, (long long)a.H * a.qd, (long long)a.H * a.qd, QM);
  if (rc == 0) rc = make_map(&k, a.kx, a.keys, (long long)a.n_heads * a.dn, (long long)a.n_heads * a.dn, KN);
  if (rc == 0) rc = make_map(&r, a.lat, a.keys, a.W, a.W, KN);
  if (rc == 0) rc = make_map(&v, a.v, (long long)a.n_heads * a.dv, a.keys, a.keys, a.dv);
  if (rc != 0) return rc;
  if (a.dn == 64 && a.dv == 64) return launch<2, 64>(a, q, k, r, v, stream);
  if (a.dn == 64) return launch<2, 128>(a, q, k, r, v, stream);
  if (a.dv == 64) return launch<3, 64>(a, q, k, r, v, stream);
  return launch<3, 128>(a, q, k, r, v, stream);
}
