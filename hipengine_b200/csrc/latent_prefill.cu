// Prefill form of latent attention: long prompt portions attend with full keys and values.
//
// The latents of every visible key lie side by side (latent_gather_kernel), tensor-core GEMMs have expanded them to keys
// [key][head][dn] and values [key][head][dv], and the rotated key part is read from the gathered latent row itself, so it
// exists once and not per head.  This form takes any head shape up to 256 columns; latent_prefill_tc.cu has the common ones.  Flash-style single pass: a CTA owns 64 MT query rows of one head (4 warps x MT x 16 rows),
// streams 32-key tiles with cp.async (double buffered), keeps running maximum / sum per row and the output in registers;
// mma.sync m16n8k16 with fp32 accumulation.  Causal, optionally only the last `window` keys, optionally with a learned term
// per head in the softmax denominator.  Segments of several requests share a launch.
#include "latent_segs.cuh"

using namespace he;

namespace {

constexpr int BN = 32;       // keys per tile
constexpr int NTHR = 128;
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ void cp_async16(void* smem, const void* gmem, bool valid) {
  const uint32_t s = (uint32_t)__cvta_generic_to_shared(smem);
  const int sz = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(s), "l"(gmem), "r"(sz) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], const void* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], const void* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
  __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&h);
}

// grid (tiles of 64 MT rows over all segments, heads of this launch)
template <int DK, int DV, int MT>
__global__ void __launch_bounds__(NTHR) latent_prefill_kernel(const __grid_constant__ LatentPrefillArgs a) {
  constexpr int BM = 64 * MT, LK = DK + 8, LV = DV + 8;     // padded row strides: conflict-free ldmatrix
  extern __shared__ __align__(16) __nv_bfloat16 sm[];
  __nv_bfloat16* sQ = sm;                    // [BM][LK]
  __nv_bfloat16* sK = sQ + BM * LK;          // [2][BN][LK]
  __nv_bfloat16* sV = sK + 2 * BN * LK;      // [2][BN][LV]
  LatentSeg seg;
  int qt;
  if (!latent_find_tile<BM>(a.seg_start, a.pos, a.n_seg, a.window, (int)gridDim.x - 1 - (int)blockIdx.x, seg, qt)) return;
  const int row0 = seg.row0, T = seg.T, pos0 = seg.pos0, lo = seg.lo, key_row0 = seg.key0;
  const int hl = blockIdx.y, h = a.head0 + hl;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, c = lane & 3;
  const int t0 = qt * BM, rows = min(BM, T - t0);
  const int kv_end = pos0 + t0 + rows;                                              // keys [kv_begin, kv_end)
  const int kv_begin = a.window > 0 ? max(lo, pos0 + t0 - a.window + 1) : 0;
  const int n_tiles = (kv_end - kv_begin + BN - 1) / BN;
  const int dn8 = a.dn / 8, qd8 = a.qd / 8, dv8 = a.dv / 8;
  const size_t k_ld = (size_t)a.n_heads * a.dn, v_ld = (size_t)a.n_heads * a.dv;

  auto load_kv = [&](int tile, int buf) {
    const int k0 = kv_begin + tile * BN;
    constexpr int CK = DK / 8, CV = DV / 8;
#pragma unroll 2
    for (int i = tid; i < BN * CK; i += NTHR) {
      const int r = i / CK, ch = i % CK, p = k0 + r;
      const size_t kr = key_row0 + min(p, kv_end - 1) - lo;
      const __nv_bfloat16* src = ch < dn8 ? a.kx + kr * k_ld + (size_t)hl * a.dn + ch * 8
                                          : a.lat + kr * a.W + a.rank_cols + (ch < qd8 ? (ch - dn8) * 8 : 0);
      cp_async16(sK + ((size_t)buf * BN + r) * LK + ch * 8, src, p < kv_end && ch < qd8);
    }
#pragma unroll 2
    for (int i = tid; i < BN * CV; i += NTHR) {
      const int r = i / CV, ch = i % CV, p = k0 + r;
      const size_t kr = key_row0 + min(p, kv_end - 1) - lo;
      const __nv_bfloat16* src = a.v + kr * v_ld + (size_t)hl * a.dv + (ch < dv8 ? ch * 8 : 0);
      cp_async16(sV + ((size_t)buf * BN + r) * LV + ch * 8, src, p < kv_end && ch < dv8);
    }
  };
  {
    constexpr int CK = DK / 8;
    for (int i = tid; i < BM * CK; i += NTHR) {
      const int r = i / CK, ch = i % CK;
      const bool valid = r < rows && ch < qd8;
      const __nv_bfloat16* src = a.q + ((size_t)(row0 + t0 + (r < rows ? r : 0)) * a.H + h) * a.qd + (ch < qd8 ? ch * 8 : 0);
      cp_async16(sQ + (size_t)r * LK + ch * 8, src, valid);
    }
  }
  load_kv(0, 0);
  cp_async_commit();

  float o[MT][DV / 8][4], m_run[MT][2], l_run[MT][2];
#pragma unroll
  for (int m = 0; m < MT; ++m) {
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) o[m][i][0] = o[m][i][1] = o[m][i][2] = o[m][i][3] = 0.f;
    m_run[m][0] = m_run[m][1] = -INFINITY;
    l_run[m][0] = l_run[m][1] = 0.f;
  }
  const float sc_log2 = a.scale * LOG2E;
  const int wrow = warp * 16 * MT;                       // first row of this warp in the tile
  const int first_pos = pos0 + t0 + wrow;

  for (int tile = 0; tile < n_tiles; ++tile) {
    const int buf = tile & 1;
    if (tile + 1 < n_tiles) load_kv(tile + 1, buf ^ 1);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const int k0 = kv_begin + tile * BN;
    // a tile no row of this warp can see is skipped (later than its last row, or before its first row's window)
    const bool seen = k0 <= first_pos + 16 * MT - 1 && !(a.window > 0 && k0 + BN <= first_pos - a.window + 1);
    if (seen) {
      float sacc[MT][BN / 8][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int j = 0; j < BN / 8; ++j) sacc[m][j][0] = sacc[m][j][1] = sacc[m][j][2] = sacc[m][j][3] = 0.f;
      const __nv_bfloat16* kb = sK + (size_t)buf * BN * LK;
#pragma unroll
      for (int kk = 0; kk < DK / 32; ++kk) {
        uint32_t qa[MT][2][4];
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          const __nv_bfloat16* qp = sQ + (size_t)(wrow + m * 16 + (lane & 15)) * LK + kk * 32 + (lane >> 4) * 8;
          ldsm_x4(qa[m][0], qp);
          ldsm_x4(qa[m][1], qp + 16);
        }
#pragma unroll
        for (int j = 0; j < BN / 8; ++j) {
          uint32_t kf[4];
          ldsm_x4(kf, kb + (size_t)(j * 8 + (lane & 7)) * LK + kk * 32 + (lane >> 3) * 8);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma_bf16(sacc[m][j], qa[m][0], kf[0], kf[1]);
            mma_bf16(sacc[m][j], qa[m][1], kf[2], kf[3]);
          }
        }
      }
      // masks only where the tile crosses an edge of what this warp's rows see
      const bool edge = k0 + BN - 1 > first_pos || k0 + BN > kv_end ||
                        (a.window > 0 && k0 <= first_pos + 16 * MT - 1 - a.window);
      uint32_t pa[MT][BN / 16][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int j = 0; j < BN / 8; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            float v = sacc[m][j][e] * sc_log2;
            if (edge) {
              const int key = k0 + j * 8 + 2 * c + (e & 1), qp = first_pos + m * 16 + g + (e >> 1) * 8;
              const bool ok = key <= qp && key < kv_end && !(a.window > 0 && key <= qp - a.window);
              v = ok ? v : -INFINITY;
            }
            sacc[m][j][e] = v;
            mx[e >> 1] = fmaxf(mx[e >> 1], v);
          }
        float corr[2], mref[2];
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
          mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
          const float mn = fmaxf(m_run[m][r], mx[r]);
          corr[r] = mn == -INFINITY ? 1.f : exp2f(m_run[m][r] - mn);
          mref[r] = mn == -INFINITY ? 0.f : mn;          // nothing seen yet: exp2(-inf) = 0 below
          m_run[m][r] = mn;
          l_run[m][r] *= corr[r];
        }
#pragma unroll
        for (int j = 0; j < BN / 8; ++j) {
          float p[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            p[e] = exp2f(sacc[m][j][e] - mref[e >> 1]);
            l_run[m][e >> 1] += p[e];
          }
          pa[m][j >> 1][(j & 1) * 2] = pack_bf16(p[0], p[1]);
          pa[m][j >> 1][(j & 1) * 2 + 1] = pack_bf16(p[2], p[3]);
        }
        if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
          for (int i = 0; i < DV / 8; ++i) {
            o[m][i][0] *= corr[0]; o[m][i][1] *= corr[0];
            o[m][i][2] *= corr[1]; o[m][i][3] *= corr[1];
          }
        }
      }
      const __nv_bfloat16* vb = sV + (size_t)buf * BN * LV;
#pragma unroll
      for (int ks = 0; ks < BN / 16; ++ks)
#pragma unroll
        for (int i = 0; i < DV / 16; ++i) {
          uint32_t vf[4];
          ldsm_x4_t(vf, vb + (size_t)(ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LV + i * 16 + (lane >> 4) * 8);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma_bf16(o[m][2 * i], pa[m][ks], vf[0], vf[1]);
            mma_bf16(o[m][2 * i + 1], pa[m][ks], vf[2], vf[3]);
          }
        }
    }
    __syncthreads();
  }

#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float l = l_run[m][r];
      l += __shfl_xor_sync(0xffffffffu, l, 1);
      l += __shfl_xor_sync(0xffffffffu, l, 2);
      const int row = wrow + m * 16 + g + r * 8;
      if (row >= rows) continue;
      float f = 1.f;
      if (a.sink != nullptr) {
        const float sk = a.sink[h] * LOG2E, mn = fmaxf(m_run[m][r], sk);
        f = exp2f(m_run[m][r] - mn);
        l = l * f + exp2f(sk - mn);
      }
      const float inv = l > 0.f ? f / l : 0.f;
      __nv_bfloat16* dst = a.out + ((size_t)(row0 + t0 + row) * a.H + h) * a.dv;
#pragma unroll
      for (int i = 0; i < DV / 8; ++i) {
        if (i < dv8)
          *reinterpret_cast<__nv_bfloat162*>(dst + i * 8 + 2 * c) =
              __floats2bfloat162_rn(o[m][i][2 * r] * inv, o[m][i][2 * r + 1] * inv);
      }
    }
}

template <int DK, int DV, int MT>
int launch(const LatentPrefillArgs& a, cudaStream_t stream) {
  const size_t smem = ((size_t)(64 * MT + 2 * BN) * (DK + 8) + (size_t)2 * BN * (DV + 8)) * sizeof(__nv_bfloat16);
  cudaError_t e = cudaFuncSetAttribute(latent_prefill_kernel<DK, DV, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  latent_prefill_kernel<DK, DV, MT><<<dim3(a.tiles, a.n_heads), NTHR, smem, stream>>>(a);
  HE_LAUNCH_CHECK();
  return 0;
}

}  // namespace

// Query rows per tile for a head shape (the caller sizes `tiles` with it); 0: no kernel for this shape.
HE_API int he_latent_prefill_tile_rows(int qd, int dv) {
  if (qd <= 192 && dv <= 128) return 128;
  if (qd <= 256 && dv <= 256) return 64;
  return 0;
}

HE_API int he_latent_prefill(const LatentPrefillArgs* args, cudaStream_t stream) {
  const LatentPrefillArgs& a = *args;
  if (a.n_seg <= 0 || a.tiles <= 0 || a.n_heads <= 0) return 0;
  if (a.dn % 8 != 0 || a.dv % 8 != 0 || a.qd % 8 != 0 || a.qd <= a.dn || a.rank_cols % 8 != 0 || a.W % 8 != 0 ||
      a.rank_cols + a.qd - a.dn > a.W || a.head0 < 0 || a.head0 + a.n_heads > a.H || a.n_heads > 65535)
    return -HE_ERR_BAD_ARG;
  if (a.qd <= 64 && a.dv <= 64) return launch<64, 64, 2>(a, stream);
  if (a.qd <= 128 && a.dv <= 64) return launch<128, 64, 2>(a, stream);
  if (a.qd <= 128 && a.dv <= 128) return launch<128, 128, 2>(a, stream);
  if (a.qd <= 192 && a.dv <= 128) return launch<192, 128, 2>(a, stream);
  if (a.qd <= 256 && a.dv <= 256) return launch<256, 256, 1>(a, stream);
  return -HE_ERR_BAD_ARG;
}
HE_API int he_latent_prefill_args_size() { return (int)sizeof(LatentPrefillArgs); }
