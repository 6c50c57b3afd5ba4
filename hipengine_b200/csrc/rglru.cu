// Scan of the real-gated linear recurrence over packed segments (prompt portions, verify chains, any mix).
//
// A linear recurrence S <- a S + d composes: a run of tokens is one pair (product of a, S from zero).  A CTA owns 16
// channels of one segment and walks it in tiles of 256 tokens: thread (group, channel) turns the gate products of its eight
// tokens into (a, d) kept in registers and composes them, a warp per channel composes the 32 groups by shuffles, and each
// thread goes through its tokens again from the state before its group.  Everything is read once; nothing is shared between
// CTAs.  The CTA then replaces the slot's state and the convolution's last inputs.  Batches of single tokens (one row per
// segment) need no composition: a thread per channel.
#include "rglru.cuh"

using namespace he;

namespace {

constexpr int CH = 16, GROUPS = 32, LEN = 8, NTHR = CH * GROUPS, TILE = GROUPS * LEN;

template <bool ACT_F32, bool ROW_F32>
__global__ void __launch_bounds__(NTHR, 2) rglru_scan_kernel(const __grid_constant__ RglruArgs a) {
  __shared__ float sA[GROUPS][CH + 1], sB[GROUPS][CH + 1];
  pdl_wait();
  pdl_launch();
  const int seg = blockIdx.y, s0 = a.seg_start[seg], s1 = a.seg_start[seg + 1], slot = a.seg_slot[seg];
  if (!HE_INDEX_OK(slot, a.n_slots, HE_SITE_STATE_SLOT)) return;
  const int ch = threadIdx.x & (CH - 1), grp = threadIdx.x / CH, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c = blockIdx.x * CH + ch, cw = blockIdx.x * CH + warp;          // own channel; channel composed by this warp
  const bool live = c < a.C;
  const int cc = live ? c : a.C - 1, b = cc / a.block_cols, cb = cc % a.block_cols;
  const float* g = a.g + (size_t)b * a.g_bs + cb;
  const size_t u0 = (size_t)b * a.u_bs + cb;
  const float gb0 = a.gb[(size_t)b * 2 * a.block_cols + cb], gb1 = a.gb[(size_t)b * 2 * a.block_cols + a.block_cols + cb];
  const float decay = a.decay[cc], yb = a.yb[cc];
  float S0 = cw < a.C ? a.S[(size_t)slot * a.C + cw] : 0.f;                  // of channel cw, before the tile
  for (int tile = s0; tile < s1; tile += TILE) {
    const int t0 = tile + grp * LEN, last = s1 - 1 - t0;                      // tokens behind the last one repeat it
    float A[LEN], d[LEN], u[LEN];
    if (last >= LEN - 1) {
      const float* gp = g + (size_t)t0 * a.g_ts;
      size_t ui = u0 + (size_t)t0 * a.u_ts;
#pragma unroll
      for (int k = 0; k < LEN; ++k) {
        A[k] = gp[0];
        d[k] = gp[a.block_cols];
        u[k] = rg_load(a.u, ACT_F32, ui);
        gp += a.g_ts;
        ui += a.u_ts;
      }
    } else {
#pragma unroll
      for (int k = 0; k < LEN; ++k) {
        const int t = min(t0 + k, s1 - 1);
        A[k] = g[(size_t)t * a.g_ts];
        d[k] = g[(size_t)t * a.g_ts + a.block_cols];
        u[k] = rg_load(a.u, ACT_F32, u0 + (size_t)t * a.u_ts);
      }
    }
    float pa = 1.f, pb = 0.f;
#pragma unroll
    for (int k = 0; k < LEN; ++k) {
      float ak, dk;
      rg_gates(A[k] + gb0, d[k] + gb1, decay, u[k], ak, dk);
      if (k > last) {
        ak = 1.f;
        dk = 0.f;
      }
      A[k] = ak;
      d[k] = dk;
      pb = ak * pb + dk;
      pa *= ak;
    }
    sA[grp][ch] = pa;
    sB[grp][ch] = pb;
    float y[LEN];                                        // on their way while the groups are composed
#pragma unroll
    for (int k = 0; k < LEN; ++k) y[k] = rg_load(a.y, ROW_F32, (size_t)min(t0 + k, s1 - 1) * a.row_stride + cc);
    __syncthreads();
    pa = sA[lane][warp];
    pb = sB[lane][warp];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float qa = __shfl_up_sync(0xffffffffu, pa, o), qb = __shfl_up_sync(0xffffffffu, pb, o);
      if (lane >= o) {
        pb = pa * qb + pb;
        pa *= qa;
      }
    }
    float ea = __shfl_up_sync(0xffffffffu, pa, 1), eb = __shfl_up_sync(0xffffffffu, pb, 1);
    if (lane == 0) {
      ea = 1.f;
      eb = 0.f;
    }
    sB[lane][warp] = ea * S0 + eb;                       // state before the group
    S0 = __shfl_sync(0xffffffffu, pa, 31) * S0 + __shfl_sync(0xffffffffu, pb, 31);
    __syncthreads();
    float S = sB[grp][ch];
#pragma unroll
    for (int k = 0; k < LEN; ++k) {
      S = A[k] * S + d[k];
      const int t = t0 + k;
      if (live && k <= last) {
        const float v = S * rg_gelu(y[k] + yb);
        const size_t o = (size_t)t * a.out_stride + c;
        if constexpr (ACT_F32) reinterpret_cast<float*>(a.out)[o] = v;
        else reinterpret_cast<__nv_bfloat16*>(a.out)[o] = f32_to_bf16(v);
        if (a.journal != nullptr) a.journal[(size_t)t * a.C + c] = S;
      }
    }
    __syncthreads();                                     // sB is written again
  }
  if (a.journal != nullptr) return;
  if (lane == 0 && cw < a.C) a.S[(size_t)slot * a.C + cw] = S0;
  if (grp == 0 && live) rg_conv_state(a, slot, c, s0, s1 - s0);
}

// one row per segment: grid (ceil(C / 256), n_seg)
template <bool ACT_F32, bool ROW_F32>
__global__ void __launch_bounds__(256) rglru_rows_kernel(const __grid_constant__ RglruArgs a) {
  pdl_wait();
  pdl_launch();
  const int t = blockIdx.y, c = blockIdx.x * 256 + threadIdx.x, slot = a.seg_slot[t];
  if (c >= a.C || !HE_INDEX_OK(slot, a.n_slots, HE_SITE_STATE_SLOT)) return;
  const int b = c / a.block_cols, cb = c % a.block_cols;
  const float* g = a.g + (size_t)b * a.g_bs + (size_t)t * a.g_ts + cb;
  const float* gb = a.gb + (size_t)b * 2 * a.block_cols + cb;
  float ak, dk;
  rg_gates(g[0] + gb[0], g[a.block_cols] + gb[a.block_cols], a.decay[c],
           rg_load(a.u, ACT_F32, (size_t)b * a.u_bs + (size_t)t * a.u_ts + cb), ak, dk);
  const float S = ak * a.S[(size_t)slot * a.C + c] + dk;
  const float v = S * rg_gelu(rg_load(a.y, ROW_F32, (size_t)t * a.row_stride + c) + a.yb[c]);
  const size_t o = (size_t)t * a.out_stride + c;
  if constexpr (ACT_F32) reinterpret_cast<float*>(a.out)[o] = v;
  else reinterpret_cast<__nv_bfloat16*>(a.out)[o] = f32_to_bf16(v);
  if (a.journal != nullptr) {
    a.journal[(size_t)t * a.C + c] = S;
    return;
  }
  a.S[(size_t)slot * a.C + c] = S;
  rg_conv_state(a, slot, c, t, 1);
}

}  // namespace

HE_API int he_rglru_scan(const RglruArgs* args, cudaStream_t stream) {
  const RglruArgs& a = *args;
  if (a.n_seg <= 0) return 0;
  if (a.C <= 0 || a.block_cols <= 0 || a.C % a.block_cols != 0 || a.taps < 1 || a.g == nullptr || a.n_seg > 65535 ||
      (a.act_f32 != 0 && a.row_dtype != 0))
    return -HE_ERR_BAD_ARG;
  if (a.T == a.n_seg) {
    const dim3 grid((a.C + 255) / 256, a.n_seg), block(256);
    return (int)(a.act_f32 ? launch_pdl(rglru_rows_kernel<true, true>, grid, block, 0, stream, a)
                 : a.row_dtype == 0 ? launch_pdl(rglru_rows_kernel<false, true>, grid, block, 0, stream, a)
                                    : launch_pdl(rglru_rows_kernel<false, false>, grid, block, 0, stream, a));
  }
  const dim3 grid((a.C + CH - 1) / CH, a.n_seg), block(NTHR);
  return (int)(a.act_f32 ? launch_pdl(rglru_scan_kernel<true, true>, grid, block, 0, stream, a)
               : a.row_dtype == 0 ? launch_pdl(rglru_scan_kernel<false, true>, grid, block, 0, stream, a)
                                  : launch_pdl(rglru_scan_kernel<false, false>, grid, block, 0, stream, a));
}
HE_API int he_rglru_args_size() { return (int)sizeof(RglruArgs); }
