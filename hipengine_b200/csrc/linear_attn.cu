// Linear attention (retention, gated delta rule), serial forms: any head sizes, any segments, journals; fp32 throughout.
//
//   step     batches of single tokens (decode): one launch from projected rows to the gated output, a CTA per (head, request)
//   prepare  rows -> rotated / convolved and normalised fp32 rows and gates
//   scan     the recurrence over packed segments; a CTA owns 32 state columns of a head, a column is shared by eight lanes
//   output   norm per head and output gate
// Long prompts go through linear_chunk.cu instead of prepare and scan.
#include "linear_attn.cuh"

using namespace he;

namespace {

// ---------------------------------------------------------------- prepare: one warp per (token, head of q / k / v), and gates
__global__ void __launch_bounds__(256) linear_prepare_kernel(const __grid_constant__ LinearArgs a) {
  pdl_wait();
  pdl_launch();
  const int lane = threadIdx.x & 31, items = 2 * a.G + a.H + (a.delta ? 1 : 0);
  const long long w = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
  if (w >= (long long)a.T * items) return;
  const int t = (int)(w / items), it = (int)(w % items);
  const int sg = a.tok_seg[t], s0 = a.seg_start[sg], slot = a.seg_slot[sg], p = a.pos[t];
  if (!HE_INDEX_OK(slot, a.n_slots, HE_SITE_STATE_SLOT)) return;
  if (it < a.G) {
    la_prepare_head(a, t, s0, slot, p, it * a.dim, a.qscale, a.qf + ((size_t)t * a.G + it) * a.dim, lane);
  } else if (it < 2 * a.G) {
    const int h = it - a.G;
    la_prepare_head(a, t, s0, slot, p, a.ck + h * a.dim, a.kscale, a.kf + ((size_t)t * a.G + h) * a.dim, lane);
  } else if (it < 2 * a.G + a.H) {
    const int h = it - 2 * a.G;
    float* v = a.vf + ((size_t)t * a.H + h) * a.vcols;
    for (int d = lane; d < a.vcols; d += 32) {
      const int c = a.cv + h * a.vdim + d;
      v[d] = d >= a.vdim ? 0.f : a.delta ? la_conv(a, t, s0, slot, p, c) : la_row(a, (size_t)t * a.stride + c);
    }
  } else {
    for (int h = lane; h < a.H; h += 32) {
      a.g1[(size_t)t * a.H + h] = expm1f(la_log_decay(a, t, h));
      a.beta[(size_t)t * a.H + h] = la_beta(a, t, h);
    }
    if (a.jring != nullptr && a.taps > 1)                      // padded columns of the convolution
      for (int c = lane; c < a.C; c += 32) {
        const bool real = c < a.G * a.dim || (c >= a.ck && c < a.ck + a.G * a.dim) || (c >= a.cv && c < a.cv + a.H * a.vdim);
        if (!real)
          for (int e = 0; e < a.taps; ++e) a.jring[((size_t)t * a.taps + e) * a.C + c] = 0.f;
      }
  }
}

// ---------------------------------------------------------------- scan
constexpr int SLICE = 32;     // state columns per CTA
constexpr int LPC = 8;        // lanes per column

// grid (n_seg, H, ceil(vcols / 32)), 256 threads; DK: dim rounded up, rows behind dim stay zero
template <int DK, bool DELTA>
__global__ void __launch_bounds__(SLICE * LPC) linear_scan_kernel(const __grid_constant__ LinearArgs a) {
  constexpr int RPL = DK / LPC, NT = SLICE * LPC, TCH = DK <= 128 ? 16 : 8, KPAD = DK + 4 * LPC;
  __shared__ __align__(16) float sq[TCH][KPAD], sk[TCH][KPAD];      // a lane's rows start 4 floats further per lane
  __shared__ float sv[TCH][SLICE], sg1[TCH], sb[TCH];
  pdl_wait();
  pdl_launch();
  const int seg = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, cw = tid / LPC, ks = tid % LPC;
  const int col = blockIdx.z * SLICE + cw, kh = h / (a.H / a.G);
  const bool live = col < a.vcols;
  const int s0 = a.seg_start[seg], s1 = a.seg_start[seg + 1], slot = a.seg_slot[seg];
  if (!HE_INDEX_OK(slot, a.n_slots, HE_SITE_STATE_SLOT)) return;
  float* Sg = a.S + ((size_t)slot * a.H + h) * a.dim * a.vcols;
  float S[RPL];
#pragma unroll
  for (int i = 0; i < RPL; ++i) {
    const int d = ks * RPL + i;
    S[i] = live && d < a.dim ? Sg[(size_t)d * a.vcols + col] : 0.f;
  }
  const int koff = ks * (RPL + 4);
  const float g_const = DELTA ? 0.f : a.gm[h];
  for (int c0 = s0; c0 < s1; c0 += TCH) {
    const int n = min(TCH, s1 - c0);
    __syncthreads();
    for (int i = tid; i < n * DK; i += NT) {
      const int tt = i / DK, d = i % DK, dst = d + (d / RPL) * 4;
      const size_t src = ((size_t)(c0 + tt) * a.G + kh) * a.dim + d;
      sq[tt][dst] = d < a.dim ? a.qf[src] : 0.f;
      sk[tt][dst] = d < a.dim ? a.kf[src] : 0.f;
    }
    for (int i = tid; i < n * SLICE; i += NT) {
      const int tt = i / SLICE, c = blockIdx.z * SLICE + i % SLICE;
      sv[tt][i % SLICE] = c < a.vcols ? a.vf[((size_t)(c0 + tt) * a.H + h) * a.vcols + c] : 0.f;
    }
    if (DELTA && tid < n) {
      sg1[tid] = a.g1[(size_t)(c0 + tid) * a.H + h];
      sb[tid] = a.beta[(size_t)(c0 + tid) * a.H + h];
    }
    __syncthreads();
    for (int tt = 0; tt < n; ++tt) {
      const float g1 = DELTA ? sg1[tt] : g_const;
      float u = sv[tt][cw];
      const float* kp = &sk[tt][koff];
      const float* qp = &sq[tt][koff];
      if constexpr (DELTA) {
        float p4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int i = 0; i < RPL; ++i) {
          S[i] = fmaf(g1, S[i], S[i]);
          p4[i & 3] += kp[i] * S[i];
        }
        float kv = (p4[0] + p4[1]) + (p4[2] + p4[3]);
#pragma unroll
        for (int o = 1; o < LPC; o <<= 1) kv += __shfl_xor_sync(0xffffffffu, kv, o);
        u = (u - kv) * sb[tt];
      }
      float o4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int i = 0; i < RPL; ++i) {
        if (!DELTA) S[i] = fmaf(g1, S[i], S[i]);
        S[i] += kp[i] * u;
        o4[i & 3] += qp[i] * S[i];
      }
      float o = (o4[0] + o4[1]) + (o4[2] + o4[3]);
#pragma unroll
      for (int of = 1; of < LPC; of <<= 1) o += __shfl_xor_sync(0xffffffffu, o, of);
      if (live && ks == 0) a.o[((size_t)(c0 + tt) * a.H + h) * a.vcols + col] = o;
      if (a.jS != nullptr && live) {
        float* J = a.jS + ((size_t)(c0 + tt) * a.H + h) * a.dim * a.vcols;
#pragma unroll
        for (int i = 0; i < RPL; ++i)
          if (ks * RPL + i < a.dim) J[(size_t)(ks * RPL + i) * a.vcols + col] = S[i];
      }
    }
  }
  if (a.jS != nullptr) return;
  if (live) {
#pragma unroll
    for (int i = 0; i < RPL; ++i)
      if (ks * RPL + i < a.dim) Sg[(size_t)(ks * RPL + i) * a.vcols + col] = S[i];
  }
  if (DELTA && a.taps > 1)                                     // the CTAs of a segment share its ring's columns
    for (int c = (h * gridDim.z + blockIdx.z) * NT + tid; c < a.C; c += a.H * gridDim.z * NT) la_ring_update(a, slot, s0, s1, c);
}

// ---------------------------------------------------------------- output: one warp per (token, head)
template <typename OutT>
__global__ void __launch_bounds__(256) linear_out_kernel(const __grid_constant__ LinearArgs a) {
  pdl_wait();
  pdl_launch();
  const long long w = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
  const int lane = threadIdx.x & 31;
  if (w >= (long long)a.T * a.H) return;
  const int t = (int)(w / a.H), h = (int)(w % a.H);
  const float* o = a.o + (size_t)w * a.vcols;
  float ss = 0.f;
  for (int i = lane; i < a.vdim; i += 32) ss += o[i] * o[i];
  const float inv = rsqrtf(warp_sum(ss) / (float)a.vdim + a.eps);
  OutT* out = reinterpret_cast<OutT*>(a.out) + (size_t)w * a.vcols;
  for (int i = lane; i < a.vcols; i += 32) {
    float v = 0.f;
    if (i < a.vdim)
      v = o[i] * inv * (a.gain != nullptr ? a.gain[i] : 1.f) * la_silu(la_row(a, (size_t)t * a.stride + a.cz + h * a.vdim + i));
    if constexpr (sizeof(OutT) == 2) out[i] = f32_to_bf16(v);
    else out[i] = v;
  }
}

// ---------------------------------------------------------------- one token per segment
constexpr int STEP_THREADS = 512;

// grid (H, T); lanes per column: 4 up to 128 rows, 16 above
template <int DK, bool DELTA, typename OutT>
__global__ void __launch_bounds__(STEP_THREADS) linear_step_kernel(const __grid_constant__ LinearArgs a) {
  constexpr int L = DK <= 128 ? 4 : 16, RPL = DK / L, COLS = STEP_THREADS / L, KPAD = DK + 4 * L;
  extern __shared__ __align__(16) float dyn[];                 // values, outputs: vcols each
  __shared__ __align__(16) float sq[KPAD], sk[KPAD];
  __shared__ float raw[2][DK], red[33], gate[2];
  pdl_launch();
  const int h = blockIdx.x, t = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int grp = a.H / a.G, kh = h / grp;
  pdl_wait();
  const int slot = a.seg_slot[t], p = a.pos[t];
  if (!HE_INDEX_OK(slot, a.n_slots, HE_SITE_STATE_SLOT)) return;
  float* sv = dyn;
  float* so = dyn + a.vcols;
  // the state's rows are on their way while the token's rows are prepared
  const int cw = tid / L, ks = tid % L;
  float* Sg = a.S + ((size_t)slot * a.H + h) * a.dim * a.vcols;
  float S[RPL];
  const auto load = [&](int col) {
#pragma unroll
    for (int i = 0; i < RPL; ++i) {
      const int d = ks * RPL + i;
      S[i] = col < a.vcols && d < a.dim ? Sg[(size_t)d * a.vcols + col] : 0.f;
    }
  };
  load(cw);
  if (warp < 2) {
    la_prepare_head(a, t, t, slot, p, (warp == 0 ? 0 : a.ck) + kh * a.dim, warp == 0 ? a.qscale : a.kscale, raw[warp], lane);
    __syncwarp();
    float* dst = warp == 0 ? sq : sk;
    for (int d = lane; d < DK; d += 32) dst[d + (d / RPL) * 4] = d < a.dim ? raw[warp][d] : 0.f;
  } else {
    for (int d = tid - 64; d < a.vcols; d += STEP_THREADS - 64) {
      const int c = a.cv + h * a.vdim + d;
      sv[d] = d >= a.vdim ? 0.f : DELTA ? la_conv(a, t, t, slot, p, c) : la_row(a, (size_t)t * a.stride + c);
    }
    if (DELTA && tid == STEP_THREADS - 1) {
      gate[0] = expm1f(la_log_decay(a, t, h));
      gate[1] = la_beta(a, t, h);
    }
  }
  __syncthreads();
  const float g1 = DELTA ? gate[0] : a.gm[h];
  const float* kp = sk + ks * (RPL + 4);
  const float* qp = sq + ks * (RPL + 4);
  float ss = 0.f;
  for (int c0 = 0; c0 < a.vcols; c0 += COLS) {
    const int col = c0 + cw;
    const bool live = col < a.vcols;
    if (c0 > 0) load(col);
    float u = live ? sv[col] : 0.f;
    if constexpr (DELTA) {
      float p4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int i = 0; i < RPL; ++i) {
        S[i] = fmaf(g1, S[i], S[i]);
        p4[i & 3] += kp[i] * S[i];
      }
      float kv = (p4[0] + p4[1]) + (p4[2] + p4[3]);
#pragma unroll
      for (int o = 1; o < L; o <<= 1) kv += __shfl_xor_sync(0xffffffffu, kv, o);
      u = (u - kv) * gate[1];
    }
    float o4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int i = 0; i < RPL; ++i) {
      if (!DELTA) S[i] = fmaf(g1, S[i], S[i]);
      S[i] += kp[i] * u;
      o4[i & 3] += qp[i] * S[i];
    }
    float o = (o4[0] + o4[1]) + (o4[2] + o4[3]);
#pragma unroll
    for (int of = 1; of < L; of <<= 1) o += __shfl_xor_sync(0xffffffffu, o, of);
    if (live) {
#pragma unroll
      for (int i = 0; i < RPL; ++i)
        if (ks * RPL + i < a.dim) Sg[(size_t)(ks * RPL + i) * a.vcols + col] = S[i];
      if (ks == 0) {
        so[col] = o;
        if (col < a.vdim) ss += o * o;
      }
    }
  }
  const float inv = rsqrtf(block_sum(ss, red) / (float)a.vdim + a.eps);      // its barriers publish so[]
  OutT* out = reinterpret_cast<OutT*>(a.out) + ((size_t)t * a.H + h) * a.vcols;
  for (int i = tid; i < a.vcols; i += STEP_THREADS) {
    float v = 0.f;
    if (i < a.vdim)
      v = so[i] * inv * (a.gain != nullptr ? a.gain[i] : 1.f) * la_silu(la_row(a, (size_t)t * a.stride + a.cz + h * a.vdim + i));
    if constexpr (sizeof(OutT) == 2) out[i] = f32_to_bf16(v);
    else out[i] = v;
  }
  if (DELTA && a.taps > 1) {
    // own value columns, and the query and key columns for the first head that shares them
    for (int i = tid; i < a.vdim; i += STEP_THREADS) la_ring_update(a, slot, t, t + 1, a.cv + h * a.vdim + i);
    if (h % grp == 0)
      for (int i = tid; i < a.dim; i += STEP_THREADS) {
        la_ring_update(a, slot, t, t + 1, kh * a.dim + i);
        la_ring_update(a, slot, t, t + 1, a.ck + kh * a.dim + i);
      }
  }
}

int dk_of(int dim) { return dim <= 64 ? 64 : dim <= 128 ? 128 : dim <= 256 ? 256 : 512; }

int check(const LinearArgs& a) {
  if (a.H < 1 || a.G < 1 || a.H % a.G != 0 || a.dim < 1 || a.dim > 512 || a.vdim < 1 || a.vcols < a.vdim || a.vcols > 512 ||
      a.H > 65535 || a.T > 65535 * 1024 || (a.delta && (a.taps < 1 || (a.taps > 1 && a.ring == nullptr))) ||
      (!a.delta && (a.gm == nullptr || a.rot_dims > a.dim || a.rot_dims % 2 != 0)))
    return -HE_ERR_BAD_ARG;
  return 0;
}

template <int DK>
int launch_scan(const LinearArgs& a, cudaStream_t stream) {
  const dim3 grid(a.n_seg, a.H, (a.vcols + SLICE - 1) / SLICE), block(SLICE * LPC);
  return (int)(a.delta ? launch_pdl(linear_scan_kernel<DK, true>, grid, block, 0, stream, a)
                       : launch_pdl(linear_scan_kernel<DK, false>, grid, block, 0, stream, a));
}

template <int DK, typename OutT>
int launch_step(const LinearArgs& a, cudaStream_t stream) {
  const dim3 grid(a.H, a.T), block(STEP_THREADS);
  const size_t smem = 2 * (size_t)a.vcols * sizeof(float);
  return (int)(a.delta ? launch_pdl(linear_step_kernel<DK, true, OutT>, grid, block, smem, stream, a)
                       : launch_pdl(linear_step_kernel<DK, false, OutT>, grid, block, smem, stream, a));
}

template <typename OutT>
int dispatch_step(const LinearArgs& a, cudaStream_t stream) {
  switch (dk_of(a.dim)) {
    case 64: return launch_step<64, OutT>(a, stream);
    case 128: return launch_step<128, OutT>(a, stream);
    case 256: return launch_step<256, OutT>(a, stream);
    default: return launch_step<512, OutT>(a, stream);
  }
}

}  // namespace

HE_API int he_linear_prepare(const LinearArgs* args, cudaStream_t stream) {
  const LinearArgs& a = *args;
  if (a.T <= 0) return 0;
  if (check(a) != 0) return -HE_ERR_BAD_ARG;
  const long long warps = (long long)a.T * (2 * a.G + a.H + (a.delta ? 1 : 0));
  return (int)launch_pdl(linear_prepare_kernel, dim3((unsigned)((warps + 7) / 8)), dim3(256), 0, stream, a);
}

HE_API int he_linear_scan(const LinearArgs* args, cudaStream_t stream) {
  const LinearArgs& a = *args;
  if (a.T <= 0 || a.n_seg <= 0) return 0;
  if (check(a) != 0) return -HE_ERR_BAD_ARG;
  switch (dk_of(a.dim)) {
    case 64: return launch_scan<64>(a, stream);
    case 128: return launch_scan<128>(a, stream);
    case 256: return launch_scan<256>(a, stream);
    default: return launch_scan<512>(a, stream);
  }
}

HE_API int he_linear_out(const LinearArgs* args, cudaStream_t stream) {
  const LinearArgs& a = *args;
  if (a.T <= 0) return 0;
  const unsigned grid = (unsigned)(((long long)a.T * a.H + 7) / 8);
  return (int)(a.out_f32 ? launch_pdl(linear_out_kernel<float>, dim3(grid), dim3(256), 0, stream, a)
                         : launch_pdl(linear_out_kernel<__nv_bfloat16>, dim3(grid), dim3(256), 0, stream, a));
}

// Every segment has one token (T == n_seg); no journal.
HE_API int he_linear_step(const LinearArgs* args, cudaStream_t stream) {
  const LinearArgs& a = *args;
  if (a.T <= 0) return 0;
  if (check(a) != 0 || a.T != a.n_seg || a.T > 65535 || a.jS != nullptr) return -HE_ERR_BAD_ARG;
  return a.out_f32 ? dispatch_step<float>(a, stream) : dispatch_step<__nv_bfloat16>(a, stream);
}
HE_API int he_linear_args_size() { return (int)sizeof(LinearArgs); }
