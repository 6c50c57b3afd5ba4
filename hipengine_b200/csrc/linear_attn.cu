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
  if (a.vdim == 128 && a.row_dtype == 1 && sizeof(OutT) == 2 && a.stride % 4 == 0 && a.cz % 4 == 0) {        // four columns per lane
    const float4 x = *reinterpret_cast<const float4*>(o + lane * 4);
    const uint2 zr = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(a.rows) + (size_t)t * a.stride + a.cz + h * 128 + lane * 4);
    float4 g = make_float4(1.f, 1.f, 1.f, 1.f);
    if (a.gain != nullptr) g = make_float4(a.gain[lane * 4], a.gain[lane * 4 + 1], a.gain[lane * 4 + 2], a.gain[lane * 4 + 3]);
    const float inv = rsqrtf(warp_sum(x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w) / 128.f + a.eps);
    const float2 z0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&zr.x)),
                 z1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&zr.y));
    __align__(8) __nv_bfloat162 r2[2] = {__floats2bfloat162_rn(x.x * inv * g.x * silu_f(z0.x), x.y * inv * g.y * silu_f(z0.y)),
                                         __floats2bfloat162_rn(x.z * inv * g.z * silu_f(z1.x), x.w * inv * g.w * silu_f(z1.y))};
    *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(a.out) + (size_t)w * 128 + lane * 4) = *reinterpret_cast<const uint2*>(r2);
    return;
  }
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
constexpr int STEP_WARPS = 16, STEP_THREADS = STEP_WARPS * 32, STEP_COLS = 128;

// grid (H, T).  A warp owns rows of the state, a lane four of 128 columns: whole lines in and out; sums over the rows meet in shared
// memory.  NB > 1: more rows than the registers hold (NB blocks), read once for S^T k and once for the update.
template <int RW, int NB, bool DELTA, typename OutT>
__global__ void __launch_bounds__(STEP_THREADS, 2) linear_step_kernel(const __grid_constant__ LinearArgs a) {
  constexpr int DK = RW * STEP_WARPS * NB;
  extern __shared__ __align__(16) float dyn[];                 // values, outputs: vcols each
  __shared__ __align__(16) float part[STEP_WARPS][STEP_COLS];
  __shared__ __align__(16) float su[STEP_COLS];
  __shared__ float sq[DK], sk[DK], red[33], gate[2], unit[2];
  pdl_launch();
  const int h = blockIdx.x, t = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int grp = a.H / a.G, kh = h / grp;
  pdl_wait();
  const int slot = a.seg_slot[t], p = a.pos[t];
  if (!HE_INDEX_OK(slot, a.n_slots, HE_SITE_STATE_SLOT)) return;
  float* sv = dyn;
  float* so = dyn + a.vcols;
  float* Sg = a.S + ((size_t)slot * a.H + h) * a.dim * a.vcols;
  float4 S[RW];
  const auto load = [&](int block, int col) {
#pragma unroll
    for (int i = 0; i < RW; ++i) {
      const int d = (block * STEP_WARPS + warp) * RW + i;
      S[i] = col < a.vcols && d < a.dim ? *reinterpret_cast<const float4*>(Sg + (size_t)d * a.vcols + col) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  // the state's rows are on their way while the token's rows are prepared
  if constexpr (NB == 1) load(0, lane * 4);
  const size_t row0 = (size_t)t * a.stride;
  if constexpr (DELTA) {
    // a channel of query, key or value per thread; the ring's entry of `back` tokens ago lies at (p - back) % taps
    const int e0 = p % a.taps, total = 2 * a.dim + a.vcols;
    const float* ring = a.taps > 1 ? a.ring + (size_t)slot * a.taps * a.C : nullptr;
    for (int i = tid; i < total; i += STEP_THREADS) {
      const int d = i < a.dim ? i : i < 2 * a.dim ? i - a.dim : i - 2 * a.dim;
      float v = 0.f;
      if (i < 2 * a.dim || d < a.vdim) {
        const int c = (i < a.dim ? kh * a.dim : i < 2 * a.dim ? a.ck + kh * a.dim : a.cv + h * a.vdim) + d;
        float acc = 0.f;
#pragma unroll 4
        for (int back = a.taps - 1; back > 0; --back)
          if (p >= back) acc += a.cw[(size_t)(a.taps - 1 - back) * a.C + c] * ring[(size_t)(e0 >= back ? e0 - back : e0 - back + a.taps) * a.C + c];
        v = la_silu(acc + a.cw[(size_t)(a.taps - 1) * a.C + c] * la_row(a, row0 + c));
      }
      if (i < a.dim) sq[d] = v;
      else if (i < 2 * a.dim) sk[d] = v;
      else sv[d] = v;
    }
    if (tid == STEP_THREADS - 1) {
      gate[0] = expm1f(la_log_decay(a, t, h));
      gate[1] = la_beta(a, t, h);
    }
  } else {
    const int half = a.rot_dims >> 1;
    for (int i = tid; i < 2 * half; i += STEP_THREADS) {       // pairs of the query, then of the key
      const bool key = i >= half;
      const int j = key ? i - half : i;
      const size_t c0 = row0 + (key ? a.ck : 0) + kh * a.dim + j;
      const float u = la_row(a, c0), v = la_row(a, c0 + half);
      float c, s;
      la_angle(a.freq[j], p, c, s);
      float* dst = key ? sk : sq;
      dst[j] = u * c - v * s;
      dst[half + j] = v * c + u * s;
    }
    for (int d = a.rot_dims + tid; d < a.dim; d += STEP_THREADS) {
      sq[d] = la_row(a, row0 + kh * a.dim + d);
      sk[d] = la_row(a, row0 + a.ck + kh * a.dim + d);
    }
    for (int d = STEP_THREADS - 1 - tid; d < a.vcols; d += STEP_THREADS)
      sv[d] = d < a.vdim ? la_row(a, row0 + a.cv + h * a.vdim + d) : 0.f;
  }
  for (int d = a.dim + tid; d < DK; d += STEP_THREADS) sq[d] = sk[d] = 0.f;
  __syncthreads();
  if (DELTA && warp < 2) {                                     // unit length: factors of query and key
    const float* x = warp == 0 ? sq : sk;
    float ss = 0.f;
    for (int d = lane; d < a.dim; d += 32) ss += x[d] * x[d];
    ss = warp_sum(ss);
    if (lane == 0) unit[warp] = (warp == 0 ? a.qscale : a.kscale) / sqrtf(ss + 1e-6f);
  }
  if (DELTA) __syncthreads();
  const float qs = DELTA ? unit[0] : a.qscale, ks = DELTA ? unit[1] : a.kscale, g1 = DELTA ? gate[0] : a.gm[h];
  float ss = 0.f;
  for (int c0 = 0; c0 < a.vcols; c0 += STEP_COLS) {
    const int col = c0 + lane * 4, mine = c0 + tid;            // columns of the lane; column summed up by the thread
    if constexpr (DELTA) {
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int nb = 0; nb < NB; ++nb) {
        if (NB > 1 || c0 > 0) load(nb, col);
#pragma unroll
        for (int i = 0; i < RW; ++i) {
          S[i].x = fmaf(g1, S[i].x, S[i].x); S[i].y = fmaf(g1, S[i].y, S[i].y);
          S[i].z = fmaf(g1, S[i].z, S[i].z); S[i].w = fmaf(g1, S[i].w, S[i].w);
          const float k = sk[(nb * STEP_WARPS + warp) * RW + i];
          acc.x += k * S[i].x; acc.y += k * S[i].y; acc.z += k * S[i].z; acc.w += k * S[i].w;
        }
      }
      *reinterpret_cast<float4*>(&part[warp][lane * 4]) = acc;
      __syncthreads();
      if (tid < STEP_COLS) {
        float kv = 0.f;
#pragma unroll
        for (int w = 0; w < STEP_WARPS; ++w) kv += part[w][tid];
        su[tid] = mine < a.vcols ? (sv[mine] - ks * kv) * gate[1] * ks : 0.f;
      }
    } else {
      if (tid < STEP_COLS) su[tid] = mine < a.vcols ? sv[mine] * ks : 0.f;
    }
    __syncthreads();
    const float4 u = *reinterpret_cast<const float4*>(su + lane * 4);
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int nb = 0; nb < NB; ++nb) {
      const bool fresh = NB > 1 || (!DELTA && c0 > 0);
      if (fresh) load(nb, col);
#pragma unroll
      for (int i = 0; i < RW; ++i) {
        const int d = (nb * STEP_WARPS + warp) * RW + i;
        if (fresh || !DELTA) {
          S[i].x = fmaf(g1, S[i].x, S[i].x); S[i].y = fmaf(g1, S[i].y, S[i].y);
          S[i].z = fmaf(g1, S[i].z, S[i].z); S[i].w = fmaf(g1, S[i].w, S[i].w);
        }
        const float k = sk[d], q = sq[d];
        S[i].x += k * u.x; S[i].y += k * u.y; S[i].z += k * u.z; S[i].w += k * u.w;
        acc.x += q * S[i].x; acc.y += q * S[i].y; acc.z += q * S[i].z; acc.w += q * S[i].w;
        if (col < a.vcols && d < a.dim) *reinterpret_cast<float4*>(Sg + (size_t)d * a.vcols + col) = S[i];
      }
    }
    *reinterpret_cast<float4*>(&part[warp][lane * 4]) = acc;
    __syncthreads();
    if (tid < STEP_COLS && mine < a.vcols) {
      float o = 0.f;
#pragma unroll
      for (int w = 0; w < STEP_WARPS; ++w) o += part[w][tid];
      o *= qs;
      so[mine] = o;
      if (mine < a.vdim) ss += o * o;
    }
    if (c0 + STEP_COLS < a.vcols) __syncthreads();             // part and su are written again
  }
  const float inv = rsqrtf(block_sum(ss, red) / (float)a.vdim + a.eps);      // its barriers publish so[]
  OutT* out = reinterpret_cast<OutT*>(a.out) + ((size_t)t * a.H + h) * a.vcols;
  for (int i = tid; i < a.vcols; i += STEP_THREADS) {
    float v = 0.f;
    if (i < a.vdim)
      v = so[i] * inv * (a.gain != nullptr ? a.gain[i] : 1.f) * la_silu(la_row(a, row0 + a.cz + h * a.vdim + i));
    if constexpr (sizeof(OutT) == 2) out[i] = f32_to_bf16(v);
    else out[i] = v;
  }
  if (DELTA && a.taps > 1) {
    // own value columns, and the query and key columns for the first head that shares them
    for (int i = tid; i < a.vdim; i += STEP_THREADS) la_ring_update(a, slot, t, t + 1, a.cv + h * a.vdim + i);
    if (h % grp == 0)
      for (int i = tid; i < 2 * a.dim; i += STEP_THREADS)
        la_ring_update(a, slot, t, t + 1, (i < a.dim ? i : a.ck + i - a.dim) + kh * a.dim);
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

template <int RW, int NB, typename OutT>
int launch_step(const LinearArgs& a, cudaStream_t stream) {
  const dim3 grid(a.H, a.T), block(STEP_THREADS);
  const size_t smem = 2 * (size_t)a.vcols * sizeof(float);
  return (int)(a.delta ? launch_pdl(linear_step_kernel<RW, NB, true, OutT>, grid, block, smem, stream, a)
                       : launch_pdl(linear_step_kernel<RW, NB, false, OutT>, grid, block, smem, stream, a));
}

template <typename OutT>
int dispatch_step(const LinearArgs& a, cudaStream_t stream) {
  switch (dk_of(a.dim)) {
    case 64: return launch_step<4, 1, OutT>(a, stream);
    case 128: return launch_step<8, 1, OutT>(a, stream);
    case 256: return launch_step<8, 2, OutT>(a, stream);
    default: return launch_step<8, 4, OutT>(a, stream);
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
