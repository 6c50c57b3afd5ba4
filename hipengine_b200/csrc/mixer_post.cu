// What happens between a layer's input projections and its mixers, in one launch: query / key / value rows get their
// biases, norm and rotation and go to the query buffer and the pages; the inputs of a recurrence go through its short causal
// convolution.
//
// grid: T * (query parts + key parts + value parts) CTAs of one token and a range of heads (staged in shared memory, a warp per
// head; a lane keeps the sines and cosines of its dimensions over the heads), then the convolution's CTAs of 1024 channels
// and one or several tokens.  Norms: per head or over the whole projection before the rotation (with
// gains), or per head after it (without).  The rotation turns (i, i + n/2) or (2i, 2i + 1) by table frequencies; angles
// are reduced to one turn in double.  The convolution's state is only read here: the recurrence, which runs later in stream
// order, replaces it.
#include "common.cuh"

using namespace he;

struct HeadRows {
  const void* x;             // [T][stride], null: none
  long long stride;          // multiple of 8, as is the column the rows start at; columns are zero-padded to a multiple of 8
  const float* bias;         // [heads * dim, padded] or null
  const float* gain;         // norm 1: [dim] or, with gain_heads, [heads][dim]; norm 2: [heads * dim, padded]
  int heads, dim, gain_heads;
};

struct MixerPostArgs {
  HeadRows q, k, v;          // k without v: the biased keys, before norm and rotation, are the values
  const double* freq;        // [rot_dims / 2]
  void* q_out;               // [T][H][D]
  void* kv_cache;            // [n_pages][2][Hkv][page][D]
  const int* block_table;    // [n_slots][max_pages]
  const int* slot;           // [T]
  const int* pos;            // [T]
  // convolution
  const void* cx;            // [T][cx_stride] inputs without bias, null: none
  long long cx_stride;
  const float* cx_bias;      // [C]
  const float* cw;           // [taps][C], oldest first
  const float* cb;           // [C]
  const float* cstate;       // [n_slots][taps - 1][C] biased inputs ahead of the segment, oldest first
  float* cjournal;           // [T][taps - 1][C] the state after every token, or null
  const int* seg_start;      // [n_seg + 1]
  const int* seg_slot;       // [n_seg]
  const int* tok_seg;        // [T]
  void* u;                   // block b, token t, channel c of the block at b * u_bs + t * u_ts + c
  long long u_ts, u_bs;
  int C, block_cols, taps, n_slots;
  int T, in_dtype, out_f32;  // 0 f32, 1 bf16; q_out, kv_cache and u in fp32
  int norm;                  // 0 none, 1 per head, 2 whole projection, 3 per head after the rotation
  int rot_dims, halves;
  int D, page, max_pages, heads_per_cta, conv_tokens;
  float eps, amp;
};

namespace {

constexpr int NTHR = 256;
constexpr int CONV_CHANNELS = NTHR * 4;
constexpr int CONV_TOKENS = 8;     // of a convolution CTA in long batches
constexpr int MAX_PAIRS = 8;       // head widths up to 512: a lane owns up to eight neighbouring pairs

__device__ __forceinline__ float4 load4(const void* p, int dtype, size_t i) {
  if (dtype == 0) return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + i);
  const uint2 v = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(p) + i);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&v);
  const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
template <typename OutT>
__device__ __forceinline__ void store4(OutT* p, float4 v) {
  if constexpr (sizeof(OutT) == 2) {
    __align__(8) __nv_bfloat162 b[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
    *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(b);
  } else {
    *reinterpret_cast<float4*>(p) = v;
  }
}
template <typename OutT>
__device__ __forceinline__ void store2(OutT* p, float a, float b) {
  if constexpr (sizeof(OutT) == 2) *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
  else *reinterpret_cast<float2*>(p) = make_float2(a, b);
}

// sum of squares of columns [0, n) of four at i
__device__ __forceinline__ float sq_upto(float4 v, int i, int n) {
  float s = i < n ? v.x * v.x : 0.f;
  if (i + 1 < n) s += v.y * v.y;
  if (i + 2 < n) s += v.z * v.z;
  if (i + 3 < n) s += v.w * v.w;
  return s;
}

// 1024 channels of `a.conv_tokens` tokens.  TAPS > 0: filter and window in registers.
template <typename OutT, int TAPS>
__device__ __forceinline__ void conv_part(const MixerPostArgs& a, int index) {
  const int chunks = (a.C + CONV_CHANNELS - 1) / CONV_CHANNELS;
  const int c = (index % chunks) * CONV_CHANNELS + threadIdx.x * 4, t0 = (index / chunks) * a.conv_tokens;
  if (c >= a.C) return;
  const int taps = TAPS > 0 ? TAPS : a.taps, past = taps - 1, t1 = min(a.T, t0 + a.conv_tokens);
  const float4 xb = *reinterpret_cast<const float4*>(a.cx_bias + c), bias = *reinterpret_cast<const float4*>(a.cb + c);
  OutT* out = reinterpret_cast<OutT*>(a.u) + (size_t)(c / a.block_cols) * a.u_bs + c % a.block_cols;
  float4 w[TAPS > 0 ? TAPS : 1], win[TAPS > 0 ? TAPS : 1];
  if constexpr (TAPS > 0)
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j] = *reinterpret_cast<const float4*>(a.cw + (size_t)j * a.C + c);
  int seg = -1, s0 = 0, slot = 0;
  for (int t = t0; t < t1; ++t) {
    const int sg = a.tok_seg[t];
    const bool first = sg != seg;
    if (first) {
      seg = sg;
      s0 = a.seg_start[sg];
      slot = a.seg_slot[sg];
    }
    if (!HE_INDEX_OK(slot, a.n_slots, HE_SITE_STATE_SLOT)) continue;
    // input `idx` of [state ++ segment], counted from the oldest one that this token needs
    const auto input = [&](int j) -> float4 {
      const int idx = t - s0 + j;
      return idx < past ? *reinterpret_cast<const float4*>(a.cstate + ((size_t)slot * past + idx) * a.C + c)
                        : add4(load4(a.cx, a.in_dtype, (size_t)(s0 + idx - past) * a.cx_stride + c), xb);
    };
    const auto journal = [&](int j, float4 x) {
      if (a.cjournal != nullptr && j > 0) *reinterpret_cast<float4*>(a.cjournal + ((size_t)t * past + j - 1) * a.C + c) = x;
    };
    float4 acc = bias;
    const auto tap = [&](float4 f, float4 x) {
      acc.x += f.x * x.x; acc.y += f.y * x.y; acc.z += f.z * x.z; acc.w += f.w * x.w;
    };
    if constexpr (TAPS > 0) {
#pragma unroll
      for (int j = 0; j < TAPS; ++j) win[j] = first || j == TAPS - 1 ? input(j) : win[j + 1];
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        tap(w[j], win[j]);
        journal(j, win[j]);
      }
    } else {
      for (int j = 0; j < taps; ++j) {
        const float4 x = input(j);
        tap(*reinterpret_cast<const float4*>(a.cw + (size_t)j * a.C + c), x);
        journal(j, x);
      }
    }
    store4(out + (size_t)t * a.u_ts, acc);
  }
}

template <typename OutT, int NP>
__global__ void __launch_bounds__(NTHR, NP <= 2 ? 4 : 2) mixer_post_kernel(const __grid_constant__ MixerPostArgs a) {
  extern __shared__ __align__(16) float sm[];    // [rot_dims] (cos, sin) pairs, then the staged columns
  __shared__ float red[33];
  pdl_launch();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, D = a.D;
  const auto parts = [&](const HeadRows& r) { return r.x == nullptr ? 0 : (r.heads + a.heads_per_cta - 1) / a.heads_per_cta; };
  const int nq = parts(a.q), nk = parts(a.k), np = nq + nk + parts(a.v);
  if ((int)blockIdx.x >= a.T * np) {
    const int i = blockIdx.x - a.T * np;
    pdl_wait();
    if (a.taps == 4) conv_part<OutT, 4>(a, i);
    else if (a.taps == 3) conv_part<OutT, 3>(a, i);
    else if (a.taps == 2) conv_part<OutT, 2>(a, i);
    else conv_part<OutT, 0>(a, i);
    return;
  }
  const int t = blockIdx.x / np;
  int y = blockIdx.x - t * np, kind = 0;         // 0 query, 1 key, 2 value
  if (y >= nq + nk) { kind = 2; y -= nq + nk; }
  else if (y >= nq) { kind = 1; y -= nq; }
  const HeadRows& r = kind == 0 ? a.q : kind == 1 ? a.k : a.v;
  const int h0 = y * a.heads_per_cta, nh = min(a.heads_per_cta, r.heads - h0), dim = r.dim;
  const int c0 = h0 * dim, n = nh * dim, all = r.heads * dim;
  const bool turned = kind < 2 && a.rot_dims > 0;
  const int norm = kind < 2 ? a.norm : 0, half = a.rot_dims >> 1;
  // columns [lo, hi) are read (the whole projection where its norm needs it), [c0, c0 + n) are kept; the first 4096 are
  // requested before the angles are computed, and what does not depend on earlier kernels before these end
  const int lo = norm == 2 ? 0 : c0, hi = norm == 2 ? all : c0 + n;
  constexpr int PRE = 4;
  float4 pre[PRE], pre_b[PRE];
  const auto bias = [&](int i) { return r.bias != nullptr ? *reinterpret_cast<const float4*>(r.bias + i) : make_float4(0.f, 0.f, 0.f, 0.f); };
#pragma unroll
  for (int k = 0; k < PRE; ++k) {
    const int i = lo + (threadIdx.x + k * NTHR) * 4;
    if (i < hi) pre_b[k] = bias(i);
  }
  const double freq0 = turned && (int)threadIdx.x < half ? a.freq[threadIdx.x] : 0.0;
  pdl_wait();
  const int p = a.pos[t];
  size_t row0 = 0;                               // of the key or value rows in the pages
  if (kind > 0) {
    const int pi = p / a.page;
    if (!HE_INDEX_OK(pi, a.max_pages, HE_SITE_KV_WRITE_PAGE)) return;       // uniform over the CTA
    const int pg = a.block_table[(size_t)a.slot[t] * a.max_pages + pi], hkv = r.heads;
    row0 = (((size_t)pg * 2 * hkv + h0) * a.page + p % a.page) * D;
  }
  float* cols = sm + ((a.rot_dims + 3) & ~3);
  const size_t in0 = (size_t)t * r.stride;
#pragma unroll
  for (int k = 0; k < PRE; ++k) {
    const int i = lo + (threadIdx.x + k * NTHR) * 4;
    if (i < hi) pre[k] = load4(r.x, a.in_dtype, in0 + i);
  }
  if (turned)
    for (int i = threadIdx.x; i < half; i += NTHR) {
      const double two_pi = 6.283185307179586476925286766559, per_turn = 0.15915494309189533576888376337251;
      const double ang = (double)p * (i < NTHR ? freq0 : a.freq[i]);
      float sn, c;
      sincosf((float)(ang - two_pi * rint(ang * per_turn)), &sn, &c);
      sm[2 * i] = c * a.amp;
      sm[2 * i + 1] = sn * a.amp;
    }
  float ss = 0.f;
  const auto keep = [&](int i, float4 v) {
    if (i >= c0 && i < c0 + n) *reinterpret_cast<float4*>(cols + i - c0) = v;
    ss += sq_upto(v, i, hi);
  };
#pragma unroll
  for (int k = 0; k < PRE; ++k) {
    const int i = lo + (threadIdx.x + k * NTHR) * 4;
    if (i < hi) keep(i, add4(pre[k], pre_b[k]));
  }
  for (int i = lo + (threadIdx.x + PRE * NTHR) * 4; i < hi; i += NTHR * 4)
    keep(i, add4(load4(r.x, a.in_dtype, in0 + i), bias(i)));
  float inv_all = 1.f;
  if (norm == 2) inv_all = rsqrtf(block_sum(ss, red) / (float)all + a.eps);
  __syncthreads();

  // value of dimension d = c * x[d] + s * x[partner]; both of a lane's neighbouring dimensions are turned or none is
  float2 cs[NP][2];
#pragma unroll
  for (int j = 0; j < NP; ++j) {
    const int d = lane * 2 + 64 * j;
    cs[j][0] = cs[j][1] = make_float2(1.f, 0.f);
    if (turned && d < a.rot_dims) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int i = a.halves ? (d + e < half ? d + e : d + e - half) : (d >> 1);
        const bool lower = a.halves ? d + e < half : e == 0;
        cs[j][e] = make_float2(sm[2 * i], lower ? -sm[2 * i + 1] : sm[2 * i + 1]);
      }
    }
  }
  const bool pairs = (dim & 1) == 0 && (!turned || !a.halves || (half & 1) == 0);   // two dimensions and their partners are neighbours
  const size_t plane = (size_t)r.heads * a.page * D;                         // from a key row to its value row
  for (int h = warp; h < nh; h += NTHR / 32) {
    float* x = cols + h * dim;
    const size_t out0 = kind == 0 ? ((size_t)t * r.heads + h0 + h) * D : row0 + (size_t)h * a.page * D;
    if (kind == 1 && a.v.x == nullptr)
      for (int d = lane * 2; d < D; d += 64)
        store2(reinterpret_cast<OutT*>(a.kv_cache) + out0 + plane + d, d < dim ? x[d] : 0.f, d + 1 < dim ? x[d + 1] : 0.f);
    __syncwarp();
    if (norm == 1 || norm == 2) {
      float inv = inv_all;
      const float* gain = norm == 1 && r.gain_heads == 0 ? r.gain : r.gain + c0 + h * dim;
      if (norm == 1) {
        float s = 0.f;
        for (int d = lane; d < dim; d += 32) s += x[d] * x[d];
        inv = rsqrtf(warp_sum(s) / (float)dim + a.eps);
      }
      for (int d = lane; d < dim; d += 32) x[d] *= inv * gain[d];
      __syncwarp();
    }
    float v[NP][2], s = 0.f;
#pragma unroll
    for (int j = 0; j < NP; ++j) {
      const int d = lane * 2 + 64 * j;
      v[j][0] = v[j][1] = 0.f;
      if (d >= dim) continue;
      const bool mine = turned && d < a.rot_dims;
      if (pairs) {
        const float2 own = *reinterpret_cast<const float2*>(x + d);
        float2 other = own;
        if (mine) {
          other = *reinterpret_cast<const float2*>(x + (!a.halves ? d : d < half ? d + half : d - half));
          if (!a.halves) other = make_float2(own.y, own.x);
        }
        v[j][0] = cs[j][0].x * own.x + cs[j][0].y * other.x;
        v[j][1] = cs[j][1].x * own.y + cs[j][1].y * other.y;
      } else {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          if (d + e >= dim) continue;
          float other = 0.f;
          if (mine) other = x[!a.halves ? d + (e ^ 1) : d + e < half ? d + e + half : d + e - half];
          v[j][e] = cs[j][e].x * x[d + e] + cs[j][e].y * other;
        }
      }
      s += v[j][0] * v[j][0] + v[j][1] * v[j][1];
    }
    const float inv = norm == 3 ? rsqrtf(warp_sum(s) / (float)dim + a.eps) : 1.f;
    OutT* out = reinterpret_cast<OutT*>(kind == 0 ? a.q_out : a.kv_cache) + out0 + (kind == 2 ? plane : 0);
#pragma unroll
    for (int j = 0; j < NP; ++j)
      if (64 * j < D) store2(out + lane * 2 + 64 * j, v[j][0] * inv, v[j][1] * inv);
  }
}

template <int NP>
int launch(const MixerPostArgs& a, dim3 grid, dim3 block, size_t smem, cudaStream_t stream) {
  return (int)(a.out_f32 ? launch_pdl(mixer_post_kernel<float, NP>, grid, block, smem, stream, a)
                         : launch_pdl(mixer_post_kernel<__nv_bfloat16, NP>, grid, block, smem, stream, a));
}

}  // namespace

HE_API int he_mixer_post(const MixerPostArgs* args, cudaStream_t stream) {
  MixerPostArgs a = *args;
  if (a.T <= 0) return 0;
  if (a.D % 64 != 0 || a.D > 64 * MAX_PAIRS || a.rot_dims < 0 || a.rot_dims % 2 != 0 || a.norm < 0 || a.norm > 3)
    return -HE_ERR_BAD_ARG;
  int widest = 1, most = 1;
  const HeadRows* rows[3] = {&a.q, &a.k, &a.v};
  for (int i = 0; i < 3; ++i) {
    const HeadRows& r = *rows[i];
    if (r.x == nullptr) continue;
    if (r.heads < 1 || r.dim < 1 || r.dim > a.D || r.stride % 8 != 0 || (i < 2 && a.rot_dims > r.dim)) return -HE_ERR_BAD_ARG;
    if (i < 2 && (a.norm == 1 || a.norm == 2) && r.gain == nullptr) return -HE_ERR_BAD_ARG;
    widest = r.dim > widest ? r.dim : widest;
    most = r.heads > most ? r.heads : most;
  }
  if (a.q.x == nullptr || (a.v.x != nullptr && (a.k.x == nullptr || a.v.heads != a.k.heads))) return -HE_ERR_BAD_ARG;
  if (a.k.x != nullptr && a.v.x == nullptr && a.norm == 2) return -HE_ERR_BAD_ARG;    // the plain keys are gone by then
  int conv = 0;
  if (a.cx != nullptr) {
    if (a.C % 8 != 0 || a.block_cols % 8 != 0 || a.taps < 1 || a.cx_stride % 8 != 0 || a.u_ts % 4 != 0 || a.u_bs % 4 != 0)
      return -HE_ERR_BAD_ARG;
    conv = (a.C + CONV_CHANNELS - 1) / CONV_CHANNELS;
  }
  // few tokens: a warp per head; many: all heads of a token in one CTA, as far as shared memory goes
  const int fit = (44 * 1024 / 4 - a.rot_dims - 16) / widest;
  int per = a.T < 148 ? 8 : most;
  if (per > fit) per = fit & ~7;
  if (per > most) per = most;
  if (per < 1) return -HE_ERR_BAD_ARG;
  a.heads_per_cta = per;
  a.conv_tokens = a.T < 148 ? 1 : CONV_TOKENS;
  const auto parts = [&](const HeadRows& r) { return r.x == nullptr ? 0 : (r.heads + per - 1) / per; };
  const size_t smem = (size_t)(((a.rot_dims + 3) & ~3) + per * widest + 8) * sizeof(float);
  const long long ctas = (long long)a.T * (parts(a.q) + parts(a.k) + parts(a.v)) +
                         (long long)conv * ((a.T + a.conv_tokens - 1) / a.conv_tokens);
  if (ctas > 0x7fffffffLL) return -HE_ERR_BAD_ARG;
  const dim3 grid((unsigned)ctas), block(NTHR);
  switch (a.D / 64) {
    case 1: return launch<1>(a, grid, block, smem, stream);
    case 2: return launch<2>(a, grid, block, smem, stream);
    case 3: case 4: return launch<4>(a, grid, block, smem, stream);
    default: return launch<8>(a, grid, block, smem, stream);
  }
}
HE_API int he_mixer_post_args_size() { return (int)sizeof(MixerPostArgs); }
