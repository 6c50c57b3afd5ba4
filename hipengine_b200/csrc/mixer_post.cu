// What happens between a layer's input projections and its mixers, in one launch: query / key / value rows get their
// biases, norm and rotation and go to the query buffer and the pages; the inputs of a recurrence go through its short causal
// convolution.
//
// grid (T, query parts + key parts + value parts + convolution parts): a CTA takes one token and a range of heads (staged in
// shared memory, a warp per head) or 1024 channels.  Norms: per head or over the whole projection before the rotation (with
// gains), or per head after it (without).  The rotation turns (i, i + n/2) or (2i, 2i + 1) by table frequencies; angles
// are reduced to one turn in double.  The convolution's state is only read here: the recurrence, which runs later in stream
// order, replaces it.
#include "common.cuh"

using namespace he;

struct HeadRows {
  const void* x;             // [T][stride], null: none
  long long stride;          // multiple of 8, as is the column the rows start at; columns are zero-padded to a multiple of 8
  const float* bias;         // [heads * dim, padded] or null
  const float* gain;         // norm 1: [dim], norm 2: [heads * dim, padded]
  int heads, dim;
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
  int D, page, max_pages, heads_per_cta;
  float eps, amp;
};

namespace {

constexpr int NTHR = 256;
constexpr int CONV_CHANNELS = NTHR * 4;
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

template <typename OutT>
__device__ __forceinline__ void conv_part(const MixerPostArgs& a, int t, int chunk) {
  const int c = chunk * CONV_CHANNELS + threadIdx.x * 4;
  if (c >= a.C) return;
  const int sg = a.tok_seg[t], s0 = a.seg_start[sg], slot = a.seg_slot[sg], local = t - s0, past = a.taps - 1;
  if (!HE_INDEX_OK(slot, a.n_slots, HE_SITE_STATE_SLOT)) return;
  const float4 xb = *reinterpret_cast<const float4*>(a.cx_bias + c);
  float4 acc = *reinterpret_cast<const float4*>(a.cb + c);
  for (int j = 0; j < a.taps; ++j) {
    const int idx = local + j;                   // of [state ++ segment]
    const float4 w = *reinterpret_cast<const float4*>(a.cw + (size_t)j * a.C + c);
    const float4 x = idx < past ? *reinterpret_cast<const float4*>(a.cstate + ((size_t)slot * past + idx) * a.C + c)
                                : add4(load4(a.cx, a.in_dtype, (size_t)(s0 + idx - past) * a.cx_stride + c), xb);
    acc.x += w.x * x.x; acc.y += w.y * x.y; acc.z += w.z * x.z; acc.w += w.w * x.w;
    if (a.cjournal != nullptr && j > 0) *reinterpret_cast<float4*>(a.cjournal + ((size_t)t * past + j - 1) * a.C + c) = x;
  }
  store4(reinterpret_cast<OutT*>(a.u) + (size_t)(c / a.block_cols) * a.u_bs + (size_t)t * a.u_ts + c % a.block_cols, acc);
}

template <typename OutT>
__global__ void __launch_bounds__(NTHR) mixer_post_kernel(const __grid_constant__ MixerPostArgs a) {
  extern __shared__ __align__(16) float sm[];    // [rot_dims] (cos, sin) pairs, then the staged columns
  __shared__ float red[33];
  pdl_wait();
  pdl_launch();
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, D = a.D;
  int y = blockIdx.y, kind = 0;                  // 0 query, 1 key, 2 value
  const auto parts = [&](const HeadRows& r) { return r.x == nullptr ? 0 : (r.heads + a.heads_per_cta - 1) / a.heads_per_cta; };
  const int nq = parts(a.q), nk = parts(a.k), nv = parts(a.v);
  if (y >= nq + nk + nv) {
    conv_part<OutT>(a, t, y - nq - nk - nv);
    return;
  }
  if (y >= nq + nk) { kind = 2; y -= nq + nk; }
  else if (y >= nq) { kind = 1; y -= nq; }
  const HeadRows& r = kind == 0 ? a.q : kind == 1 ? a.k : a.v;
  const int h0 = y * a.heads_per_cta, nh = min(a.heads_per_cta, r.heads - h0), dim = r.dim;
  const int c0 = h0 * dim, n = nh * dim, all = r.heads * dim;
  const bool turned = kind < 2 && a.rot_dims > 0;
  const int norm = kind < 2 ? a.norm : 0, p = a.pos[t], half = a.rot_dims >> 1;
  size_t row0 = 0;                               // of the key or value rows in the pages
  if (kind > 0) {
    const int pi = p / a.page;
    if (!HE_INDEX_OK(pi, a.max_pages, HE_SITE_KV_WRITE_PAGE)) return;       // uniform over the CTA
    const int pg = a.block_table[(size_t)a.slot[t] * a.max_pages + pi], hkv = r.heads;
    row0 = (((size_t)pg * 2 * hkv + h0) * a.page + p % a.page) * D;
  }
  float* cols = sm + ((a.rot_dims + 3) & ~3);
  const size_t in0 = (size_t)t * r.stride;
  float ss = 0.f;
  for (int i = threadIdx.x * 4; i < n; i += NTHR * 4) {
    float4 v = load4(r.x, a.in_dtype, in0 + c0 + i);
    if (r.bias != nullptr) v = add4(v, *reinterpret_cast<const float4*>(r.bias + c0 + i));
    *reinterpret_cast<float4*>(cols + i) = v;
    ss += sq_upto(v, i, n);
  }
  if (turned)
    for (int i = threadIdx.x; i < half; i += NTHR) {
      const double two_pi = 6.283185307179586476925286766559;
      const double ang = (double)p * a.freq[i];
      float sn, c;
      sincosf((float)(ang - two_pi * rint(ang / two_pi)), &sn, &c);
      sm[2 * i] = c * a.amp;
      sm[2 * i + 1] = sn * a.amp;
    }
  if (norm == 2) {
    if (n < all) {                               // a part of the heads: the squares of the whole projection again
      ss = 0.f;
      for (int i = threadIdx.x * 4; i < all; i += NTHR * 4) {
        float4 v = load4(r.x, a.in_dtype, in0 + i);
        if (r.bias != nullptr) v = add4(v, *reinterpret_cast<const float4*>(r.bias + i));
        ss += sq_upto(v, i, all);
      }
    }
    const float inv = rsqrtf(block_sum(ss, red) / (float)all + a.eps);
    for (int i = threadIdx.x * 4; i < n; i += NTHR * 4) {                   // the columns this thread staged
      float4 v = *reinterpret_cast<float4*>(cols + i);
      const float4 g = *reinterpret_cast<const float4*>(r.gain + c0 + i);
      *reinterpret_cast<float4*>(cols + i) = make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w);
    }
  }
  __syncthreads();

  for (int h = warp; h < nh; h += NTHR / 32) {
    float* x = cols + h * dim;
    const size_t out0 = kind == 0 ? ((size_t)t * r.heads + h0 + h) * D : row0 + (size_t)h * a.page * D;
    const size_t plane = (size_t)r.heads * a.page * D;                       // from a key row to its value row
    if (kind == 1 && a.v.x == nullptr)
      for (int d = lane * 2; d < D; d += 64)
        store2(reinterpret_cast<OutT*>(a.kv_cache) + out0 + plane + d, d < dim ? x[d] : 0.f, d + 1 < dim ? x[d + 1] : 0.f);
    __syncwarp();
    if (norm == 1) {
      float s = 0.f;
      for (int d = lane; d < dim; d += 32) s += x[d] * x[d];
      const float inv = rsqrtf(warp_sum(s) / (float)dim + a.eps);
      for (int d = lane; d < dim; d += 32) x[d] *= inv * r.gain[d];
    }
    __syncwarp();
    const auto value = [&](int d) -> float {
      if (d >= dim) return 0.f;
      const float v = x[d];
      if (!turned || d >= a.rot_dims) return v;
      if (a.halves) {
        const int i = d < half ? d : d - half;
        const float c = sm[2 * i], s = sm[2 * i + 1];
        return d < half ? v * c - x[d + half] * s : v * c + x[i] * s;
      }
      const float c = sm[d & ~1], s = sm[d | 1];
      return (d & 1) == 0 ? v * c - x[d + 1] * s : v * c + x[d - 1] * s;
    };
    float v[MAX_PAIRS][2], s = 0.f;
#pragma unroll
    for (int j = 0; j < MAX_PAIRS; ++j) {
      const int d = lane * 2 + 64 * j;
      if (64 * j < D) {
        v[j][0] = value(d);
        v[j][1] = value(d + 1);
        s += v[j][0] * v[j][0] + v[j][1] * v[j][1];
      }
    }
    const float inv = norm == 3 ? rsqrtf(warp_sum(s) / (float)dim + a.eps) : 1.f;
    OutT* out = reinterpret_cast<OutT*>(kind == 0 ? a.q_out : a.kv_cache) + out0 + (kind == 2 ? plane : 0);
#pragma unroll
    for (int j = 0; j < MAX_PAIRS; ++j)
      if (64 * j < D) store2(out + lane * 2 + 64 * j, v[j][0] * inv, v[j][1] * inv);
  }
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
  const auto parts = [&](const HeadRows& r) { return r.x == nullptr ? 0 : (r.heads + per - 1) / per; };
  const size_t smem = (size_t)(((a.rot_dims + 3) & ~3) + per * widest + 8) * sizeof(float);
  const dim3 grid(a.T, parts(a.q) + parts(a.k) + parts(a.v) + conv), block(NTHR);
  return (int)(a.out_f32 ? launch_pdl(mixer_post_kernel<float>, grid, block, smem, stream, a)
                         : launch_pdl(mixer_post_kernel<__nv_bfloat16>, grid, block, smem, stream, a));
}
HE_API int he_mixer_post_args_size() { return (int)sizeof(MixerPostArgs); }
