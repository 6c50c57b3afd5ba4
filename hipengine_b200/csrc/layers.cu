// Row-wise layer glue: RMSNorm, activation*mul, fused split-Q|gate + QK-RMSNorm + partial RoPE + paged
// KV write, causal conv1d + SiLU with rolling state, embedding-free bookkeeping kernels.
//
// Behavioural references: hipengine/kernels/hip_gfx1100/fused/gguf_ops.hip (GGUF F32-weight RMSNorm,
// fused split-qgate + head RMSNorm + partial rotary), attention/paged_kv_write.hip (append K/V through
// the live-span block table), linear_attn/conv.hip (depthwise causal conv, kernel 4, rolling state),
// runtime/state.hip (device-side position bookkeeping so a decode step can live in one graph).
#include "common.cuh"

using namespace he;

namespace {

// ---------------------------------------------------------------- RMSNorm rows: fp32 [T][H] -> bf16/f32 [T][H]
template <typename OutT>
__global__ void __launch_bounds__(256) rmsnorm_rows_kernel(const float* __restrict__ x, const float* __restrict__ w,
                                                           OutT* __restrict__ out, int H, float eps,
                                                           long long x_stride, long long out_stride, int n_mean) {
  pdl_wait();      // launched with programmatic stream serialization: order after all earlier kernels
  pdl_launch();
  __shared__ float red[33];
  const float* xr = x + (size_t)blockIdx.x * x_stride;
  float ss = 0.f;
  for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
    const float4 v = *reinterpret_cast<const float4*>(xr + i);
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  ss = block_sum(ss, red);
  const float inv = rsqrtf(ss / (float)n_mean + eps);    // zero-padded rows: n_mean < H real columns
  OutT* orow = out + (size_t)blockIdx.x * out_stride;
  for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
    const float4 v = *reinterpret_cast<const float4*>(xr + i);
    float4 g = make_float4(1.f, 1.f, 1.f, 1.f);
    if (w != nullptr) g = *reinterpret_cast<const float4*>(w + i);
    const float o0 = v.x * inv * g.x, o1 = v.y * inv * g.y, o2 = v.z * inv * g.z, o3 = v.w * inv * g.w;
    if constexpr (sizeof(OutT) == 2) {
      __nv_bfloat162 a = __floats2bfloat162_rn(o0, o1), b = __floats2bfloat162_rn(o2, o3);
      uint2 pk;
      pk.x = *reinterpret_cast<uint32_t*>(&a);
      pk.y = *reinterpret_cast<uint32_t*>(&b);
      *reinterpret_cast<uint2*>(orow + i) = pk;
    } else {
      *reinterpret_cast<float4*>(orow + i) = make_float4(o0, o1, o2, o3);
    }
  }
}

// ---------------------------------------------------------------- RMSNorm rows + token shift
// h[t] = norm(x[t]) and hs[t] = h[t] + shift * (h[t-1] - h[t]) for packed segments; the row before a segment's first one is
// the slot's state (zeros for a new request).  The CTA of that first row also replaces the state with the segment's last
// normalised row (recomputed here), so the only reader and the only writer of a state row are the same threads.  With a
// journal (verify chains) the state stays and every row's h is recorded instead.
struct NormShiftArgs {
  const float* x;            // [T][ldx] residual rows
  long long ldx;
  const float* w;            // [H] norm gains (zero in padded columns)
  const float* shift;        // [H]
  float* state;              // [n_slots][H]
  float* journal;            // [T][H] or null
  const int* seg_start;      // [n_seg + 1]
  const int* seg_slot;       // [n_seg]
  const int* tok_seg;        // [T]
  void* h;                   // [T][H] bf16 or fp32
  void* hs;
  int T, H, n_mean, out_bf16, n_slots;
  float eps;
};

template <typename OutT>
__device__ __forceinline__ void store4(OutT* p, float4 v) {
  if constexpr (sizeof(OutT) == 2) {
    __align__(8) __nv_bfloat162 b[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
    *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(b);
  } else {
    *reinterpret_cast<float4*>(p) = v;
  }
}
__device__ __forceinline__ float sq4(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
__device__ __forceinline__ float4 mul4(float4 v, float4 g, float s) {
  return make_float4(v.x * s * g.x, v.y * s * g.y, v.z * s * g.z, v.w * s * g.w);
}

template <typename OutT>
__global__ void __launch_bounds__(256) norm_shift_kernel(const NormShiftArgs a) {
  pdl_wait();
  pdl_launch();
  __shared__ float red[33];
  const int t = blockIdx.x, seg = a.tok_seg[t], first = a.seg_start[seg], last = a.seg_start[seg + 1] - 1;
  const int slot = a.seg_slot[seg];
  if (!HE_INDEX_OK(slot, a.n_slots, HE_SITE_STATE_SLOT)) return;
  const bool head = t == first, upd = head && a.journal == nullptr;
  const float* xt = a.x + (size_t)t * a.ldx;
  const float* xp = head ? xt : xt - a.ldx;
  const float* xl = a.x + (size_t)last * a.ldx;
  float st = 0.f, sp = 0.f, sl = 0.f;
  for (int i = threadIdx.x * 4; i < a.H; i += 1024) {
    st += sq4(*reinterpret_cast<const float4*>(xt + i));
    if (!head) sp += sq4(*reinterpret_cast<const float4*>(xp + i));
    if (upd && last != t) sl += sq4(*reinterpret_cast<const float4*>(xl + i));
  }
  const float n = (float)a.n_mean;
  const float it = rsqrtf(block_sum(st, red) / n + a.eps);
  float ip = 0.f, il = it;                   // conditions are uniform over the CTA
  if (!head) ip = rsqrtf(block_sum(sp, red) / n + a.eps);
  if (upd && last != t) il = rsqrtf(block_sum(sl, red) / n + a.eps);
  float* state = a.state + (size_t)slot * a.H;
  OutT* ho = reinterpret_cast<OutT*>(a.h) + (size_t)t * a.H;
  OutT* so = reinterpret_cast<OutT*>(a.hs) + (size_t)t * a.H;
  for (int i = threadIdx.x * 4; i < a.H; i += 1024) {
    const float4 g = *reinterpret_cast<const float4*>(a.w + i), s = *reinterpret_cast<const float4*>(a.shift + i);
    const float4 h = mul4(*reinterpret_cast<const float4*>(xt + i), g, it);
    const float4 p = head ? *reinterpret_cast<const float4*>(state + i)
                          : mul4(*reinterpret_cast<const float4*>(xp + i), g, ip);
    store4(ho + i, h);
    store4(so + i, make_float4(h.x + (p.x - h.x) * s.x, h.y + (p.y - h.y) * s.y, h.z + (p.z - h.z) * s.z,
                               h.w + (p.w - h.w) * s.w));
    if (upd) *reinterpret_cast<float4*>(state + i) = mul4(*reinterpret_cast<const float4*>(xl + i), g, il);
    if (a.journal != nullptr) *reinterpret_cast<float4*>(a.journal + (size_t)t * a.H + i) = h;
  }
}

// act codes: 0 silu(g) * u, 1 gelu_tanh(g) * u, 2 clamped GLU with `limit`
__device__ __forceinline__ float act_pair(float g, float u, int act, float limit) {
  if (act == 2) return clamped_glu_f(g, u, limit);
  return (act == 0 ? silu_f(g) : gelu_tanh_f(g)) * u;
}

// ---------------------------------------------------------------- act(gate) * up over packed [T][2F] bf16 -> [T][F] bf16
__global__ void act_mul_kernel(const __nv_bfloat16* __restrict__ gu, __nv_bfloat16* __restrict__ out, long long T,
                               int F, int act, float limit) {
  pdl_wait();      // launched with programmatic stream serialization: order after all earlier kernels
  pdl_launch();
  const long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (i >= T * F) return;
  const long long t = i / F;
  const int f = (int)(i % F);
  const uint4 gv = *reinterpret_cast<const uint4*>(gu + (size_t)t * 2 * F + f);
  const uint4 uv = *reinterpret_cast<const uint4*>(gu + (size_t)t * 2 * F + F + f);
  const __nv_bfloat162* g2 = reinterpret_cast<const __nv_bfloat162*>(&gv);
  const __nv_bfloat162* u2 = reinterpret_cast<const __nv_bfloat162*>(&uv);
  __align__(16) __nv_bfloat162 o[4];
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const float2 g = __bfloat1622float2(g2[k]), u = __bfloat1622float2(u2[k]);
    o[k] = __floats2bfloat162_rn(act_pair(g.x, u.x, act, limit), act_pair(g.y, u.y, act, limit));
  }
  *reinterpret_cast<uint4*>(out + i) = *reinterpret_cast<const uint4*>(o);
}

// same with the packed gate | up rows in fp32 (split-K accumulators of small batches); bf16 or fp32 result
template <typename OutT>
__global__ void act_mul_f32_kernel(const float* __restrict__ gu, OutT* __restrict__ out, long long T, int F, int act,
                                   float limit) {
  pdl_wait();      // launched with programmatic stream serialization: order after all earlier kernels
  pdl_launch();
  const long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (i >= T * F) return;
  const long long t = i / F;
  const int f = (int)(i % F);
  const float4 g = *reinterpret_cast<const float4*>(gu + (size_t)t * 2 * F + f);
  const float4 u = *reinterpret_cast<const float4*>(gu + (size_t)t * 2 * F + F + f);
  const float gx[4] = {g.x, g.y, g.z, g.w}, ux[4] = {u.x, u.y, u.z, u.w};
  float y[4];
#pragma unroll
  for (int k = 0; k < 4; ++k) y[k] = act_pair(gx[k], ux[k], act, limit);
  if constexpr (sizeof(OutT) == 2) {
    __align__(8) __nv_bfloat162 o[2] = {__floats2bfloat162_rn(y[0], y[1]), __floats2bfloat162_rn(y[2], y[3])};
    *reinterpret_cast<uint2*>(out + i) = *reinterpret_cast<const uint2*>(o);
  } else {
    *reinterpret_cast<float4*>(out + i) = make_float4(y[0], y[1], y[2], y[3]);
  }
}

// ---------------------------------------------------------------- residual add: h (fp32) += y (bf16)
__global__ void resid_add_bf16_kernel(float* __restrict__ h, const __nv_bfloat16* __restrict__ y, long long n) {
  pdl_wait();      // launched with programmatic stream serialization: order after all earlier kernels
  pdl_launch();
  const long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (i >= n) return;
  float4 hv = *reinterpret_cast<float4*>(h + i);
  const uint2 yv = *reinterpret_cast<const uint2*>(y + i);
  const __nv_bfloat162* y2 = reinterpret_cast<const __nv_bfloat162*>(&yv);
  const float2 a = __bfloat1622float2(y2[0]), b = __bfloat1622float2(y2[1]);
  hv.x += a.x; hv.y += a.y; hv.z += b.x; hv.w += b.y;
  *reinterpret_cast<float4*>(h + i) = hv;
}

// ---------------------------------------------------------------- fused QK-norm + partial RoPE + KV write
struct QkvArgs {
  const void* q;      // [T][q_stride]: per head [Q(D) | gate(D)] when gated, else [Q(D)]
  const void* k;      // [T][k_stride]
  const void* v;      // [T][v_stride]
  int in_dtype;       // 0 f32, 1 bf16
  long long q_stride, k_stride, v_stride;
  const float* q_norm;   // [D] or null
  const float* k_norm;   // [D] or null
  int v_norm;            // 1: weightless RMSNorm on V (Gemma)
  __nv_bfloat16* q_out;    // [T][H][D]
  __nv_bfloat16* gate_out; // [T][H][D] or null
  __nv_bfloat16* kv_cache; // [n_pages][2][Hkv][PAGE][D]
  const int* block_table;  // [n_slots][max_pages]
  const int* slot;         // [T] row of block_table per token
  const int* pos;          // [T] absolute position
  int max_pages;
  int H, Hkv, D, page;
  int gated;
  int rope_dim;
  float theta;
  float eps;
  float q_scale;           // multiplied into Q after norm/rope (1 = none)
  int rope_denom;          // frequency spacing: inv_freq_i = theta^(-2i / rope_denom); 0 -> rope_dim
  int d_in, dv_in;         // head widths of the projections (0 -> D): narrower heads are zero-padded to D
  int out_f32;             // 1: q_out and kv_cache hold fp32 (the float32 compute dtype)
};

__device__ __forceinline__ float load_in(const void* p, int dtype, size_t i) {
  return dtype == 0 ? reinterpret_cast<const float*>(p)[i] : bf16_to_f32(reinterpret_cast<const __nv_bfloat16*>(p)[i]);
}

// grid (T, H + 2*Hkv); block D threads (D <= 512, multiple of 32)
__global__ void qkv_post_kernel(const QkvArgs a) {
  extern __shared__ float sh[];  // [D]
  __shared__ float red[33];
  const int t = blockIdx.x, hh = blockIdx.y, d = threadIdx.x;
  const int D = a.D;
  pdl_wait();
  pdl_launch();
  int kind, h;  // 0 q, 1 k, 2 v
  if (hh < a.H) { kind = 0; h = hh; }
  else if (hh < a.H + a.Hkv) { kind = 1; h = hh - a.H; }
  else { kind = 2; h = hh - a.H - a.Hkv; }
  const int din = kind == 2 ? (a.dv_in > 0 ? a.dv_in : D) : (a.d_in > 0 ? a.d_in : D);
  float x = 0.f;
  if (d < din) {
    if (kind == 0) x = load_in(a.q, a.in_dtype, (size_t)t * a.q_stride + (size_t)h * din * (a.gated ? 2 : 1) + d);
    else if (kind == 1) x = load_in(a.k, a.in_dtype, (size_t)t * a.k_stride + (size_t)h * din + d);
    else x = load_in(a.v, a.in_dtype, (size_t)t * a.v_stride + (size_t)h * din + d);
  }

  const float* nw = kind == 0 ? a.q_norm : (kind == 1 ? a.k_norm : nullptr);
  const bool do_norm = (kind < 2 && nw != nullptr) || (kind == 2 && a.v_norm);
  if (do_norm) {
    const float ss = block_sum(x * x, red);
    x = x * rsqrtf(ss / (float)din + a.eps);
    if (nw != nullptr && d < din) x *= nw[d];
  }
  const int p = a.pos[t];
  if (kind < 2 && a.rope_dim > 0) {
    sh[d] = x;
    __syncthreads();
    const int half = a.rope_dim >> 1;
    if (d < a.rope_dim) {
      const int i = d < half ? d : d - half;
      const float inv_freq = powf(a.theta, -2.0f * (float)i / (float)(a.rope_denom > 0 ? a.rope_denom : a.rope_dim));
      float sn, cs;
      sincosf((float)p * inv_freq, &sn, &cs);
      const float other = sh[d < half ? d + half : d - half];
      x = d < half ? x * cs - other * sn : x * cs + other * sn;
    }
  }
  if (kind == 0) {
    const size_t qo = ((size_t)t * a.H + h) * D + d;
    if (a.out_f32) reinterpret_cast<float*>(a.q_out)[qo] = x * a.q_scale;
    else a.q_out[qo] = f32_to_bf16(x * a.q_scale);
    if (a.gated && a.gate_out != nullptr) {
      const float g = load_in(a.q, a.in_dtype, (size_t)t * a.q_stride + (size_t)h * D * 2 + D + d);
      a.gate_out[((size_t)t * a.H + h) * D + d] = f32_to_bf16(g);
    }
  } else {
    const int s = a.slot[t];
    if (!HE_INDEX_OK(p / a.page, a.max_pages, HE_SITE_KV_WRITE_PAGE)) return;
    const int page_id = a.block_table[(size_t)s * a.max_pages + p / a.page];
    const size_t off = ((((size_t)page_id * 2 + (kind - 1)) * a.Hkv + h) * a.page + (p % a.page)) * D + d;
    if (a.out_f32) reinterpret_cast<float*>(a.kv_cache)[off] = x;
    else a.kv_cache[off] = f32_to_bf16(x);
  }
}

// ---------------------------------------------------------------- causal conv1d (k<=4) + SiLU with rolling state
struct ConvArgs {
  const void* x;        // [T][x_stride] (first C columns used)
  int in_dtype;
  long long x_stride;
  const float* w;       // [C][KW]
  float* state;         // [n_slots][C][KW-1]  (oldest first)
  const int* seg_start; // [n_seg+1] cumulative token offsets
  const int* seg_slot;  // [n_seg]
  const int* tok_seg;   // [T] segment of each token
  float* out;           // [T][C] fp32
  float* journal;       // optional [T][C][KW-1]: state after each token (verify chains), else null
  int C, KW, T, n_seg;
};

// one thread per (8 channels, CONV_TOK consecutive tokens); the 8 x KW filter taps are loaded once per thread
// and reused for all its tokens (they used to dominate the load traffic at one token per thread).
constexpr int CONV_TOK = 8;
template <int KWT>
__global__ void __launch_bounds__(256) conv_fwd_kernel(const ConvArgs a) {
  pdl_wait();      // launched with programmatic stream serialization: order after all earlier kernels
  pdl_launch();
  const int C8 = a.C >> 3;
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  const int n_tchunks = (a.T + CONV_TOK - 1) / CONV_TOK;
  if (i >= (long long)n_tchunks * C8) return;
  const int t_first = (int)(i / C8) * CONV_TOK, c = (int)(i % C8) * 8;
  constexpr int KW = KWT;
  float wreg[8][KW];
  if constexpr (KW == 4) {
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const float4 w4 = __ldg(reinterpret_cast<const float4*>(a.w + (size_t)(c + e) * 4));
      wreg[e][0] = w4.x; wreg[e][1] = w4.y; wreg[e][2] = w4.z; wreg[e][3] = w4.w;
    }
  } else {
#pragma unroll
    for (int e = 0; e < 8; ++e)
#pragma unroll
      for (int k = 0; k < KW; ++k) wreg[e][k] = __ldg(a.w + (size_t)(c + e) * KW + k);
  }
  const int t_last = min(a.T, t_first + CONV_TOK);
  for (int t = t_first; t < t_last; ++t) {
    const int sg = a.tok_seg[t];
    const int s0 = a.seg_start[sg];
    const int local = t - s0;
    const float* st = a.state + ((size_t)a.seg_slot[sg] * a.C + c) * (KW - 1);
    float acc[8], win[KW][8];
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] = 0.f;
#pragma unroll
    for (int k = 0; k < KW; ++k) {
      const int idx = local + k;  // index into [state(KW-1) ++ x_seg]
      if (idx < KW - 1) {
#pragma unroll
        for (int e = 0; e < 8; ++e) win[k][e] = st[(size_t)e * (KW - 1) + idx];
      } else {
        const size_t off = (size_t)(s0 + idx - (KW - 1)) * a.x_stride + c;
        if (a.in_dtype == 0) {
          const float4 v0 = *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(a.x) + off);
          const float4 v1 = *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(a.x) + off + 4);
          win[k][0] = v0.x; win[k][1] = v0.y; win[k][2] = v0.z; win[k][3] = v0.w;
          win[k][4] = v1.x; win[k][5] = v1.y; win[k][6] = v1.z; win[k][7] = v1.w;
        } else {
          const uint4 u = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(a.x) + off);
          const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float2 f = __bfloat1622float2(h2[e]);
            win[k][2 * e] = f.x; win[k][2 * e + 1] = f.y;
          }
        }
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[e] += win[k][e] * wreg[e][k];
    }
    float* o = a.out + (size_t)t * a.C + c;
    *reinterpret_cast<float4*>(o) = make_float4(silu_f(acc[0]), silu_f(acc[1]), silu_f(acc[2]), silu_f(acc[3]));
    *reinterpret_cast<float4*>(o + 4) = make_float4(silu_f(acc[4]), silu_f(acc[5]), silu_f(acc[6]), silu_f(acc[7]));
    if (a.journal != nullptr) {
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        float* j = a.journal + ((size_t)t * a.C + c + e) * (KW - 1);
#pragma unroll
        for (int k = 1; k < KW; ++k) j[k - 1] = win[k][e];
      }
    }
  }
}

// one thread per (segment, channel): new state = last KW-1 entries of [state ++ x_seg]
__global__ void conv_state_kernel(const ConvArgs a) {
  pdl_wait();      // launched with programmatic stream serialization: order after all earlier kernels
  pdl_launch();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)a.n_seg * a.C) return;
  const int sg = (int)(i / a.C), c = (int)(i % a.C);
  const int s0 = a.seg_start[sg], n = a.seg_start[sg + 1] - s0;
  const int KW = a.KW;
  float* st = a.state + ((size_t)a.seg_slot[sg] * a.C + c) * (KW - 1);
  float nv[3];
  for (int j = 0; j < KW - 1; ++j) {
    const int idx = n + j;
    nv[j] = idx < KW - 1 ? st[idx] : load_in(a.x, a.in_dtype, (size_t)(s0 + idx - (KW - 1)) * a.x_stride + c);
  }
  for (int j = 0; j < KW - 1; ++j) st[j] = nv[j];
}

// ---------------------------------------------------------------- bookkeeping
__global__ void advance_positions_kernel(int* pos, int* ctx_len, const int* active, int n, int delta) {
  pdl_wait();      // launched with programmatic stream serialization: order after all earlier kernels
  pdl_launch();
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  if (active == nullptr || active[i]) {
    pos[i] += delta;
    if (ctx_len != nullptr) ctx_len[i] += delta;
  }
}

}  // namespace

HE_API int he_rmsnorm_rows(const void* x, const void* w, void* out, int out_bf16, int T, int H, float eps,
                           long long x_stride, long long out_stride, int n_mean, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H % 4 != 0 || n_mean <= 0 || n_mean > H) return -HE_ERR_BAD_ARG;
  if (out_bf16)
    (void)launch_pdl(rmsnorm_rows_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, stream, (const float*)x, (const float*)w, (__nv_bfloat16*)out, H,
                                                              eps, x_stride, out_stride, n_mean);
  else
    (void)launch_pdl(rmsnorm_rows_kernel<float>, dim3(T), dim3(256), 0, stream, (const float*)x, (const float*)w, (float*)out, H, eps, x_stride,
                                                      out_stride, n_mean);
  HE_LAUNCH_CHECK();
  return 0;
}

HE_API int he_norm_shift(const NormShiftArgs* args, cudaStream_t stream) {
  const NormShiftArgs& a = *args;
  if (a.T <= 0) return 0;
  if (a.H % 4 != 0 || a.ldx % 4 != 0 || a.n_mean <= 0 || a.n_mean > a.H) return -HE_ERR_BAD_ARG;
  return (int)(a.out_bf16 ? launch_pdl(norm_shift_kernel<__nv_bfloat16>, dim3(a.T), dim3(256), 0, stream, a)
                          : launch_pdl(norm_shift_kernel<float>, dim3(a.T), dim3(256), 0, stream, a));
}
HE_API int he_norm_shift_args_size() { return (int)sizeof(NormShiftArgs); }

HE_API int he_act_mul(const void* gu, void* out, long long T, int F, int act, float limit, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (F % 8 != 0) return -HE_ERR_BAD_ARG;
  const long long n = T * F / 8;
  (void)launch_pdl(act_mul_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, stream, (const __nv_bfloat16*)gu, (__nv_bfloat16*)out, T, F,
                                                                   act, limit);
  HE_LAUNCH_CHECK();
  return 0;
}

HE_API int he_act_mul_f32(const void* gu, void* out, int out_bf16, long long T, int F, int act, float limit,
                          cudaStream_t stream) {
  if (T <= 0) return 0;
  if (F % 4 != 0) return -HE_ERR_BAD_ARG;
  const long long n = T * F / 4;
  const dim3 grid((unsigned)((n + 255) / 256));
  if (out_bf16)
    (void)launch_pdl(act_mul_f32_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, (const float*)gu, (__nv_bfloat16*)out, T, F, act, limit);
  else
    (void)launch_pdl(act_mul_f32_kernel<float>, grid, dim3(256), 0, stream, (const float*)gu, (float*)out, T, F, act, limit);
  HE_LAUNCH_CHECK();
  return 0;
}

HE_API int he_resid_add_bf16(void* h, const void* y, long long n, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (n % 4 != 0) return -HE_ERR_BAD_ARG;
  (void)launch_pdl(resid_add_bf16_kernel, dim3((unsigned)((n / 4 + 255) / 256)), dim3(256), 0, stream, (float*)h, (const __nv_bfloat16*)y, n);
  HE_LAUNCH_CHECK();
  return 0;
}

__global__ void resid_add_f32_kernel(float* __restrict__ h, const float* __restrict__ y, long long n) {
  pdl_wait();      // launched with programmatic stream serialization: order after all earlier kernels
  pdl_launch();
  const long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (i >= n) return;
  float4 a = *reinterpret_cast<float4*>(h + i);
  const float4 b = *reinterpret_cast<const float4*>(y + i);
  a.x += b.x; a.y += b.y; a.z += b.z; a.w += b.w;
  *reinterpret_cast<float4*>(h + i) = a;
}

// h[i] += y[i] (fp32, contiguous, n % 4 == 0): residual add after a reduced row-parallel projection
HE_API int he_resid_add_f32(void* h, const void* y, long long n, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (n % 4 != 0) return -HE_ERR_BAD_ARG;
  (void)launch_pdl(resid_add_f32_kernel, dim3((unsigned)((n / 4 + 255) / 256)), dim3(256), 0, stream, (float*)h, (const float*)y, n);
  HE_LAUNCH_CHECK();
  return 0;
}

// ---------------------------------------------------------------- sandwich-norm residual updates (Gemma)
// h[t] += RMSNorm(y[t]) * w        (y fp32 or bf16; one CTA per row)
__global__ void __launch_bounds__(256) norm_add_kernel(float* __restrict__ h, long long ldh, const void* __restrict__ y,
                                                       int y_dtype, long long ldy, const float* __restrict__ w, int H,
                                                       float eps) {
  pdl_wait();      // launched with programmatic stream serialization: order after all earlier kernels
  pdl_launch();
  __shared__ float red[33];
  const int t = blockIdx.x;
  float ss = 0.f;
  for (int i = threadIdx.x; i < H; i += 256) {
    const float v = load_in(y, y_dtype, (size_t)t * ldy + i);
    ss += v * v;
  }
  ss = block_sum(ss, red);
  const float inv = rsqrtf(ss / (float)H + eps);
  for (int i = threadIdx.x; i < H; i += 256)
    h[(size_t)t * ldh + i] += load_in(y, y_dtype, (size_t)t * ldy + i) * inv * w[i];
}

// h[t] = (h[t] + RMSNorm(RMSNorm(d[t])*w1 + RMSNorm(e[t])*w2) * w3) * scalar[0]
// d: dense-branch output, e: expert-branch output (either fp32 or bf16).
__global__ void __launch_bounds__(256) ffn_combine_kernel(float* __restrict__ h, long long ldh,
                                                          const void* __restrict__ d, int d_dtype, long long ldd,
                                                          const void* __restrict__ e, int e_dtype, long long lde,
                                                          const float* __restrict__ w1, const float* __restrict__ w2,
                                                          const float* __restrict__ w3,
                                                          const float* __restrict__ scalar, int H, float eps) {
  pdl_wait();      // launched with programmatic stream serialization: order after all earlier kernels
  pdl_launch();
  extern __shared__ float buf[];   // [H]
  __shared__ float red[33];
  const int t = blockIdx.x;
  float sd = 0.f, se = 0.f;
  for (int i = threadIdx.x; i < H; i += 256) {
    const float a = load_in(d, d_dtype, (size_t)t * ldd + i), b = load_in(e, e_dtype, (size_t)t * lde + i);
    sd += a * a; se += b * b;
  }
  sd = block_sum(sd, red);
  se = block_sum(se, red);
  const float id = rsqrtf(sd / (float)H + eps), ie = rsqrtf(se / (float)H + eps);
  float sc = 0.f;
  for (int i = threadIdx.x; i < H; i += 256) {
    const float c = load_in(d, d_dtype, (size_t)t * ldd + i) * id * w1[i] +
                    load_in(e, e_dtype, (size_t)t * lde + i) * ie * w2[i];
    buf[i] = c;
    sc += c * c;
  }
  sc = block_sum(sc, red);
  const float ic = rsqrtf(sc / (float)H + eps);
  const float s = scalar != nullptr ? scalar[0] : 1.f;
  for (int i = threadIdx.x; i < H; i += 256)
    h[(size_t)t * ldh + i] = (h[(size_t)t * ldh + i] + buf[i] * ic * w3[i]) * s;
}

// ---------------------------------------------------------------- looped layers: input of a pass
// h[t] += x0[t] (the embedding output; null on the first pass) + step (one vector for all rows).  H % 4 == 0.
__global__ void __launch_bounds__(256) resid_inject_kernel(float* __restrict__ h, const float* __restrict__ x0,
                                                           const float* __restrict__ step, long long T, int H) {
  pdl_wait();
  pdl_launch();
  const long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (i >= T * H) return;
  float4 v = *reinterpret_cast<const float4*>(h + i);
  if (x0 != nullptr) {
    const float4 e = *reinterpret_cast<const float4*>(x0 + i);
    v.x += e.x; v.y += e.y; v.z += e.z; v.w += e.w;
  }
  const float4 s = *reinterpret_cast<const float4*>(step + i % H);
  v.x += s.x; v.y += s.y; v.z += s.z; v.w += s.w;
  *reinterpret_cast<float4*>(h + i) = v;
}

HE_API int he_resid_inject(void* h, const void* x0, const void* step, long long T, int H, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H % 4 != 0 || step == nullptr) return -HE_ERR_BAD_ARG;
  const long long n = T * H / 4;
  return (int)launch_pdl(resid_inject_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, stream, (float*)h,
                         (const float*)x0, (const float*)step, T, H);
}

HE_API int he_norm_add(void* h, long long ldh, const void* y, int y_dtype, long long ldy, const void* w, int T, int H,
                       float eps, cudaStream_t stream) {
  if (T <= 0) return 0;
  (void)launch_pdl(norm_add_kernel, dim3(T), dim3(256), 0, stream, (float*)h, ldh, y, y_dtype, ldy, (const float*)w, H, eps);
  HE_LAUNCH_CHECK();
  return 0;
}

HE_API int he_ffn_combine(void* h, long long ldh, const void* d, int d_dtype, long long ldd, const void* e, int e_dtype,
                          long long lde, const void* w1, const void* w2, const void* w3, const void* scalar, int T,
                          int H, float eps, cudaStream_t stream) {
  if (T <= 0) return 0;
  if ((size_t)H * sizeof(float) > 48 * 1024) return -HE_ERR_BAD_ARG;
  (void)launch_pdl(ffn_combine_kernel, dim3(T), dim3(256), (size_t)H * sizeof(float), stream, (float*)h, ldh, d, d_dtype, ldd, e, e_dtype, lde,
                                                                    (const float*)w1, (const float*)w2,
                                                                    (const float*)w3, (const float*)scalar, H, eps);
  HE_LAUNCH_CHECK();
  return 0;
}

HE_API int he_qkv_post(const QkvArgs* args, int T, cudaStream_t stream) {
  const QkvArgs& a = *args;
  if (T <= 0) return 0;
  if (a.D % 32 != 0 || a.D > 512 || a.d_in > a.D || a.dv_in > a.D) return -HE_ERR_BAD_ARG;
  if ((a.d_in > 0 && a.d_in < a.D) && (a.gated || a.rope_dim > 0)) return -HE_ERR_BAD_ARG;
  dim3 grid(T, a.H + 2 * a.Hkv);
  cudaError_t le = launch_pdl(qkv_post_kernel, grid, dim3(a.D), a.D * sizeof(float), stream, a);
  if (le != cudaSuccess) return (int)le;
  return 0;
}
HE_API int he_qkv_args_size() { return (int)sizeof(QkvArgs); }

HE_API int he_conv1d(const ConvArgs* args, int update_state, cudaStream_t stream) {
  const ConvArgs& a = *args;
  if (a.T <= 0) return 0;
  if (a.KW < 2 || a.KW > 4) return -HE_ERR_BAD_ARG;
  if (a.C % 8 != 0) return -HE_ERR_BAD_ARG;
  const long long n = (long long)((a.T + CONV_TOK - 1) / CONV_TOK) * (a.C / 8);
  const unsigned nblk = (unsigned)((n + 255) / 256);
  if (a.KW == 4) (void)launch_pdl(conv_fwd_kernel<4>, dim3(nblk), dim3(256), 0, stream, a);
  else if (a.KW == 3) (void)launch_pdl(conv_fwd_kernel<3>, dim3(nblk), dim3(256), 0, stream, a);
  else (void)launch_pdl(conv_fwd_kernel<2>, dim3(nblk), dim3(256), 0, stream, a);
  HE_LAUNCH_CHECK();
  if (update_state) {
    const long long m = (long long)a.n_seg * a.C;
    (void)launch_pdl(conv_state_kernel, dim3((unsigned)((m + 255) / 256)), dim3(256), 0, stream, a);
    HE_LAUNCH_CHECK();
  }
  return 0;
}
HE_API int he_conv_args_size() { return (int)sizeof(ConvArgs); }

HE_API int he_advance_positions(void* pos, void* ctx_len, const void* active, int n, int delta, cudaStream_t stream) {
  if (n <= 0) return 0;
  (void)launch_pdl(advance_positions_kernel, dim3((n + 127) / 128), dim3(128), 0, stream, (int*)pos, (int*)ctx_len, (const int*)active, n, delta);
  HE_LAUNCH_CHECK();
  return 0;
}

// ---------------------------------------------------------------- skinny fp32 GEMM: out[T][N] = x[T][K] * W[N][K]^T
// For the few projections whose weights stay F32 in GGUF files (router, ssm_alpha/beta) at prefill row counts, and every
// projection of the float32 compute dtype.  grid.z repeats the product at the batch strides (one matrix per head).
// mode 0: store, 1: add (times col_scale[n], or plus col_bias[n], when given), 2: store relu(v)^2.
namespace {
constexpr int SG_TM = 64, SG_TN = 64, SG_TK = 16;
__global__ void __launch_bounds__(256) small_gemm_f32_kernel(const void* __restrict__ x, int x_dtype,
                                                             long long x_stride, const void* __restrict__ w,
                                                             int w_dtype, long long w_stride,
                                                             float* __restrict__ out, long long out_stride, int T,
                                                             int N, int K, int mode,
                                                             const float* __restrict__ col_scale,
                                                             const float* __restrict__ col_bias, long long x_bs,
                                                             long long w_bs, long long out_bs) {
  __shared__ float xs[SG_TK][SG_TM + 1];
  __shared__ float ws[SG_TK][SG_TN + 1];
  const int t0 = blockIdx.y * SG_TM, n0 = blockIdx.x * SG_TN;
  const size_t x0 = (size_t)blockIdx.z * x_bs, w0 = (size_t)blockIdx.z * w_bs;
  out += (size_t)blockIdx.z * out_bs;
  const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;  // 16 x 16 threads, 4x4 outputs each
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += SG_TK) {
    for (int i = threadIdx.x; i < SG_TM * SG_TK; i += 256) {
      const int r = i / SG_TK, kk = i % SG_TK;
      const int t = t0 + r, k = k0 + kk;
      xs[kk][r] = (t < T && k < K) ? load_in(x, x_dtype, x0 + (size_t)t * x_stride + k) : 0.f;
    }
    for (int i = threadIdx.x; i < SG_TN * SG_TK; i += 256) {
      const int r = i / SG_TK, kk = i % SG_TK;
      const int n = n0 + r, k = k0 + kk;
      ws[kk][r] = (n < N && k < K) ? load_in(w, w_dtype, w0 + (size_t)n * w_stride + k) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < SG_TK; ++kk) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = xs[kk][ty * 4 + i]; b[i] = ws[kk][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += a[i] * b[j];
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int t = t0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (t < T && n < N) {
        float* o = out + (size_t)t * out_stride + n;
        const float v = acc[i][j] + (mode == 1 && col_scale == nullptr && col_bias != nullptr ? col_bias[n] : 0.f);
        *o = mode == 1 ? *o + (col_scale != nullptr ? v * col_scale[n] : v) : mode == 2 ? relu2_f(v) : v;
      }
    }
}
}  // namespace

HE_API int he_small_gemm_f32(const void* x, int x_dtype, long long x_stride, const void* w, int w_dtype,
                             long long w_stride, void* out, long long out_stride, int T, int N, int K, int mode,
                             const void* col_scale, const void* col_bias, int n_batch, long long x_bs, long long w_bs, long long out_bs,
                             cudaStream_t stream) {
  if (T <= 0 || N <= 0) return 0;
  if (mode < 0 || mode > 2 || n_batch < 1 || n_batch > 65535 || (col_scale != nullptr && col_bias != nullptr)) return -HE_ERR_BAD_ARG;
  dim3 grid((N + SG_TN - 1) / SG_TN, (T + SG_TM - 1) / SG_TM, n_batch);
  small_gemm_f32_kernel<<<grid, 256, 0, stream>>>(x, x_dtype, x_stride, w, w_dtype, w_stride, (float*)out, out_stride, T,
                                                  N, K, mode, (const float*)col_scale, (const float*)col_bias, x_bs, w_bs, out_bs);
  HE_LAUNCH_CHECK();
  return 0;
}
