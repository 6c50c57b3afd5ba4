// fp32 forms of the operations whose served forms use bfloat16 tensor cores (the float32 compute dtype): attention over
// fp32 KV pages and the selected experts.  Plain CUDA-core kernels with fp32 operands and fp32 accumulation; bf16
// weights are widened exactly.  The projections are he_small_gemm_f32 (layers.cu).
#include "common.cuh"

using namespace he;

struct ExactAttnArgs {
  const float* q;            // [R][H][D]
  const float* kv_cache;     // [n_pages][2][Hkv][page][D]
  const int* block_table;    // [n_slots][max_pages]
  const int* slot;           // [R]
  const int* ctx_len;        // [R] keys visible to the row
  float* out;                // [R][H*D]
  int R, H, Hkv, D, page, max_pages;
  float scale, softcap;      // softcap 0: none
  int window;                // > 0: only the last `window` keys are visible
  const float* sink;         // [H] or null: score of one more term in the softmax denominator
  const float* head_gate;    // [R][head_gate_stride] or null: outputs times sigmoid(head_gate[r][h])
  long long head_gate_stride;
  int keep_first;            // with a window: the first `keep_first` keys stay visible
};

struct ExactMoeArgs {
  const float* x;            // gate/up: normalised rows [T][ldx]
  long long ldx;
  const int* ids;
  const float* wts;
  const float* sg;           // gate logit of the shared expert, or null
  long long ld_sg;
  const __nv_bfloat16* w1;   // gate/up [E][2F][K]; down [E][N][F]
  const __nv_bfloat16* w1s;
  int E, T, k, K, F, Fs, N;
  float* rows;               // [T*k][F]
  float* rows_s;             // [T][Fs]
  float* h;
  long long ldh;
  int act;                   // 0 SiLU, 2 clamped GLU
  float limit;
};

namespace {

constexpr int AW = 4;        // warps per (row, head)

// One CTA per (row, head): the warps take the keys in turn, a lane owns D/32 value columns; running maximum and sum per
// warp, merged at the end.
template <int DL>
__global__ void __launch_bounds__(AW * 32) attn_exact_kernel(const ExactAttnArgs a) {
  constexpr int D = DL * 32;
  __shared__ float m_s[AW], l_s[AW], o_s[AW][D];
  pdl_wait();
  pdl_launch();
  const int r = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int hk = h / (a.H / a.Hkv), ctx = a.ctx_len[r];
  const int* bt = a.block_table + (size_t)a.slot[r] * a.max_pages;
  float q[DL], o[DL];
#pragma unroll
  for (int i = 0; i < DL; ++i) {
    q[i] = a.q[((size_t)r * a.H + h) * D + i * 32 + lane];
    o[i] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  const int start = a.window > 0 && ctx > a.window ? ctx - a.window : 0, kept = min(a.keep_first, start);
  for (int i = warp; i < ctx - start + kept; i += AW) {
    const int p = i < kept ? i : i - kept + start;
    const int pg = bt[HE_INDEX_OK(p / a.page, a.max_pages, HE_SITE_ATTN_DECODE_PAGE) ? p / a.page : 0];
    const float* kr = a.kv_cache + (((size_t)pg * 2 * a.Hkv + hk) * a.page + p % a.page) * D;
    const float* vr = kr + (size_t)a.Hkv * a.page * D;
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < DL; ++i) s += q[i] * kr[i * 32 + lane];
    s = warp_sum(s) * a.scale;
    if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
    const float mn = fmaxf(m, s), corr = expf(m - mn), w = expf(s - mn);
    l = l * corr + w;
#pragma unroll
    for (int i = 0; i < DL; ++i) o[i] = o[i] * corr + w * vr[i * 32 + lane];
    m = mn;
  }
  if (lane == 0) {
    m_s[warp] = m;
    l_s[warp] = l;
  }
#pragma unroll
  for (int i = 0; i < DL; ++i) o_s[warp][i * 32 + lane] = o[i];
  __syncthreads();
  float mt = -INFINITY, lt = 0.f;
#pragma unroll
  for (int w = 0; w < AW; ++w) mt = fmaxf(mt, m_s[w]);
  if (a.sink != nullptr) {
    mt = fmaxf(mt, a.sink[h]);
    lt = expf(a.sink[h] - mt);
  }
#pragma unroll
  for (int w = 0; w < AW; ++w) lt += l_s[w] > 0.f ? l_s[w] * expf(m_s[w] - mt) : 0.f;
  const float gate = a.head_gate != nullptr ? 1.f / (1.f + expf(-a.head_gate[(size_t)r * a.head_gate_stride + h])) : 1.f;
  for (int d = threadIdx.x; d < D; d += AW * 32) {
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < AW; ++w) v += l_s[w] > 0.f ? o_s[w][d] * expf(m_s[w] - mt) : 0.f;
    a.out[((size_t)r * a.H + h) * D + d] = lt > 0.f ? v / lt * gate : 0.f;
  }
}

__device__ __forceinline__ float dot_row(const __nv_bfloat16* w, const float* x, int n, int lane) {
  float s = 0.f;
  for (int i = lane; i < n; i += 32) s += bf16_to_f32(w[i]) * x[i];
  return warp_sum(s);
}

__device__ __forceinline__ float sigmoid_exact(float x) { return 1.f / (1.f + expf(-x)); }

// grid (T * k [+ T], ceil(max(F, Fs) / 8)), one warp per activation column
__global__ void __launch_bounds__(256) moe_gateup_exact_kernel(const ExactMoeArgs a) {
  pdl_wait();
  pdl_launch();
  const int lane = threadIdx.x & 31, n = blockIdx.y * 8 + (threadIdx.x >> 5), p = blockIdx.x;
  const bool shared = p >= a.T * a.k;
  const int t = shared ? p - a.T * a.k : p / a.k, F = shared ? a.Fs : a.F;
  if (n >= F) return;
  int e = shared ? 0 : a.ids[p];
  if (e < 0 || e >= a.E) e = 0;
  const __nv_bfloat16* base = shared ? a.w1s : a.w1 + (size_t)e * 2 * F * a.K;
  const float* x = a.x + (size_t)t * a.ldx;
  const float g = dot_row(base + (size_t)n * a.K, x, a.K, lane), u = dot_row(base + (size_t)(F + n) * a.K, x, a.K, lane);
  if (lane != 0) return;
  const float wt = shared ? (a.sg != nullptr ? sigmoid_exact(a.sg[(size_t)t * a.ld_sg]) : 1.f) : a.wts[p];
  float v;
  if (a.act == 2) {
    const float gc = fminf(g, a.limit);
    v = gc * sigmoid_exact(1.702f * gc) * (fminf(fmaxf(u, -a.limit), a.limit) + 1.f) * wt;
  } else {
    v = g * sigmoid_exact(g) * u * wt;
  }
  if (shared) a.rows_s[(size_t)t * F + n] = v;
  else a.rows[(size_t)p * F + n] = v;
}

// grid (T, ceil(N / 8)), one warp per output column
__global__ void __launch_bounds__(256) moe_down_exact_kernel(const ExactMoeArgs a) {
  pdl_wait();
  pdl_launch();
  const int lane = threadIdx.x & 31, n = blockIdx.y * 8 + (threadIdx.x >> 5), t = blockIdx.x;
  if (n >= a.N) return;
  float s = 0.f;
  for (int j = 0; j < a.k; ++j) {
    int e = a.ids[(size_t)t * a.k + j];
    if (e < 0 || e >= a.E) e = 0;
    s += dot_row(a.w1 + ((size_t)e * a.N + n) * a.F, a.rows + ((size_t)t * a.k + j) * a.F, a.F, lane);
  }
  if (a.w1s != nullptr) s += dot_row(a.w1s + (size_t)n * a.Fs, a.rows_s + (size_t)t * a.Fs, a.Fs, lane);
  if (lane == 0) a.h[(size_t)t * a.ldh + n] += s;
}

}  // namespace

HE_API int he_attn_exact(const ExactAttnArgs* args, cudaStream_t stream) {
  const ExactAttnArgs& a = *args;
  if (a.R <= 0) return 0;
  if (a.H % a.Hkv != 0) return -HE_ERR_BAD_ARG;
  const dim3 grid(a.R, a.H), block(AW * 32);
  switch (a.D) {
    case 64: return (int)launch_pdl(attn_exact_kernel<2>, grid, block, 0, stream, a);
    case 128: return (int)launch_pdl(attn_exact_kernel<4>, grid, block, 0, stream, a);
    case 256: return (int)launch_pdl(attn_exact_kernel<8>, grid, block, 0, stream, a);
    case 512: return (int)launch_pdl(attn_exact_kernel<16>, grid, block, 0, stream, a);
    default: return -HE_ERR_BAD_ARG;
  }
}
HE_API int he_exact_attn_args_size() { return (int)sizeof(ExactAttnArgs); }

HE_API int he_moe_gateup_exact(const ExactMoeArgs* args, cudaStream_t stream) {
  const ExactMoeArgs& a = *args;
  if (a.T <= 0) return 0;
  if (a.act != 0 && a.act != 2) return -HE_ERR_BAD_ARG;
  const int F = a.w1s != nullptr && a.Fs > a.F ? a.Fs : a.F;
  const dim3 grid(a.T * a.k + (a.w1s != nullptr ? a.T : 0), (F + 7) / 8);
  return (int)launch_pdl(moe_gateup_exact_kernel, grid, dim3(256), 0, stream, a);
}

HE_API int he_moe_down_exact(const ExactMoeArgs* args, cudaStream_t stream) {
  const ExactMoeArgs& a = *args;
  if (a.T <= 0) return 0;
  return (int)launch_pdl(moe_down_exact_kernel, dim3(a.T, (a.N + 7) / 8), dim3(256), 0, stream, a);
}
HE_API int he_exact_moe_args_size() { return (int)sizeof(ExactMoeArgs); }
