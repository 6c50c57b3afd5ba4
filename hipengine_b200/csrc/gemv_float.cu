// Streaming matrix-vector products with bfloat16 weights for 1..16 activation rows (decode and short portions).
//
// One CTA of eight warps owns 16 weight rows (or 16 gate rows and the same 16 up rows); the warps split K in 64-column
// units, so a unit of one row is a full 128-byte line.  The product runs on mma.sync m16n8k16 with the WEIGHTS as the
// 16-row operand and the activation rows as the 8 (or 16) columns: a lane reads 16 consecutive bytes of a weight row
// from global memory straight into fragment registers, because any permutation of the K order is allowed as long as both
// operands use the same one.  Weights pass through no shared memory and are read exactly once; the first unit batch is
// requested before the kernel waits for its predecessor.
//   norm      : RMS norm needs no separate pass: sum over k of w[k] (x[k] g[k]) is scaled by 1/rms(x) at the end, and
//               every warp accumulates the squares of the columns it reads anyway (fp32)
//   epilogue  : fp32 / bf16 store, fp32 residual add, squared ReLU, or act(gate) * up (SiLU, tanh-GELU, clamped GLU)
//   batches   : grid.y repeats the product with other weights and rows (one small matrix per attention head)
//   sums      : the two output projections of a layer whose sublayers run side by side are one launch: each has its own
//               rows and columns, both accumulators get their per-column factors and meet in the residual add
//   recurrence: one token of a gated linear recurrence per row; both gate products of 16 channels end in the CTA that then
//               steps these channels' state and multiplies the output gate in
// The expert forms add an indirection: grid.y is a (token, expert) pair or a token, the weight base comes from the
// routed expert id, and the down projection walks the concatenated columns of all selected experts (and the shared
// one), which adds the k expert outputs in a fixed order inside the accumulator.
#include "common.cuh"
#include "rglru.cuh"

using namespace he;

struct FloatGemvSeg {
  const __nv_bfloat16* w;
  const __nv_bfloat16* w2;   // gate/up pair: the up rows
  void* out;
  const void* x;             // activation rows of this segment (same type and stride as FloatGemvArgs::x); null: those
  long long out_stride;
  int n_rows;
  int epi;                   // 0 f32, 1 bf16, 2 f32 +=, 3 silu(g)*u, 4 gelu_tanh(g)*u, 5 clamped GLU, 6 relu(v)^2 (3..6 bf16)
};

struct FloatGemvArgs {
  FloatGemvSeg seg[4];
  int n_seg;
  int K;                     // columns, multiple of 8
  long long ldw;             // elements between weight rows (all segments)
  int R;
  int x_dtype;               // 0 f32, 1 bf16
  const void* x;
  long long x_stride;
  const float* norm_w;       // fp32 rows only
  float eps;
  int norm_n;                // columns the mean square is taken over (zero-padded rows are wider)
  float limit;               // epi 5
  int n_batch;               // grid.y; every pointer advances by its stride (elements) per batch
  long long w_bs, x_bs, out_bs;
};

struct FloatSumArgs {        // out[r][n] += bias[n] + sum over i of scale_i[n] * (x_i[r] . w_i[n]),  bf16 rows and weights
  const __nv_bfloat16* w[2];
  const __nv_bfloat16* x[2];
  const float* scale[2];     // null: 1
  long long ldw[2], x_stride[2];
  int K[2];                  // multiples of 8; K[1] = 0: one product
  float* out;
  long long out_stride;
  int n_rows, R;
  const float* bias;         // [n_rows] added as well, or null
};

struct FloatMoeArgs {
  const void* x;             // gate/up: rows [T][ldx], fp32 (with norm_w: residual rows) or bf16
  long long ldx;
  const float* norm_w;
  float eps;
  int norm_n;
  const int* ids;            // [T][k]
  const float* wts;          // [T][k]
  const float* sg;           // [T] (stride ld_sg) logit of the shared expert's gate, or null
  long long ld_sg;
  const __nv_bfloat16* w1;   // gate/up: [E][2F][K] (gate rows, then up rows); down: [E][N][F]
  const __nv_bfloat16* w1s;  // shared expert, same form with Fs, or null
  int E, T, k, K, F, Fs, N;
  int act;                   // epilogue code 3..5
  float limit;
  __nv_bfloat16* rows;       // [T*k][F] activations of the selected experts, routing weight folded in
  __nv_bfloat16* rows_s;     // [T][Fs] activations of the shared expert, gate folded in
  float* h;                  // down: residual rows, added in place
  long long ldh;
  int x_dtype;               // 0 f32, 1 bf16
};

namespace {

constexpr int NW = 8;         // warps per CTA
constexpr int UK = 64;        // columns per unit

__device__ __forceinline__ void mma_16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0,
                                          uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack2(float a, float b) {
  __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&h);
}

__device__ __forceinline__ float glu_f(float g, float u, int epi, float limit) {
  if (epi == 3) return silu_f(g) * u;
  if (epi == 4) return gelu_tanh_f(g) * u;
  return clamped_glu_f(g, u, limit);
}

// eight activation values of row `r` at column k as four bf16x2 words (zero outside); fp32 rows are scaled by the norm
// weight and their squares go into ss
template <bool XF32>
__device__ __forceinline__ uint4 load_x(const void* x, size_t off, bool live, const float* norm_w, int k, float& ss) {
  if (!live) return make_uint4(0u, 0u, 0u, 0u);
  if constexpr (XF32) {
    const float4* p = reinterpret_cast<const float4*>(reinterpret_cast<const float*>(x) + off);
    float4 a = p[0], b = p[1];
    if (norm_w != nullptr) {
      ss += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w + b.x * b.x + b.y * b.y + b.z * b.z + b.w * b.w;
      const float4 u = __ldg(reinterpret_cast<const float4*>(norm_w + k));
      const float4 v = __ldg(reinterpret_cast<const float4*>(norm_w + k + 4));
      a.x *= u.x; a.y *= u.y; a.z *= u.z; a.w *= u.w;
      b.x *= v.x; b.y *= v.y; b.z *= v.z; b.w *= v.w;
    }
    return make_uint4(pack2(a.x, a.y), pack2(a.z, a.w), pack2(b.x, b.y), pack2(b.z, b.w));
  } else {
    return *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(x) + off);
  }
}

template <int MT, int NT>
struct Tile {
  float part[NW][MT * 16][NT * 8 + 1];
  float ssq[NW][NT * 8];
};

template <int MT, int NT>
__device__ __forceinline__ void store_partials(Tile<MT, NT>& sm, const float (&acc)[MT][NT][4], float (&ss)[NT]) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, c = lane & 3;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      sm.part[warp][m * 16 + g][n * 8 + 2 * c] = acc[m][n][0];
      sm.part[warp][m * 16 + g][n * 8 + 2 * c + 1] = acc[m][n][1];
      sm.part[warp][m * 16 + g + 8][n * 8 + 2 * c] = acc[m][n][2];
      sm.part[warp][m * 16 + g + 8][n * 8 + 2 * c + 1] = acc[m][n][3];
    }
#pragma unroll
  for (int n = 0; n < NT; ++n) {
    ss[n] += __shfl_xor_sync(0xffffffffu, ss[n], 1);
    ss[n] += __shfl_xor_sync(0xffffffffu, ss[n], 2);
    if (c == 0) sm.ssq[warp][n * 8 + g] = ss[n];
  }
}

template <int MT, int NT>
__device__ __forceinline__ float sum_partials(const Tile<MT, NT>& sm, int row, int col) {
  float v = 0.f;
#pragma unroll
  for (int w = 0; w < NW; ++w) v += sm.part[w][row][col];
  return v;
}

template <int MT, int NT>
__device__ __forceinline__ float inv_rms_of(const Tile<MT, NT>& sm, int col, int n, float eps) {
  float s = 0.f;
#pragma unroll
  for (int w = 0; w < NW; ++w) s += sm.ssq[w][col];
  return rsqrtf(s / (float)n + eps);
}

// acc += W[16 MT rows][K] x[K][8 NT]: this warp's units (every STEP-th one).  wrow[m][half] points at column 8c of row (g + 8 half) of tile m.
// EARLY: the weights do not depend on earlier kernels, so the first batch is requested before griddepcontrol.wait; ``after``
// runs right behind the wait (loads for the epilogue).
struct Nothing {
  __device__ void operator()() const {}
};
template <int MT, int NT, bool XF32, bool EARLY, int STEP = NW, typename After = Nothing>
__device__ __forceinline__ void product(const __nv_bfloat16* const (&wrow)[MT][2], int K, const void* x,
                                        long long x_stride, int R, const float* norm_w, float (&acc)[MT][NT][4],
                                        float (&ss)[NT], After after = After()) {
  constexpr int UN = MT == 1 ? 4 : 2;                    // units in flight per warp: 16 x 16 bytes per lane
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, c = lane & 3;
  const int units = (K + UK - 1) / UK, first = STEP == NW ? warp : 0;
  uint4 A[UN][2][MT][2];
  auto load_a = [&](int u0) {
#pragma unroll
    for (int i = 0; i < UN; ++i)
#pragma unroll
      for (int s = 0; s < 2; ++s) {
        const int k = (u0 + i * STEP) * UK + s * 32;
        const bool live = k + 8 * c < K;
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int hf = 0; hf < 2; ++hf)
            A[i][s][m][hf] = live ? ldg128_stream(wrow[m][hf] + k) : make_uint4(0u, 0u, 0u, 0u);
      }
  };
  if (EARLY) {
    load_a(first);
    pdl_wait();
    after();
  }
  for (int u0 = first; u0 < units; u0 += UN * STEP) {
    if (!EARLY || u0 != first) load_a(u0);
#pragma unroll
    for (int i = 0; i < UN; ++i)
#pragma unroll
      for (int s = 0; s < 2; ++s) {
        const int k = (u0 + i * STEP) * UK + s * 32 + 8 * c;
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          const int r = n * 8 + g;
          const uint4 b = load_x<XF32>(x, (size_t)r * x_stride + k, r < R && k < K, norm_w, k, ss[n]);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma_16816(acc[m][n], A[i][s][m][0].x, A[i][s][m][1].x, A[i][s][m][0].y, A[i][s][m][1].y, b.x, b.y);
            mma_16816(acc[m][n], A[i][s][m][0].z, A[i][s][m][1].z, A[i][s][m][0].w, A[i][s][m][1].w, b.z, b.w);
          }
        }
      }
  }
}

// grid: items of all segments (16 rows, or 16 gate/up row pairs when MT == 2)
template <int MT, int NT, bool XF32>
__global__ void __launch_bounds__(NW * 32, 2) gemv_float_kernel(const __grid_constant__ FloatGemvArgs a) {
  __shared__ Tile<MT, NT> sm;
  pdl_launch();
  const int lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
  int item = blockIdx.x, si = 0;
  while (si < a.n_seg - 1 && item >= (a.seg[si].n_rows + 15) / 16) {
    item -= (a.seg[si].n_rows + 15) / 16;
    ++si;
  }
  const FloatGemvSeg& sg = a.seg[si];
  const int row0 = item * 16;
  const size_t bt = blockIdx.y;
  const size_t x_off = bt * a.x_bs, o_off = bt * a.out_bs;
  const void* xs = sg.x != nullptr ? sg.x : a.x;
  xs = XF32 ? (const void*)(reinterpret_cast<const float*>(xs) + x_off)
            : (const void*)(reinterpret_cast<const __nv_bfloat16*>(xs) + x_off);
  const __nv_bfloat16* wrow[MT][2];
#pragma unroll
  for (int hf = 0; hf < 2; ++hf) {
    const size_t off = bt * a.w_bs + (size_t)min(row0 + g + 8 * hf, sg.n_rows - 1) * a.ldw + 8 * c;
    wrow[0][hf] = sg.w + off;
    if constexpr (MT == 2) wrow[1][hf] = sg.w2 + off;
  }
  float acc[MT][NT][4] = {};
  float ss[NT] = {};
  product<MT, NT, XF32, true>(wrow, a.K, xs, a.x_stride, a.R, a.norm_w, acc, ss);
  store_partials<MT, NT>(sm, acc, ss);
  __syncthreads();
  for (int o = threadIdx.x; o < 16 * NT * 8; o += NW * 32) {
    const int row = o & 15, col = o >> 4, n = row0 + row;
    if (col >= a.R || n >= sg.n_rows) continue;
    const float inv = a.norm_w != nullptr ? inv_rms_of<MT, NT>(sm, col, a.norm_n, a.eps) : 1.f;
    const float v = sum_partials<MT, NT>(sm, row, col) * inv;
    const size_t off = o_off + (size_t)col * sg.out_stride + n;
    if constexpr (MT == 2) {
      const float u = sum_partials<MT, NT>(sm, 16 + row, col) * inv;
      reinterpret_cast<__nv_bfloat16*>(sg.out)[off] = f32_to_bf16(glu_f(v, u, sg.epi, a.limit));
    } else if (sg.epi == 0) {
      reinterpret_cast<float*>(sg.out)[off] = v;
    } else if (sg.epi == 1 || sg.epi == 6) {
      reinterpret_cast<__nv_bfloat16*>(sg.out)[off] = f32_to_bf16(sg.epi == 6 ? relu2_f(v) : v);
    } else {
      reinterpret_cast<float*>(sg.out)[off] += v;
    }
  }
}

// Short rows (K too small to share between the warps of a CTA): every warp owns 16 output columns and all of K.
// grid (ceil(n_rows / 128), batches), one segment, plain store
template <int NT, bool XF32>
__global__ void __launch_bounds__(NW * 32, 2) gemv_short_kernel(const __grid_constant__ FloatGemvArgs a) {
  pdl_launch();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, c = lane & 3;
  const FloatGemvSeg& sg = a.seg[0];
  const size_t bt = blockIdx.y;
  const int row0 = (blockIdx.x * NW + warp) * 16;
  if (row0 >= sg.n_rows) return;
  const void* xs = XF32 ? (const void*)(reinterpret_cast<const float*>(a.x) + bt * a.x_bs)
                        : (const void*)(reinterpret_cast<const __nv_bfloat16*>(a.x) + bt * a.x_bs);
  const __nv_bfloat16* w0 = sg.w + bt * a.w_bs + 8 * c;
  const __nv_bfloat16* wrow[1][2] = {{w0 + (size_t)min(row0 + g, sg.n_rows - 1) * a.ldw,
                                      w0 + (size_t)min(row0 + g + 8, sg.n_rows - 1) * a.ldw}};
  float acc[1][NT][4] = {};
  float ss[NT] = {};
  product<1, NT, XF32, true, 1>(wrow, a.K, xs, a.x_stride, a.R, nullptr, acc, ss);
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int row = row0 + g + (e >> 1) * 8, col = n * 8 + 2 * c + (e & 1);
      if (row >= sg.n_rows || col >= a.R) continue;
      const size_t off = bt * a.out_bs + (size_t)col * sg.out_stride + row;
      if (sg.epi == 0) reinterpret_cast<float*>(sg.out)[off] = acc[0][n][e];
      else reinterpret_cast<__nv_bfloat16*>(sg.out)[off] = f32_to_bf16(acc[0][n][e]);
    }
}

// grid: items of 16 output columns
template <int NT>
__global__ void __launch_bounds__(NW * 32, 2) gemv_sum_kernel(const __grid_constant__ FloatSumArgs a) {
  __shared__ Tile<1, NT> sm;
  pdl_launch();
  const int lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
  const int row0 = blockIdx.x * 16;
  const int ra = min(row0 + g, a.n_rows - 1), rb = min(row0 + g + 8, a.n_rows - 1);
  const __nv_bfloat16* wrow[1][2] = {{a.w[0] + (size_t)ra * a.ldw[0] + 8 * c, a.w[0] + (size_t)rb * a.ldw[0] + 8 * c}};
  float acc[1][NT][4] = {};
  float ss[NT] = {};
  product<1, NT, false, true>(wrow, a.K[0], a.x[0], a.x_stride[0], a.R, nullptr, acc, ss);
  if (a.scale[0] != nullptr) {
    const float sa = a.scale[0][ra], sb = a.scale[0][rb];
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      acc[0][n][0] *= sa; acc[0][n][1] *= sa;
      acc[0][n][2] *= sb; acc[0][n][3] *= sb;
    }
  }
  if (a.K[1] > 0) {
    wrow[0][0] = a.w[1] + (size_t)ra * a.ldw[1] + 8 * c;
    wrow[0][1] = a.w[1] + (size_t)rb * a.ldw[1] + 8 * c;
    float acc2[1][NT][4] = {};
    product<1, NT, false, false>(wrow, a.K[1], a.x[1], a.x_stride[1], a.R, nullptr, acc2, ss);
    const float sa = a.scale[1] != nullptr ? a.scale[1][ra] : 1.f, sb = a.scale[1] != nullptr ? a.scale[1][rb] : 1.f;
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      acc[0][n][0] += sa * acc2[0][n][0]; acc[0][n][1] += sa * acc2[0][n][1];
      acc[0][n][2] += sb * acc2[0][n][2]; acc[0][n][3] += sb * acc2[0][n][3];
    }
  }
  store_partials<1, NT>(sm, acc, ss);
  __syncthreads();
  for (int o = threadIdx.x; o < 16 * NT * 8; o += NW * 32) {
    const int row = o & 15, col = o >> 4, n = row0 + row;
    if (col < a.R && n < a.n_rows)
      a.out[(size_t)col * a.out_stride + n] += sum_partials<1, NT>(sm, row, col) + (a.bias != nullptr ? a.bias[n] : 0.f);
  }
}

// grid (ceil(max(F, Fs) / 16), T * k [+ T]): activation rows of the selected experts, then of the shared expert
template <bool XF32>
__global__ void __launch_bounds__(NW * 32, 2) moe_gateup_float_kernel(const __grid_constant__ FloatMoeArgs a) {
  __shared__ Tile<2, 1> sm;
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
  const int p = blockIdx.y;
  const bool shared = p >= a.T * a.k;
  const int t = shared ? p - a.T * a.k : p / a.k;
  const int F = shared ? a.Fs : a.F;
  const int row0 = blockIdx.x * 16;
  if (row0 >= F) return;
  int e = shared ? 0 : a.ids[p];
  if (!shared && (!HE_INDEX_OK(e, a.E, HE_SITE_MOE_EXPERT_ID) || e < 0 || e >= a.E)) e = 0;
  const __nv_bfloat16* base = shared ? a.w1s : a.w1 + (size_t)e * 2 * F * a.K;
  const __nv_bfloat16* wrow[2][2];
#pragma unroll
  for (int hf = 0; hf < 2; ++hf) {
    const int r = min(row0 + g + 8 * hf, F - 1);
    wrow[0][hf] = base + (size_t)r * a.K + 8 * c;
    wrow[1][hf] = base + (size_t)(F + r) * a.K + 8 * c;
  }
  float acc[2][1][4] = {};
  float ss[1] = {};
  const char* x = reinterpret_cast<const char*>(a.x) + (size_t)t * a.ldx * (XF32 ? 4 : 2);
  product<2, 1, XF32, false>(wrow, a.K, x, a.ldx, 1, a.norm_w, acc, ss);
  store_partials<2, 1>(sm, acc, ss);
  __syncthreads();
  const int row = threadIdx.x, n = row0 + row;
  if (row < 16 && n < F) {
    const float inv = a.norm_w != nullptr ? inv_rms_of<2, 1>(sm, 0, a.norm_n, a.eps) : 1.f;
    const float gv = sum_partials<2, 1>(sm, row, 0) * inv, uv = sum_partials<2, 1>(sm, 16 + row, 0) * inv;
    const float wt = shared ? (a.sg != nullptr ? sigmoid_f(a.sg[(size_t)t * a.ld_sg]) : 1.f) : a.wts[p];
    const float v = glu_f(gv, uv, a.act, a.limit) * wt;
    if (shared) a.rows_s[(size_t)t * F + n] = f32_to_bf16(v);
    else a.rows[(size_t)p * F + n] = f32_to_bf16(v);
  }
}

// grid (ceil(N / 16), T): h[t] += sum over the token's experts (and the shared one) of W_down row . activation row
__global__ void __launch_bounds__(NW * 32, 2) moe_down_float_kernel(const __grid_constant__ FloatMoeArgs a) {
  __shared__ Tile<1, 1> sm;
  __shared__ int e_s[32];
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, c = lane & 3;
  const int t = blockIdx.y, row0 = blockIdx.x * 16;
  if (threadIdx.x < a.k) {
    int e = a.ids[(size_t)t * a.k + threadIdx.x];
    if (!HE_INDEX_OK(e, a.E, HE_SITE_MOE_EXPERT_ID) || e < 0 || e >= a.E) e = 0;
    e_s[threadIdx.x] = e;
  }
  __syncthreads();
  const int upe = (a.F + UK - 1) / UK, ups = a.w1s != nullptr ? (a.Fs + UK - 1) / UK : 0;
  const int units = a.k * upe + ups;
  const int ra = min(row0 + g, a.N - 1), rb = min(row0 + g + 8, a.N - 1);
  float acc[1][1][4] = {};
  float ss[1] = {};
  constexpr int UN = 4;
  for (int u0 = warp; u0 < units; u0 += UN * NW) {
    uint4 A[UN][2][2], B[UN][2];
#pragma unroll
    for (int i = 0; i < UN; ++i) {
      const int u = u0 + i * NW;
      const bool sh = u >= a.k * upe;
      const int j = sh ? 0 : u / upe;
      const int k0 = (sh ? u - a.k * upe : u - j * upe) * UK;
      const int F = sh ? a.Fs : a.F;
      const __nv_bfloat16* wb = sh ? a.w1s : a.w1 + (size_t)e_s[j] * a.N * F;
      const __nv_bfloat16* xb = sh ? a.rows_s + (size_t)t * F : a.rows + ((size_t)t * a.k + j) * F;
#pragma unroll
      for (int s = 0; s < 2; ++s) {
        const int k = k0 + s * 32 + 8 * c;
        const bool live = u < units && k < F;
        A[i][s][0] = live ? ldg128_stream(wb + (size_t)ra * F + k) : make_uint4(0u, 0u, 0u, 0u);
        A[i][s][1] = live ? ldg128_stream(wb + (size_t)rb * F + k) : make_uint4(0u, 0u, 0u, 0u);
        B[i][s] = live && g == 0 ? *reinterpret_cast<const uint4*>(xb + k) : make_uint4(0u, 0u, 0u, 0u);
      }
    }
#pragma unroll
    for (int i = 0; i < UN; ++i)
#pragma unroll
      for (int s = 0; s < 2; ++s) {
        mma_16816(acc[0][0], A[i][s][0].x, A[i][s][1].x, A[i][s][0].y, A[i][s][1].y, B[i][s].x, B[i][s].y);
        mma_16816(acc[0][0], A[i][s][0].z, A[i][s][1].z, A[i][s][0].w, A[i][s][1].w, B[i][s].z, B[i][s].w);
      }
  }
  store_partials<1, 1>(sm, acc, ss);
  __syncthreads();
  const int n = row0 + (int)threadIdx.x;
  if (threadIdx.x < 16 && n < a.N) a.h[(size_t)t * a.ldh + n] += sum_partials<1, 1>(sm, threadIdx.x, 0);
}

// One token of every segment through the gated linear recurrence: segment r is row r.  grid (ceil(block_cols / 16), blocks)
template <int NT>
__global__ void __launch_bounds__(NW * 32, 2) rglru_step_kernel(const __grid_constant__ RglruArgs a) {
  __shared__ Tile<2, NT> sm;
  pdl_launch();
  const int lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3, bc = a.block_cols, b = blockIdx.y, row0 = blockIdx.x * 16;
  const __nv_bfloat16* wrow[2][2];
#pragma unroll
  for (int hf = 0; hf < 2; ++hf) {
    const int n = min(row0 + g + 8 * hf, bc - 1);
    wrow[0][hf] = a.gw + ((size_t)b * 2 * bc + n) * bc + 8 * c;
    wrow[1][hf] = wrow[0][hf] + (size_t)bc * bc;
  }
  const __nv_bfloat16* u = reinterpret_cast<const __nv_bfloat16*>(a.u) + (size_t)b * a.u_bs;
  float acc[2][NT][4] = {};
  float ss[NT] = {};
  // what the epilogue of this thread's channel and token needs, requested ahead of the product
  static_assert(16 * NT * 8 <= NW * 32, "one output per thread");
  constexpr int PAST = 3;                                  // convolution inputs kept in registers
  const int row = threadIdx.x & 15, r = threadIdx.x >> 4, n = row0 + row, ch = b * bc + n, past = a.taps - 1;
  int slot = 0;
  bool live = r < NT * 8 && r < a.n_seg && n < bc;
  float S = 0.f, y = 0.f, un = 0.f, dec = 0.f, g0 = 0.f, g1 = 0.f, x = 0.f, hist[PAST] = {};
  const auto ahead = [&]() {
    if (!live) return;
    slot = a.seg_slot[r];
    if (!HE_INDEX_OK(slot, a.n_slots, HE_SITE_STATE_SLOT)) {
      live = false;
      return;
    }
    S = a.S[(size_t)slot * a.C + ch];
    y = rg_load(a.y, a.row_dtype == 0, (size_t)r * a.row_stride + ch) + a.yb[ch];
    un = bf16_to_f32(u[(size_t)r * a.u_ts + n]);
    dec = a.decay[ch];
    g0 = a.gb[(size_t)b * 2 * bc + n];
    g1 = a.gb[(size_t)b * 2 * bc + bc + n];
    if (past >= 1 && past <= PAST) {
      x = rg_load(a.x, a.row_dtype == 0, (size_t)r * a.row_stride + ch) + a.xb[ch];
#pragma unroll
      for (int j = 1; j < PAST; ++j)
        if (j < past) hist[j] = a.cstate[((size_t)slot * past + j) * a.C + ch];
    }
  };
  product<2, NT, false, true, NW>(wrow, bc, u, a.u_ts, a.n_seg, nullptr, acc, ss, ahead);
  store_partials<2, NT>(sm, acc, ss);
  __syncthreads();
  if (!live) return;
  float av, dv;
  rg_gates(sum_partials<2, NT>(sm, row, r) + g0, sum_partials<2, NT>(sm, 16 + row, r) + g1, dec, un, av, dv);
  S = av * S + dv;
  a.S[(size_t)slot * a.C + ch] = S;
  reinterpret_cast<__nv_bfloat16*>(a.out)[(size_t)r * a.out_stride + ch] = f32_to_bf16(S * rg_gelu(y));
  if (past > PAST) {
    rg_conv_state(a, slot, ch, r, 1);
    return;
  }
#pragma unroll
  for (int j = 1; j <= PAST; ++j)
    if (j <= past) a.cstate[((size_t)slot * past + j - 1) * a.C + ch] = j == past ? x : hist[j < PAST ? j : 0];
}

template <int MT>
int launch_rows(const FloatGemvArgs& a, int items, cudaStream_t stream) {
  cudaError_t e;
  const dim3 grid(items, a.n_batch > 1 ? a.n_batch : 1), block(NW * 32);
  if (a.x_dtype == 0) {
    e = a.R <= 8 ? launch_pdl(gemv_float_kernel<MT, 1, true>, grid, block, 0, stream, a)
                 : launch_pdl(gemv_float_kernel<MT, 2, true>, grid, block, 0, stream, a);
  } else {
    e = a.R <= 8 ? launch_pdl(gemv_float_kernel<MT, 1, false>, grid, block, 0, stream, a)
                 : launch_pdl(gemv_float_kernel<MT, 2, false>, grid, block, 0, stream, a);
  }
  return (int)e;
}

}  // namespace

// Rows of x (fp32 with an optional fused RMS norm, or bf16) times up to four bf16 weight segments of the same width.
// All segments of a launch are plain (epi 0..2, 6) or all are gate/up pairs (epi 3..5).
HE_API int he_gemv_float(const FloatGemvArgs* args, cudaStream_t stream) {
  const FloatGemvArgs& a = *args;
  if (a.R < 1 || a.R > 16 || a.n_seg < 1 || a.n_seg > 4 || a.K <= 0 || a.K % 8 != 0 || a.ldw % 8 != 0 || a.ldw < a.K)
    return -HE_ERR_BAD_ARG;
  if (a.x_stride % 8 != 0 || (a.norm_w != nullptr && (a.x_dtype != 0 || a.norm_n <= 0))) return -HE_ERR_BAD_ARG;
  const auto is_pair = [](int epi) { return epi >= 3 && epi <= 5; };
  const bool pair = is_pair(a.seg[0].epi);
  if (a.n_batch > 65535 || a.w_bs % 8 != 0 || a.x_bs % 8 != 0) return -HE_ERR_BAD_ARG;
  int items = 0;
  for (int i = 0; i < a.n_seg; ++i) {
    if (is_pair(a.seg[i].epi) != pair || a.seg[i].epi < 0 || a.seg[i].epi > 6 || a.seg[i].n_rows <= 0 ||
        (pair && a.seg[i].w2 == nullptr))
      return -HE_ERR_BAD_ARG;
    items += (a.seg[i].n_rows + 15) / 16;
  }
  if (a.n_seg == 1 && a.norm_w == nullptr && a.seg[0].epi <= 1 && a.seg[0].x == nullptr && a.K <= 4 * UK && a.n_batch > 1) {
    const dim3 grid((a.seg[0].n_rows + NW * 16 - 1) / (NW * 16), a.n_batch), block(NW * 32);
    if (a.x_dtype == 0)
      return (int)(a.R <= 8 ? launch_pdl(gemv_short_kernel<1, true>, grid, block, 0, stream, a)
                            : launch_pdl(gemv_short_kernel<2, true>, grid, block, 0, stream, a));
    return (int)(a.R <= 8 ? launch_pdl(gemv_short_kernel<1, false>, grid, block, 0, stream, a)
                          : launch_pdl(gemv_short_kernel<2, false>, grid, block, 0, stream, a));
  }
  return pair ? launch_rows<2>(a, items, stream) : launch_rows<1>(a, items, stream);
}
HE_API int he_gemv_float_args_size() { return (int)sizeof(FloatGemvArgs); }

HE_API int he_gemv_sum(const FloatSumArgs* args, cudaStream_t stream) {
  const FloatSumArgs& a = *args;
  if (a.R < 1 || a.R > 16 || a.n_rows <= 0 || a.K[0] <= 0 || a.K[1] < 0) return -HE_ERR_BAD_ARG;
  for (int i = 0; i < (a.K[1] > 0 ? 2 : 1); ++i)
    if (a.K[i] % 8 != 0 || a.ldw[i] % 8 != 0 || a.ldw[i] < a.K[i] || a.x_stride[i] % 8 != 0) return -HE_ERR_BAD_ARG;
  const dim3 grid((a.n_rows + 15) / 16), block(NW * 32);
  return (int)(a.R <= 8 ? launch_pdl(gemv_sum_kernel<1>, grid, block, 0, stream, a)
                        : launch_pdl(gemv_sum_kernel<2>, grid, block, 0, stream, a));
}
HE_API int he_gemv_sum_args_size() { return (int)sizeof(FloatSumArgs); }

HE_API int he_rglru_step(const RglruArgs* args, cudaStream_t stream) {
  const RglruArgs& a = *args;
  if (a.n_seg <= 0) return 0;
  if (a.n_seg > 16 || a.block_cols <= 0 || a.block_cols % 8 != 0 || a.C % a.block_cols != 0 || a.taps < 1 || a.act_f32 != 0 ||
      a.gw == nullptr || a.journal != nullptr || a.u_ts % 8 != 0 || a.u_bs % 8 != 0 || a.C / a.block_cols > 65535)
    return -HE_ERR_BAD_ARG;
  const dim3 grid((a.block_cols + 15) / 16, a.C / a.block_cols), block(NW * 32);
  return (int)(a.n_seg <= 8 ? launch_pdl(rglru_step_kernel<1>, grid, block, 0, stream, a)
                            : launch_pdl(rglru_step_kernel<2>, grid, block, 0, stream, a));
}

static int check_moe(const FloatMoeArgs& a) {
  if (a.k <= 0 || a.k > 32 || a.E < a.k || a.F <= 0 || a.F % 8 != 0 || (a.w1s != nullptr && (a.Fs <= 0 || a.Fs % 8 != 0)))
    return -HE_ERR_BAD_ARG;
  return 0;
}

HE_API int he_moe_gateup_float(const FloatMoeArgs* args, cudaStream_t stream) {
  const FloatMoeArgs& a = *args;
  if (a.T <= 0) return 0;
  if (check_moe(a) != 0 || a.K % 8 != 0 || a.ldx % 8 != 0 || a.act < 3 || a.act > 5 ||
      (a.x_dtype != 0 && a.norm_w != nullptr))
    return -HE_ERR_BAD_ARG;
  const int F = a.w1s != nullptr && a.Fs > a.F ? a.Fs : a.F;
  const dim3 grid((F + 15) / 16, a.T * a.k + (a.w1s != nullptr ? a.T : 0));
  return (int)(a.x_dtype == 0 ? launch_pdl(moe_gateup_float_kernel<true>, grid, dim3(NW * 32), 0, stream, a)
                              : launch_pdl(moe_gateup_float_kernel<false>, grid, dim3(NW * 32), 0, stream, a));
}

HE_API int he_moe_down_float(const FloatMoeArgs* args, cudaStream_t stream) {
  const FloatMoeArgs& a = *args;
  if (a.T <= 0) return 0;
  if (check_moe(a) != 0 || a.N <= 0) return -HE_ERR_BAD_ARG;
  return (int)launch_pdl(moe_down_float_kernel, dim3((a.N + 15) / 16, a.T), dim3(NW * 32), 0, stream, a);
}
HE_API int he_moe_float_args_size() { return (int)sizeof(FloatMoeArgs); }
