// Latent attention over a paged latent cache: cache write with rotation, single-token / short-portion attention, gather for
// long portions, and the fp32 forms.
//
// A token's cache row is [latent (rank columns, zero-padded to a multiple of 16) | rotated key part | zeros] of W columns
// (a multiple of 32); the plane of a layer run is [n_pages][page][W].  A head's key is a linear map of the latent plus the
// rotated part, its value another linear map of the latent.  Decode never builds them: the key map is moved onto the query
// (q_lat = [W_k^T q | rotated q], W columns) and the value map behind the weighted sum, so all heads of a request attend to
// one W-wide row per token, which is read once and serves as key and value.
#include "latent_segs.cuh"

using namespace he;

struct LatentPostArgs {
  const void* down;          // [T][down_stride]: rank latent columns, then rot_dim
  const void* q;             // [T][q_stride]: H heads of [dn unrotated | rotated], q_cols each
  const float* norm_w;       // [rank_cols] gains of the latent norm (zero in padded columns)
  const double* freq;        // [rot_dim / 2]
  void* cache;               // [n_pages][page][W]
  void* q_out;               // [T][H][q_cols] or null; may be q itself when the types agree
  void* q_lat;               // [T][H][W] or null: columns [rank_cols, W) are written here
  const int* block_table;    // [n_slots][max_pages]
  const int* slot;           // [T]
  const int* pos;            // [T]
  long long down_stride, q_stride;
  int down_dtype, q_dtype;   // 0 f32, 1 bf16
  int out_f32;               // type of cache, q_out and q_lat
  int T, H, dn, rot_dim, q_cols, rank, rank_cols, W, page, max_pages;
  float eps, amp;
};

struct LatentDecArgs {
  const void* q;             // [R][H][W]
  const void* cache;         // [n_pages][page][W]
  const int* block_table;
  const int* slot;           // [R]
  const int* ctx_len;        // [R] keys up to and including the row's own
  float* partial;            // [R][H][max_splits][rank_cols], then (maximum, sum) [R][H][max_splits][2]
  void* out;                 // [R][H][rank_cols]
  const float* sink;         // [H] or null: one more term in the softmax denominator
  int R, H, W, rank_cols, page, max_pages, split_len, max_splits, window;
  float scale;
};

struct LatentGatherArgs {
  const __nv_bfloat16* cache;
  const int* block_table;
  const int* seg_start;      // [n_seg + 1] absolute rows
  const int* seg_slot;       // [n_seg]
  const int* pos;            // [rows]
  __nv_bfloat16* out;        // [keys][W]
  int n_seg, keys, W, page, max_pages, window;
};

namespace {

__device__ __forceinline__ float load_in(const void* p, int dtype, size_t i) {
  return dtype == 0 ? reinterpret_cast<const float*>(p)[i] : bf16_to_f32(reinterpret_cast<const __nv_bfloat16*>(p)[i]);
}
template <typename T>
__device__ __forceinline__ T from_f32(float v) {
  if constexpr (sizeof(T) == 2) return f32_to_bf16(v);
  else return v;
}

constexpr int POST_HEADS = 8;      // heads per CTA of the query part

// grid (T, 1 + ceil(H / POST_HEADS)): y = 0 norms the latent and writes the cache row, the others rotate query heads
template <typename OutT>
__global__ void __launch_bounds__(256) latent_post_kernel(const LatentPostArgs a) {
  extern __shared__ float2 cs[];     // [rot_dim / 2] (cos, sin) times the amplitude
  __shared__ float red[33];
  pdl_wait();
  pdl_launch();
  const int t = blockIdx.x, p = a.pos[t], half = a.rot_dim / 2;
  for (int i = threadIdx.x; i < half; i += 256) {
    // the angle is reduced to one turn in double, so late positions keep full fp32 accuracy
    const double two_pi = 6.283185307179586476925286766559;
    const double ang = (double)p * a.freq[i];
    float sn, c;
    sincosf((float)(ang - two_pi * rint(ang / two_pi)), &sn, &c);
    cs[i] = make_float2(c * a.amp, sn * a.amp);
  }
  if (blockIdx.y == 0) {
    const size_t in0 = (size_t)t * a.down_stride;
    float ss = 0.f;
    for (int i = threadIdx.x; i < a.rank; i += 256) {
      const float v = load_in(a.down, a.down_dtype, in0 + i);
      ss += v * v;
    }
    const float inv = rsqrtf(block_sum(ss, red) / (float)a.rank + a.eps);     // its barriers also publish cs
    const int pi = p / a.page;
    if (!HE_INDEX_OK(pi, a.max_pages, HE_SITE_KV_WRITE_PAGE)) return;
    const int pg = a.block_table[(size_t)a.slot[t] * a.max_pages + pi];
    OutT* row = reinterpret_cast<OutT*>(a.cache) + ((size_t)pg * a.page + p % a.page) * a.W;
    for (int i = threadIdx.x; i < a.rank_cols; i += 256)
      row[i] = from_f32<OutT>(i < a.rank ? load_in(a.down, a.down_dtype, in0 + i) * inv * a.norm_w[i] : 0.f);
    for (int i = threadIdx.x; 2 * i < a.W - a.rank_cols; i += 256) {
      float u = 0.f, v = 0.f;
      if (i < half) {
        const float x = load_in(a.down, a.down_dtype, in0 + a.rank + 2 * i);
        const float y = load_in(a.down, a.down_dtype, in0 + a.rank + 2 * i + 1);
        u = x * cs[i].x - y * cs[i].y;
        v = y * cs[i].x + x * cs[i].y;
      }
      row[a.rank_cols + 2 * i] = from_f32<OutT>(u);
      row[a.rank_cols + 2 * i + 1] = from_f32<OutT>(v);
    }
    return;
  }
  __syncthreads();
  const int h0 = (blockIdx.y - 1) * POST_HEADS, nh = min(POST_HEADS, a.H - h0);
  const bool copy = a.q_out != nullptr && a.q_out != a.q;
  const int lat_pairs = (a.W - a.rank_cols) / 2, rot_pairs = max((a.q_cols - a.dn) / 2, lat_pairs);
  const int skip = copy ? 0 : a.dn / 2, pairs = a.dn / 2 + rot_pairs - skip;
  for (int e = threadIdx.x; e < nh * pairs; e += 256) {
    const int h = h0 + e / pairs, j = e % pairs + skip, i = j - a.dn / 2;     // pair j of the head, pair i of its rotated part
    const size_t qi = (size_t)t * a.q_stride + (size_t)h * a.q_cols + 2 * j;
    float u = 0.f, v = 0.f;
    if (i < half) {
      u = load_in(a.q, a.q_dtype, qi);
      v = load_in(a.q, a.q_dtype, qi + 1);
      if (i >= 0) {
        const float x = u, y = v;
        u = x * cs[i].x - y * cs[i].y;
        v = y * cs[i].x + x * cs[i].y;
      }
    }
    if (a.q_out != nullptr && 2 * j < a.q_cols) {
      OutT* o = reinterpret_cast<OutT*>(a.q_out) + ((size_t)t * a.H + h) * a.q_cols + 2 * j;
      o[0] = from_f32<OutT>(u);
      o[1] = from_f32<OutT>(v);
    }
    if (a.q_lat != nullptr && i >= 0 && i < lat_pairs) {
      OutT* o = reinterpret_cast<OutT*>(a.q_lat) + ((size_t)t * a.H + h) * a.W + a.rank_cols + 2 * i;
      o[0] = from_f32<OutT>(u);
      o[1] = from_f32<OutT>(v);
    }
  }
}

// ---------------------------------------------------------------- split-K attention of single rows
__device__ __forceinline__ void cp_async16(void* smem, const void* gmem) {
  const uint32_t s = (uint32_t)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(s), "l"(gmem) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

constexpr int DEC_WARPS = 16;

template <int MT, int TK>
__host__ __device__ inline size_t dec_smem(int W) {
  return (size_t)(MT * 16 + 2 * TK) * (W * 2 + 16) +
         (size_t)MT * 16 * ((256 / TK) * (TK + 4) * 4 + (TK * 2 + 16)) + MT * 16 * 3 * 4;
}

// One CTA per (key span, chunk of up to 16 MT heads, row).  Tiles of TK latent rows are double-buffered with cp.async (rows
// padded by 16 bytes: conflict-free ldmatrix).  Per tile: partial scores (the warps split 16-key groups and the columns, so
// the queries are read from shared memory TK / 16 times and not once per warp), running maximum and sum per head, then the
// weighted sum (a warp owns every sixteenth block of 16 latent columns, up to NB blocks).
template <int MT, int NB, int TK>
__global__ void __launch_bounds__(DEC_WARPS * 32) latent_decode_kernel(const LatentDecArgs a) {
  extern __shared__ __align__(16) uint8_t smem[];
  constexpr int MR = MT * 16, SP = TK + 4, PP = TK * 2 + 16;
  constexpr int KG = TK / 16, KS = DEC_WARPS / KG;        // key groups, column shares
  const int pitch = a.W * 2 + 16, chunks16 = a.W / 8;
  uint8_t* q_s = smem;                                    // [MR][pitch]
  uint8_t* kv_s = q_s + (size_t)MR * pitch;               // [2][TK][pitch]
  uint8_t* p_s = kv_s + (size_t)2 * TK * pitch;           // [MR][PP] bf16 weights
  float* sc = reinterpret_cast<float*>(p_s + MR * PP);    // [KS][MR][SP] partial scores
  float* m_s = sc + KS * MR * SP;
  float* l_s = m_s + MR;
  float* corr_s = l_s + MR;
  const int sp = blockIdx.x, r = blockIdx.z, per = (a.H + gridDim.y - 1) / gridDim.y, h0 = blockIdx.y * per;
  const int gc = min(per, a.H - h0);
  pdl_wait();
  pdl_launch();
  if (gc <= 0) return;
  const int ctx = a.ctx_len[r];
  const int start = (a.window > 0 && ctx > a.window) ? ctx - a.window : 0;
  const int k0 = start + sp * a.split_len;
  if (k0 >= ctx) return;
  const int n = min(a.split_len, ctx - k0), n_tiles = (n + TK - 1) / TK;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c = lane & 3;
  const int* bt = a.block_table + (size_t)a.slot[r] * a.max_pages;
  const __nv_bfloat16* cache = reinterpret_cast<const __nv_bfloat16*>(a.cache);

  auto load_tile = [&](int t, int buf) {
    for (int i = warp; i < TK; i += DEC_WARPS) {
      const int pos = k0 + min(t * TK + i, n - 1);        // rows past the span repeat its last key; their weight is zero
      const int pi = pos / a.page;
      const int pg = bt[HE_INDEX_OK(pi, a.max_pages, HE_SITE_ATTN_DECODE_PAGE) ? pi : 0];
      const __nv_bfloat16* src = cache + ((size_t)pg * a.page + pos % a.page) * a.W;
      uint8_t* dst = kv_s + ((size_t)buf * TK + i) * pitch;
      for (int ch = lane; ch < chunks16; ch += 32) cp_async16(dst + ch * 16, src + ch * 8);
    }
  };
  load_tile(0, 0);
  cp_async_commit();
  const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(a.q) + ((size_t)r * a.H + h0) * a.W;
  for (int i = warp; i < MR; i += DEC_WARPS)
    for (int ch = lane; ch < chunks16; ch += 32)
      *reinterpret_cast<uint4*>(q_s + (size_t)i * pitch + ch * 16) =
          i < gc ? *reinterpret_cast<const uint4*>(q + (size_t)i * a.W + ch * 8) : make_uint4(0u, 0u, 0u, 0u);
  for (int i = tid; i < MR * PP / 16; i += DEC_WARPS * 32) reinterpret_cast<uint4*>(p_s)[i] = make_uint4(0u, 0u, 0u, 0u);
  if (tid < MR) {
    m_s[tid] = -INFINITY;
    l_s[tid] = 0.f;
    corr_s[tid] = 0.f;
  }

  const int n_blk = a.rank_cols / 16, kg = warp % KG, kq = warp / KG;
  float o[MT][NB][2][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < NB; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[m][j][0][e] = o[m][j][1][e] = 0.f;

  for (int t = 0; t < n_tiles; ++t) {
    const int buf = t & 1, live = min(TK, n - t * TK);
    if (t + 1 < n_tiles) load_tile(t + 1, buf ^ 1);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const uint8_t* kt = kv_s + (size_t)buf * TK * pitch;
    // ---- partial scores of 16 keys over this warp's columns (every KS-th group of 32)
    {
      float s[MT][2][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[m][0][e] = s[m][1][e] = 0.f;
      const uint32_t k_addr = smem_addr(kt + (size_t)(kg * 16 + (lane & 7)) * pitch + (lane >> 3) * 16);
      const uint32_t q_addr = smem_addr(q_s + (size_t)(lane & 15) * pitch + (lane >> 4) * 16);
      if (kg * 16 < live) {
#pragma unroll 2
        for (int ks = kq; ks < a.W / 32; ks += KS) {
          uint32_t ka[4], kb[4];
          ldsm_x4(k_addr + ks * 64, ka);
          ldsm_x4(k_addr + 8 * pitch + ks * 64, kb);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            uint32_t qa[4], qb[4];
            ldsm_x4(q_addr + m * 16 * pitch + ks * 64, qa);
            ldsm_x4(q_addr + m * 16 * pitch + ks * 64 + 32, qb);
            mma_bf16(s[m][0], qa, ka[0], ka[1]);
            mma_bf16(s[m][1], qa, kb[0], kb[1]);
            mma_bf16(s[m][0], qb, ka[2], ka[3]);
            mma_bf16(s[m][1], qb, kb[2], kb[3]);
          }
        }
      }
      float* dst = sc + (size_t)kq * MR * SP + kg * 16 + 2 * c;
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int b = 0; b < 2; ++b) {
          *reinterpret_cast<float2*>(dst + (m * 16 + g) * SP + b * 8) = make_float2(s[m][b][0], s[m][b][1]);
          *reinterpret_cast<float2*>(dst + (m * 16 + g + 8) * SP + b * 8) = make_float2(s[m][b][2], s[m][b][3]);
        }
    }
    __syncthreads();
    // ---- running maximum and sum per head
#pragma unroll
    for (int hh = 0; hh < MT; ++hh) {
      const int h = warp + hh * DEC_WARPS;
      if (h >= gc) break;
      float v[TK / 32], mx = m_s[h];
      const float m_old = mx;
#pragma unroll
      for (int i = 0; i < TK / 32; ++i) {
        float x = 0.f;
#pragma unroll
        for (int k = 0; k < KS; ++k) x += sc[(k * MR + h) * SP + i * 32 + lane];
        v[i] = i * 32 + lane < live ? x * a.scale : -INFINITY;
        mx = fmaxf(mx, v[i]);
      }
      mx = warp_max(mx);
      float l = 0.f;
#pragma unroll
      for (int i = 0; i < TK / 32; ++i) {
        const float w = __expf(v[i] - mx);
        l += w;
        reinterpret_cast<__nv_bfloat16*>(p_s + h * PP)[i * 32 + lane] = f32_to_bf16(w);
      }
      l = warp_sum(l);
      if (lane == 0) {
        const float cr = __expf(m_old - mx);
        corr_s[h] = cr;
        l_s[h] = l_s[h] * cr + l;
        m_s[h] = mx;
      }
    }
    __syncthreads();
    // ---- weighted sum of the latents
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float c0 = corr_s[m * 16 + g], c1 = corr_s[m * 16 + g + 8];
#pragma unroll
      for (int j = 0; j < NB; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          o[m][j][e][0] *= c0; o[m][j][e][1] *= c0;
          o[m][j][e][2] *= c1; o[m][j][e][3] *= c1;
        }
    }
#pragma unroll
    for (int kk = 0; kk < TK / 16; ++kk) {
      if (kk * 16 >= live) break;
      uint32_t pa[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
        ldsm_x4(smem_addr(p_s + (size_t)(m * 16 + (lane & 15)) * PP + (kk * 16 + (lane >> 4) * 8) * 2), pa[m]);
      const uint32_t v_addr =
          smem_addr(kt + (size_t)(kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * pitch + (lane >> 4) * 16);
#pragma unroll
      for (int j = 0; j < NB; ++j) {
        const int blk = warp + DEC_WARPS * j;
        if (blk < n_blk) {
          uint32_t vf[4];
          ldsm_x4_t(v_addr + blk * 32, vf);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma_bf16(o[m][j][0], pa[m], vf[0], vf[1]);
            mma_bf16(o[m][j][1], pa[m], vf[2], vf[3]);
          }
        }
      }
    }
    __syncthreads();
  }
  float* part = a.partial + (((size_t)r * a.H + h0) * a.max_splits + sp) * a.rank_cols;
  const size_t head_stride = (size_t)a.max_splits * a.rank_cols;
  if (tid < gc) {
    float2* ml = reinterpret_cast<float2*>(a.partial + (size_t)a.R * a.H * head_stride);
    ml[((size_t)r * a.H + h0 + tid) * a.max_splits + sp] = make_float2(m_s[tid], l_s[tid]);
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < NB; ++j) {
      const int blk = warp + DEC_WARPS * j;
      if (blk >= n_blk) continue;
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int h = m * 16 + g + hf * 8;
        if (h >= gc) continue;
        float* dst = part + h * head_stride + blk * 16 + 2 * c;
        *reinterpret_cast<float2*>(dst) = make_float2(o[m][j][0][2 * hf], o[m][j][0][2 * hf + 1]);
        *reinterpret_cast<float2*>(dst + 8) = make_float2(o[m][j][1][2 * hf], o[m][j][1][2 * hf + 1]);
      }
    }
}

// grid (H, R, ceil(rank_cols / 128)): merge the spans (the eight warps take them in turn, a lane owns four columns), add the
// sink to the denominator, round to bf16
constexpr int RED_WARPS = 8;
__global__ void __launch_bounds__(RED_WARPS * 32) latent_reduce_kernel(const LatentDecArgs a) {
  extern __shared__ float wsm[];     // [max_splits]
  __shared__ float red[33];
  __shared__ float4 acc_s[RED_WARPS][32];
  pdl_wait();
  pdl_launch();
  const int h = blockIdx.x, r = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int ctx = a.ctx_len[r];
  const int start = (a.window > 0 && ctx > a.window) ? ctx - a.window : 0;
  const int ns = min((ctx - start + a.split_len - 1) / a.split_len, a.max_splits);
  const size_t row = ((size_t)r * a.H + h) * a.max_splits;
  const float2* ml = reinterpret_cast<const float2*>(a.partial + (size_t)a.R * a.H * a.max_splits * a.rank_cols) + row;
  const int d = blockIdx.z * 128 + lane * 4;
  const float* pb = a.partial + row * a.rank_cols + d;
  const bool mine = d < a.rank_cols;
  // the first spans' columns are requested before their weights are known
  constexpr int AHEAD = 4;
  float4 x[AHEAD];
#pragma unroll
  for (int u = 0; u < AHEAD; ++u) {
    const int s = warp + u * RED_WARPS;
    x[u] = mine && s < ns ? *reinterpret_cast<const float4*>(pb + (size_t)s * a.rank_cols) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  float m = a.sink != nullptr ? a.sink[h] : -INFINITY;
  const float sk = m;
  for (int s = threadIdx.x; s < ns; s += RED_WARPS * 32) m = fmaxf(m, ml[s].x);
  m = block_max(m, red);
  float den = 0.f;
  for (int s = threadIdx.x; s < ns; s += RED_WARPS * 32) {
    const float2 v = ml[s];
    const float w = __expf(v.x - m);
    wsm[s] = w;
    den += w * v.y;
  }
  den = block_sum(den, red);         // its barriers also publish wsm
  if (a.sink != nullptr) den += __expf(sk - m);
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int s0 = warp; s0 < ns; s0 += AHEAD * RED_WARPS) {
    if (s0 != warp) {
#pragma unroll
      for (int u = 0; u < AHEAD; ++u) {
        const int s = s0 + u * RED_WARPS;
        x[u] = mine && s < ns ? *reinterpret_cast<const float4*>(pb + (size_t)s * a.rank_cols) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
    }
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
      const int s = s0 + u * RED_WARPS;
      const float w = s < ns ? wsm[s] : 0.f;
      acc.x += w * x[u].x; acc.y += w * x[u].y; acc.z += w * x[u].z; acc.w += w * x[u].w;
    }
  }
  acc_s[warp][lane] = acc;
  __syncthreads();
  if (warp != 0 || !mine) return;
#pragma unroll
  for (int w = 1; w < RED_WARPS; ++w) {
    const float4 v = acc_s[w][lane];
    acc.x += v.x; acc.y += v.y; acc.z += v.z; acc.w += v.w;
  }
  const float inv = den > 0.f ? 1.f / den : 0.f;
  __align__(8) __nv_bfloat162 b[2] = {__floats2bfloat162_rn(acc.x * inv, acc.y * inv), __floats2bfloat162_rn(acc.z * inv, acc.w * inv)};
  *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(a.out) + ((size_t)r * a.H + h) * a.rank_cols + d) =
      *reinterpret_cast<const uint2*>(b);
}

// ---------------------------------------------------------------- fp32: one CTA per (row, head)
constexpr int EX_THREADS = 128, EX_COLS = 8;       // columns per thread: latents up to 1024 wide
__global__ void __launch_bounds__(EX_THREADS) latent_exact_kernel(const LatentDecArgs a) {
  extern __shared__ float q_s[];     // [W]
  __shared__ float s_s[EX_THREADS], red[33];
  __shared__ int row_s[EX_THREADS];
  pdl_wait();
  pdl_launch();
  const int r = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int ctx = a.ctx_len[r], start = (a.window > 0 && ctx > a.window) ? ctx - a.window : 0;
  const int* bt = a.block_table + (size_t)a.slot[r] * a.max_pages;
  const float* q = reinterpret_cast<const float*>(a.q) + ((size_t)r * a.H + h) * a.W;
  const float* cache = reinterpret_cast<const float*>(a.cache);
  for (int i = tid; i < a.W; i += EX_THREADS) q_s[i] = q[i];
  float acc[EX_COLS] = {}, m = -INFINITY, l = 0.f;
  for (int k0 = start; k0 < ctx; k0 += EX_THREADS) {
    const int n = min(EX_THREADS, ctx - k0);
    __syncthreads();
    if (tid < n) {
      const int p = k0 + tid, pi = p / a.page;
      row_s[tid] = bt[HE_INDEX_OK(pi, a.max_pages, HE_SITE_ATTN_DECODE_PAGE) ? pi : 0] * a.page + p % a.page;
    }
    __syncthreads();
    for (int k = warp; k < n; k += EX_THREADS / 32) {
      const float* kr = cache + (size_t)row_s[k] * a.W;
      float s = 0.f;
      for (int i = lane; i < a.W; i += 32) s += q_s[i] * kr[i];
      s = warp_sum(s);
      if (lane == 0) s_s[k] = s * a.scale;
    }
    __syncthreads();
    const float mine = tid < n ? s_s[tid] : -INFINITY;
    const float mn = fmaxf(m, block_max(mine, red)), corr = expf(m - mn), w = tid < n ? expf(mine - mn) : 0.f;
    s_s[tid] = w;
    l = l * corr + block_sum(w, red);              // its barriers also publish the weights
    m = mn;
#pragma unroll
    for (int j = 0; j < EX_COLS; ++j) {
      const int col = tid + j * EX_THREADS;
      if (col < a.rank_cols) {
        float v = acc[j] * corr;
        for (int k = 0; k < n; ++k) v += s_s[k] * cache[(size_t)row_s[k] * a.W + col];
        acc[j] = v;
      }
    }
  }
  if (a.sink != nullptr) {
    const float mn = fmaxf(m, a.sink[h]), corr = expf(m - mn);
    l = l * corr + expf(a.sink[h] - mn);
#pragma unroll
    for (int j = 0; j < EX_COLS; ++j) acc[j] *= corr;
  }
  float* out = reinterpret_cast<float*>(a.out) + ((size_t)r * a.H + h) * a.rank_cols;
#pragma unroll
  for (int j = 0; j < EX_COLS; ++j)
    if (tid + j * EX_THREADS < a.rank_cols) out[tid + j * EX_THREADS] = l > 0.f ? acc[j] / l : 0.f;
}

// ---------------------------------------------------------------- cache rows of long portions, side by side
// Segment s contributes the keys its rows can see, in segment order, padded with zero rows (latent_segs.cuh).
__global__ void __launch_bounds__(256) latent_gather_kernel(const LatentGatherArgs a) {
  pdl_wait();
  pdl_launch();
  const int lane = threadIdx.x & 31, row = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (row >= a.keys) return;
  uint4* dst = reinterpret_cast<uint4*>(a.out + (size_t)row * a.W);
  int k = row;
  for (int s = 0; s < a.n_seg; ++s) {
    const LatentSeg g = latent_seg(a.seg_start, a.pos, s, a.window, 0);
    if (k < g.keys) {
      const int p = g.lo + k, pi = p / a.page;
      const int* bt = a.block_table + (size_t)a.seg_slot[s] * a.max_pages;
      const int pg = bt[HE_INDEX_OK(pi, a.max_pages, HE_SITE_ATTN_DECODE_PAGE) ? pi : 0];
      const uint4* src = reinterpret_cast<const uint4*>(a.cache + ((size_t)pg * a.page + p % a.page) * a.W);
      for (int i = lane; i < a.W / 8; i += 32) dst[i] = src[i];
      return;
    }
    k -= latent_seg_rows(g);
    if (k < 0) break;                                    // padding of this segment
  }
  for (int i = lane; i < a.W / 8; i += 32) dst[i] = make_uint4(0u, 0u, 0u, 0u);
}

template <int MT, int NB, int TK>
int launch_decode(const LatentDecArgs& a, cudaStream_t stream) {
  const size_t smem = dec_smem<MT, TK>(a.W);
  if (smem > 227 * 1024) return -HE_ERR_BAD_ARG;
  cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<MT, NB, TK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  const dim3 grid(a.max_splits, (a.H + MT * 16 - 1) / (MT * 16), a.R);
  return (int)launch_pdl(latent_decode_kernel<MT, NB, TK>, grid, dim3(DEC_WARPS * 32), smem, stream, a);
}

// Tiles of 64 keys and 32 heads where they fit and the spans are whole tiles, else smaller ones.
template <int NB>
int pick_decode(const LatentDecArgs& a, cudaStream_t stream) {
  const bool big = a.split_len % 64 == 0;
  if (a.H > 16 && big && dec_smem<2, 64>(a.W) <= 227 * 1024) return launch_decode<2, NB, 64>(a, stream);
  if (a.H > 16 && dec_smem<2, 32>(a.W) <= 227 * 1024) return launch_decode<2, NB, 32>(a, stream);
  if (big && dec_smem<1, 64>(a.W) <= 227 * 1024) return launch_decode<1, NB, 64>(a, stream);
  return launch_decode<1, NB, 32>(a, stream);
}

}  // namespace

HE_API int he_latent_post(const LatentPostArgs* args, cudaStream_t stream) {
  const LatentPostArgs& a = *args;
  if (a.T <= 0) return 0;
  if (a.rot_dim % 2 != 0 || a.dn % 2 != 0 || a.q_cols % 2 != 0 || a.q_cols < a.dn + a.rot_dim || a.rank > a.rank_cols ||
      a.W < a.rank_cols + a.rot_dim || (a.W - a.rank_cols) % 2 != 0)
    return -HE_ERR_BAD_ARG;
  if (a.q_out == a.q && (a.q_dtype == 0) != (a.out_f32 != 0)) return -HE_ERR_BAD_ARG;
  const dim3 grid(a.T, 1 + ((a.q_out != nullptr || a.q_lat != nullptr) ? (a.H + POST_HEADS - 1) / POST_HEADS : 0));
  const size_t smem = (size_t)(a.rot_dim / 2) * sizeof(float2);
  return (int)(a.out_f32 ? launch_pdl(latent_post_kernel<float>, grid, dim3(256), smem, stream, a)
                         : launch_pdl(latent_post_kernel<__nv_bfloat16>, grid, dim3(256), smem, stream, a));
}
HE_API int he_latent_post_args_size() { return (int)sizeof(LatentPostArgs); }

static int check_decode(const LatentDecArgs& a) {
  if (a.H <= 0 || a.W % 32 != 0 || a.rank_cols % 16 != 0 || a.rank_cols <= 0 || a.rank_cols > a.W || a.rank_cols > 1024)
    return -HE_ERR_BAD_ARG;
  return 0;
}

// Scratch: R * H * max_splits * (rank_cols + 2) floats in `partial`.
HE_API int he_latent_decode(const LatentDecArgs* args, cudaStream_t stream) {
  const LatentDecArgs& a = *args;
  if (a.R <= 0) return 0;
  if (check_decode(a) != 0 || a.split_len <= 0 || a.max_splits <= 0 || a.R > 65535) return -HE_ERR_BAD_ARG;
  const int nb = (a.rank_cols / 16 + DEC_WARPS - 1) / DEC_WARPS;
  int rc;
  if (nb <= 1) rc = pick_decode<1>(a, stream);
  else if (nb <= 2) rc = pick_decode<2>(a, stream);
  else rc = launch_decode<1, 4, 32>(a, stream);
  if (rc != 0) return rc;
  return (int)launch_pdl(latent_reduce_kernel, dim3(a.H, a.R, (a.rank_cols + 127) / 128), dim3(RED_WARPS * 32),
                         (size_t)a.max_splits * sizeof(float), stream, a);
}
HE_API int he_latent_dec_args_size() { return (int)sizeof(LatentDecArgs); }

HE_API int he_latent_exact(const LatentDecArgs* args, cudaStream_t stream) {
  const LatentDecArgs& a = *args;
  if (a.R <= 0) return 0;
  if (check_decode(a) != 0 || a.H > 65535) return -HE_ERR_BAD_ARG;
  return (int)launch_pdl(latent_exact_kernel, dim3(a.R, a.H), dim3(EX_THREADS), (size_t)a.W * sizeof(float), stream, a);
}

HE_API int he_latent_gather(const LatentGatherArgs* args, cudaStream_t stream) {
  const LatentGatherArgs& a = *args;
  if (a.keys <= 0 || a.n_seg <= 0) return 0;
  if (a.W % 8 != 0) return -HE_ERR_BAD_ARG;
  return (int)launch_pdl(latent_gather_kernel, dim3((a.keys + 7) / 8), dim3(256), 0, stream, a);
}
HE_API int he_latent_gather_args_size() { return (int)sizeof(LatentGatherArgs); }
