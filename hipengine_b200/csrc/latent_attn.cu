// Latent attention over a paged latent cache: cache write with rotation, single-token / short-portion attention, gather for
// long portions, and the fp32 forms.
//
// A token's cache row is [latent (rank columns, zero-padded to a multiple of 16) | rotated key part | zeros] of W columns
// (a multiple of 32); the plane of a layer run is [n_pages][page][W].  A head's key is a linear map of the latent plus the
// rotated part, its value another linear map of the latent.  Decode never builds them: the key map is moved onto the query
// (q_lat = [W_k^T q | rotated q], W columns) and the value map behind the weighted sum, so all heads of a request attend to
// one W-wide row per token, which is read once and serves as key and value.
#include "latent_segs.cuh"
#include "sm100.cuh"

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
  float* partial;            // more than one cluster per row: [R][H][clusters][rank_cols], then (maximum, sum) pairs
  void* out;                 // [R][H][rank_cols]
  const float* sink;         // [H] or null: one more term in the softmax denominator
  int R, H, W, rank_cols, page, max_pages, window;
  int spans, cluster, tile;  // CTAs per row and head chunk, how many of them merge on chip, keys per tile (32 or 64)
  float scale;
  int* status;               // a bounded wait that gave up records its code here (split form)
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
  // the latent row and the page are requested before anything waits for them
  constexpr int PER = 4;                                   // latents up to 1024 wide
  const size_t in0 = (size_t)t * a.down_stride;
  float lat[PER] = {};
  int pg = 0;
  const int pi = p / a.page;
  const bool page_ok = HE_INDEX_OK(pi, a.max_pages, HE_SITE_KV_WRITE_PAGE);
  if (blockIdx.y == 0) {
#pragma unroll
    for (int k = 0; k < PER; ++k)
      if (threadIdx.x + 256 * k < a.rank) lat[k] = load_in(a.down, a.down_dtype, in0 + threadIdx.x + 256 * k);
    if (page_ok) pg = a.block_table[(size_t)a.slot[t] * a.max_pages + pi];
  }
  for (int i = threadIdx.x; i < half; i += 256) {
    // the angle is reduced to one turn in double, so late positions keep full fp32 accuracy
    const double two_pi = 6.283185307179586476925286766559;
    const double ang = (double)p * a.freq[i];
    float sn, c;
    sincosf((float)(ang - two_pi * rint(ang / two_pi)), &sn, &c);
    cs[i] = make_float2(c * a.amp, sn * a.amp);
  }
  if (blockIdx.y == 0) {
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < PER; ++k) ss += lat[k] * lat[k];
    const float inv = rsqrtf(block_sum(ss, red) / (float)a.rank + a.eps);     // its barriers also publish cs
    if (!page_ok) return;
    OutT* row = reinterpret_cast<OutT*>(a.cache) + ((size_t)pg * a.page + p % a.page) * a.W;
#pragma unroll
    for (int k = 0; k < PER; ++k) {
      const int i = threadIdx.x + 256 * k;
      if (i < a.rank_cols) row[i] = from_f32<OutT>(i < a.rank ? lat[k] * inv * a.norm_w[i] : 0.f);
    }
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

__device__ __forceinline__ uint32_t cluster_rank() {
  uint32_t v;
  asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(v));
  return v;
}
__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }
// shared-memory address `addr` of this CTA as seen in CTA `rank` of the cluster
__device__ __forceinline__ uint32_t map_peer(uint32_t addr, uint32_t rank) {
  uint32_t v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(v) : "r"(addr), "r"(rank));
  return v;
}
__device__ __forceinline__ float ld_peer(uint32_t addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
  return v;
}
__device__ __forceinline__ float4 ld_peer4(uint32_t addr) {
  float4 v;
  asm volatile("ld.shared::cluster.v4.f32 {%0,%1,%2,%3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(addr) : "memory");
  return v;
}
__device__ __forceinline__ void store_bf16x4(__nv_bfloat16* dst, float4 v, float f) {
  __align__(8) __nv_bfloat162 b[2] = {__floats2bfloat162_rn(v.x * f, v.y * f), __floats2bfloat162_rn(v.z * f, v.w * f)};
  *reinterpret_cast<uint2*>(dst) = *reinterpret_cast<const uint2*>(b);
}

__device__ __forceinline__ void bulk_row(void* smem_dst, const void* gsrc, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               :
               : "r"(smem_addr(smem_dst)), "l"(gsrc), "r"(bytes), "r"(smem_addr(bar))
               : "memory");
}

// One CTA per (key span, chunk of up to 16 MT heads, row).  A row's visible keys are cut into `spans` equal spans of whole
// tiles, from its own context, so a launch sized for longer contexts stays balanced.  Tiles of TK latent rows are double-buffered: a lane
// copies one whole row in bulk (rows padded by 16 bytes: conflict-free ldmatrix).  Per tile: partial scores (the warps split 16-key groups and the columns, so
// the queries are read from shared memory TK / 16 times and not once per warp), running maximum and sum per head, then the
// weighted sum (a warp owns every sixteenth block of 16 latent columns, up to NB blocks).
// Merge: the CTAs of a cluster leave their sums in shared memory and each adds up one share of the columns over all of them
// (distributed shared memory).  With one cluster per row that is the result; with several, latent_reduce_kernel merges theirs.
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
  if (gc <= 0) return;                                    // the whole cluster: it shares the head chunk
  const int ctx = a.ctx_len[r];
  const int start = (a.window > 0 && ctx > a.window) ? ctx - a.window : 0;
  const int tiles = (ctx - start + TK - 1) / TK, span = (tiles + a.spans - 1) / a.spans * TK;
  const int k0 = start + sp * span;
  const int n = max(0, min(span, ctx - k0)), n_tiles = (n + TK - 1) / TK;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c = lane & 3;
  const int* bt = a.block_table + (size_t)a.slot[r] * a.max_pages;
  const __nv_bfloat16* cache = reinterpret_cast<const __nv_bfloat16*>(a.cache);

  __shared__ uint64_t full_s[2];
  __shared__ int abort_s;
  if (tid == 0) {
    sm100::mbar_init(&full_s[0], 1);
    sm100::mbar_init(&full_s[1], 1);
    abort_s = 0;
    sm100::mbar_fence_init();
  }
  __syncthreads();
  const int page_log2 = 31 - __clz(a.page);               // pages are powers of two (checked by the launcher)
  const auto load_tile = [&](int t, int buf) {
    if (tid >= TK) return;
    const int pos = k0 + min(t * TK + tid, n - 1);        // rows past the span repeat its last key; their weight is zero
    const int pi = pos >> page_log2;
    const int pg = bt[HE_INDEX_OK(pi, a.max_pages, HE_SITE_ATTN_DECODE_PAGE) ? pi : 0];
    if (tid == 0) sm100::mbar_expect_tx(&full_s[buf], (uint32_t)TK * a.W * 2);
    bulk_row(kv_s + ((size_t)buf * TK + tid) * pitch, cache + (((size_t)pg << page_log2) + (pos & (a.page - 1))) * a.W, a.W * 2,
             &full_s[buf]);
  };
  if (n > 0) load_tile(0, 0);
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
    const bool landed = sm100::mbar_wait(&full_s[buf], (t >> 1) & 1, &abort_s, a.status, 501);
    if (__syncthreads_or(!landed)) {
      // give up: no copy may still be in flight when the buffers are written below
      if (t + 1 < n_tiles)
        for (uint32_t w = 0; w < sm100::WAIT_LIMIT && !sm100::mbar_try_wait(&full_s[buf ^ 1], ((t + 1) >> 1) & 1); ++w) {}
      __syncthreads();
      break;
    }
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
    // ---- running maximum and sum per head: half a warp per head
    for (int h = warp * 2 + (lane >> 4); h < MR; h += DEC_WARPS * 2) {
      const int k = (lane & 15) * (TK / 16);              // this lane's neighbouring keys
      float v[TK / 16], mx = m_s[h];
      const float m_old = mx;
#pragma unroll
      for (int i = 0; i < TK / 16; ++i) v[i] = 0.f;
#pragma unroll
      for (int q = 0; q < KS; ++q) {
        const float* src = sc + (q * MR + h) * SP + k;
        if constexpr (TK == 64) {
          const float4 x = *reinterpret_cast<const float4*>(src);
          v[0] += x.x; v[1] += x.y; v[2] += x.z; v[3] += x.w;
        } else {
          const float2 x = *reinterpret_cast<const float2*>(src);
          v[0] += x.x; v[1] += x.y;
        }
      }
#pragma unroll
      for (int i = 0; i < TK / 16; ++i) {
        v[i] = k + i < live ? v[i] * a.scale : -INFINITY;
        mx = fmaxf(mx, v[i]);
      }
#pragma unroll
      for (int d = 8; d > 0; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
      float l = 0.f;
#pragma unroll
      for (int i = 0; i < TK / 16; ++i) {
        v[i] = __expf(v[i] - mx);
        l += v[i];
      }
      uint32_t* dst = reinterpret_cast<uint32_t*>(p_s + h * PP) + k / 2;
#pragma unroll
      for (int i = 0; i < TK / 32; ++i) {
        __nv_bfloat162 b = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
        dst[i] = *reinterpret_cast<uint32_t*>(&b);
      }
#pragma unroll
      for (int d = 8; d > 0; d >>= 1) l += __shfl_xor_sync(0xffffffffu, l, d);
      if ((lane & 15) == 0) {
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
  // ---- merge.  This CTA's sums go where its tiles were (every warp is past its last tile).
  __syncthreads();
  float* o_s = reinterpret_cast<float*>(kv_s);            // [MR][rank_cols]
  float* w_s = sc;                                        // [cluster or clusters][MR] weights, then [MR] sums
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < NB; ++j) {
      const int blk = warp + DEC_WARPS * j;
      if (blk >= n_blk) continue;
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        float* dst = o_s + (size_t)(m * 16 + g + hf * 8) * a.rank_cols + blk * 16 + 2 * c;
        *reinterpret_cast<float2*>(dst) = make_float2(o[m][j][0][2 * hf], o[m][j][0][2 * hf + 1]);
        *reinterpret_cast<float2*>(dst + 8) = make_float2(o[m][j][1][2 * hf], o[m][j][1][2 * hf + 1]);
      }
    }
  const int C = a.cluster, cl = sp / C, n_cl = a.spans / C;
  const uint32_t me = C > 1 ? cluster_rank() : 0u;
  if (C > 1) {
    cluster_arrive();
    cluster_wait();
  } else {
    __syncthreads();
  }
  const int share = ((a.rank_cols + C - 1) / C + 3) / 4 * 4, d0 = (int)me * share, d1 = min(a.rank_cols, d0 + share);
  const int quads = max(0, d1 - d0) / 4;
  __shared__ float M_s[MR], L_s[MR];
  float* pl_s = w_s + 128 * MR;                           // peers' sums, then nothing
  if (tid < C * MR) {
    const int p = tid / MR, h = tid % MR;
    w_s[tid] = ld_peer(map_peer(smem_addr(m_s + h), p));
    pl_s[tid] = ld_peer(map_peer(smem_addr(l_s + h), p));
  }
  __syncthreads();
  if (tid < gc) {
    float M = -INFINITY, L = 0.f;
    for (int p = 0; p < C; ++p) M = fmaxf(M, w_s[p * MR + tid]);
    for (int p = 0; p < C; ++p) {
      const float mp = w_s[p * MR + tid], w = mp == -INFINITY ? 0.f : __expf(mp - M);
      w_s[p * MR + tid] = w;
      L += w * pl_s[p * MR + tid];
    }
    M_s[tid] = M;
    L_s[tid] = L;
  }
  __syncthreads();
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + ((size_t)r * a.H + h0) * a.rank_cols + d0;
  float* part = a.partial + (((size_t)r * a.H + h0) * n_cl + cl) * a.rank_cols + d0;
  const size_t head_stride = (size_t)n_cl * a.rank_cols;
  for (int e = tid; e < gc * quads; e += DEC_WARPS * 32) {
    const int h = e / quads, d = (e % quads) * 4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    const uint32_t src = smem_addr(o_s + (size_t)h * a.rank_cols + d0 + d);
    float4 x[8];
#pragma unroll
    for (int p = 0; p < 8; ++p) x[p] = p < C ? ld_peer4(map_peer(src, p)) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int p = 0; p < 8; ++p) {
      const float w = p < C ? w_s[p * MR + h] : 0.f;      // an idle CTA's sums are zeros
      v.x += w * x[p].x; v.y += w * x[p].y; v.z += w * x[p].z; v.w += w * x[p].w;
    }
    if (n_cl == 1) {
      float f = 1.f, L = L_s[h];
      if (a.sink != nullptr) {
        const float sk = a.sink[h0 + h], mn = fmaxf(M_s[h], sk);
        f = __expf(M_s[h] - mn);
        L = L * f + __expf(sk - mn);
      }
      store_bf16x4(out + (size_t)h * a.rank_cols + d, v, L > 0.f ? f / L : 0.f);
    } else {
      *reinterpret_cast<float4*>(part + h * head_stride + d) = v;
    }
  }
  __syncwarp();
  if (C > 1) cluster_arrive();                            // done with the peers' shared memory
  if (n_cl > 1 && me == 0 && tid < gc) {
    float2* ml = reinterpret_cast<float2*>(a.partial + (size_t)a.R * a.H * head_stride);
    ml[((size_t)r * a.H + h0 + tid) * n_cl + cl] = make_float2(M_s[tid], L_s[tid]);
  }
  if (C > 1) cluster_wait();
}

// grid (H, R, ceil(rank_cols / 128)): merge the clusters' sums (the eight warps take them in turn, a lane owns four columns), add the
// sink to the denominator, round to bf16
constexpr int RED_WARPS = 8, MAX_CLUSTERS = 128;
__global__ void __launch_bounds__(RED_WARPS * 32) latent_reduce_kernel(const LatentDecArgs a) {
  __shared__ float red[33], wsm[MAX_CLUSTERS];
  __shared__ float4 acc_s[RED_WARPS][32];
  pdl_wait();
  pdl_launch();
  const int h = blockIdx.x, r = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int ns = a.spans / a.cluster;
  const size_t row = ((size_t)r * a.H + h) * ns;
  const float2* ml = reinterpret_cast<const float2*>(a.partial + (size_t)a.R * a.H * ns * a.rank_cols) + row;
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
    const float w = v.x == -INFINITY ? 0.f : __expf(v.x - m);      // an idle cluster
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
  store_bf16x4(reinterpret_cast<__nv_bfloat16*>(a.out) + ((size_t)r * a.H + h) * a.rank_cols + d, acc,
               den > 0.f ? 1.f / den : 0.f);
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
  if (smem > 226 * 1024) return -HE_ERR_BAD_ARG;          // a few hundred bytes are static
  cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<MT, NB, TK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(a.spans, (a.H + MT * 16 - 1) / (MT * 16), a.R);
  cfg.blockDim = dim3(DEC_WARPS * 32);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = a.cluster;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = pdl_enabled() ? 2 : 1;
  return (int)cudaLaunchKernelEx(&cfg, latent_decode_kernel<MT, NB, TK>, a);
}

// Tiles of 64 keys and 32 heads where they fit and the spans are whole tiles, else smaller ones.
template <int NB>
int pick_decode(const LatentDecArgs& a, cudaStream_t stream) {
  const bool big = a.tile == 64;
  if (a.H > 16 && big && dec_smem<2, 64>(a.W) <= 226 * 1024) return launch_decode<2, NB, 64>(a, stream);
  if (a.H > 16 && dec_smem<2, 32>(a.W) <= 226 * 1024) return launch_decode<2, NB, 32>(a, stream);
  if (big && dec_smem<1, 64>(a.W) <= 226 * 1024) return launch_decode<1, NB, 64>(a, stream);
  return launch_decode<1, NB, 32>(a, stream);
}

}  // namespace

HE_API int he_latent_post(const LatentPostArgs* args, cudaStream_t stream) {
  const LatentPostArgs& a = *args;
  if (a.T <= 0) return 0;
  if (a.rank_cols > 1024 || a.rot_dim % 2 != 0 || a.dn % 2 != 0 || a.q_cols % 2 != 0 || a.q_cols < a.dn + a.rot_dim || a.rank > a.rank_cols ||
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

// With more than one cluster per row (spans > cluster): `partial` holds R * H * (spans / cluster) * (rank_cols + 2) floats.
HE_API int he_latent_decode(const LatentDecArgs* args, cudaStream_t stream) {
  const LatentDecArgs& a = *args;
  if (a.R <= 0) return 0;
  if (check_decode(a) != 0 || a.cluster < 1 || a.cluster > 8 || a.spans < a.cluster || a.spans % a.cluster != 0 ||
      a.spans / a.cluster > MAX_CLUSTERS || (a.tile != 32 && a.tile != 64) || a.R > 65535)
    return -HE_ERR_BAD_ARG;
  if ((a.spans > a.cluster && a.partial == nullptr) || a.page <= 0 || (a.page & (a.page - 1)) != 0) return -HE_ERR_BAD_ARG;
  const int nb = (a.rank_cols / 16 + DEC_WARPS - 1) / DEC_WARPS;
  const int rc = nb <= 1 ? pick_decode<1>(a, stream) : nb <= 2 ? pick_decode<2>(a, stream) : launch_decode<1, 4, 32>(a, stream);
  if (rc != 0 || a.spans == a.cluster) return rc;
  // in plain stream order: started early beside CTAs that fill their SMs, this small grid costs a decode step up to 40 us a layer
  latent_reduce_kernel<<<dim3(a.H, a.R, (a.rank_cols + 127) / 128), dim3(RED_WARPS * 32), 0, stream>>>(a);
  HE_LAUNCH_CHECK();
  return 0;
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
