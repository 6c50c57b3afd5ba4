// Linear attention (retention, gated delta rule) over prompt portions, 64 tokens at a time on tensor cores.
//
// With c_t the product of the decays from the chunk's start up to token t, S the state before the chunk, and for the delta rule
// A_tj = beta_t (c_t / c_j)(k_t . k_j) below the diagonal:
//   R = beta (V - c K S);  D = (I + A)^-1 R            retention: D = V
//   O = c Q S + P D,  P_tj = (c_t / c_j)(q_t . k_j) up to the diagonal
//   S <- c_64 S + K^T E,  E_j = (c_64 / c_j) D_j
// What does not depend on S is done for all chunks at once (prepare): rows from projections (rotation, or convolution, silu and
// unit length) and the 64 x 64 matrices P and (I + A)^-1.  The scan then walks the chunks of a segment: a CTA owns 32 columns of
// a head's state, kept in fp32 registers, and prefetches what the next phases need.
//
// Operands are fp32 numbers as pairs of bf16 (value and remainder, 2^-17 of relative error); a product is three mma.sync with fp32
// accumulation.  Decays are ratios of at most one, from sums of logarithms (or a table of powers).
#include "linear_attn.cuh"

using namespace he;

namespace {

constexpr int CK = 64;             // tokens per chunk
constexpr int NTHR = 256;
constexpr int NV = 32;             // state columns per CTA of the scan
constexpr int LDM = CK + 8;        // row pitch of 64-column tiles

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const __nv_bfloat16* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], const __nv_bfloat16* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void split(float x, __nv_bfloat16& hi, __nv_bfloat16& lo) {
  hi = f32_to_bf16(x);
  lo = f32_to_bf16(x - bf16_to_f32(hi));
}
__device__ __forceinline__ void cp16(void* dst, const void* src, bool live) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  const int n = live ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void cp4(void* dst, const void* src, bool live) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  const int n = live ? 4 : 0;
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(d), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// lane's place in the 8 x 8 blocks of a 16 x 16 operand tile stored with `ld` columns:
//   rows of A, and columns of a transposed A;   two neighbouring 8-column blocks of B stored as [column][k]
__device__ __forceinline__ int a_off(int lane, int ld) { return (lane & 15) * ld + (lane >> 4) * 8; }
__device__ __forceinline__ int at_off(int lane, int ld) { return ((lane & 7) + ((lane >> 4) & 1) * 8) * ld + ((lane >> 3) & 1) * 8; }
__device__ __forceinline__ int b_off(int lane, int ld) { return ((lane & 7) + ((lane >> 4) & 1) * 8) * ld + ((lane >> 3) & 1) * 8; }

// segment and chunk inside it of chunk `c` of the batch; false: there is no such chunk
__device__ __forceinline__ bool find_chunk(const LinearArgs& a, int c, int& seg, int& first) {
  for (seg = 0; seg < a.n_seg; ++seg) {
    const int n = (a.seg_start[seg + 1] - a.seg_start[seg] + CK - 1) / CK;
    if (c < n) {
      first = a.seg_start[seg] + c * CK;
      return true;
    }
    c -= n;
  }
  return false;
}

// ---------------------------------------------------------------- prepare
template <int DK>
struct PrepSmem {
  static constexpr int LD = DK + 8;
  __nv_bfloat16 q[2][CK * LD], k[2][CK * LD];      // value, remainder
  union {
    float tile[(CK + 15) * DK];                    // rows of a projection, those the convolution needs ahead of them first
    float A[CK][CK + 4];
  };
  float b[CK], beta[CK];
};

// dst[past + 64][DK] <- columns [col, col + width) of tokens t0 - past .. t0 + 63 (zero behind n tokens and behind width; ahead of
// the segment from the ring)
template <int DK>
__device__ __forceinline__ void stage_tile(const LinearArgs& a, float* dst, int t0, int n, int s0, int slot, int past, int col, int width) {
  const bool vec = (col & 7) == 0 && (width & 7) == 0 && (a.stride & 7) == 0;
  const int p0 = a.pos[s0];
  for (int i = threadIdx.x; i < (past + CK) * (DK / 8); i += NTHR) {
    const int r = i / (DK / 8), d = i % (DK / 8) * 8, t = t0 - past + r;
    float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (r < past + n && d < width) {
      if (t >= s0) {
        const size_t o = (size_t)t * a.stride + col + d;
        if (vec && a.row_dtype == 1) {
          const uint4 u = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(a.rows) + o);
          const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float2 f2 = __bfloat1622float2(h2[e]);
            v[2 * e] = f2.x;
            v[2 * e + 1] = f2.y;
          }
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e)
            if (d + e < width) v[e] = la_row(a, o + e);
        }
      } else if (p0 - (s0 - t) >= 0) {
        const float* src = a.ring + ((size_t)slot * a.taps + (p0 - (s0 - t)) % a.taps) * a.C + col + d;
#pragma unroll
        for (int e = 0; e < 8; ++e)
          if (d + e < width) v[e] = src[e];
      }
    }
    *reinterpret_cast<float4*>(dst + r * DK + d) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(dst + r * DK + d + 4) = make_float4(v[4], v[5], v[6], v[7]);
  }
}

__device__ __forceinline__ float silu_fast(float x) { return __fdividef(x, 1.f + __expf(fminf(-x, 80.f))); }

// Convolution and silu of eight tokens (from row r0 of the tile on) for NC columns at d: each(token, values).  TAPS 0: any number
template <int DK, int TAPS, typename Each>
__device__ __forceinline__ void conv_tokens(const LinearArgs& a, const float* tile, int r0, int d, int col, int width, Each each) {
  constexpr int NC = DK / 32;
  const int taps = TAPS > 0 ? TAPS : a.taps;
  constexpr int WN = TAPS > 0 ? TAPS : 1;
  float w[WN][NC], x[WN][NC];
  const auto weight = [&](int j, int e) { return d + e < width ? a.cw[(size_t)j * a.C + col + d + e] : 0.f; };
  if constexpr (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
      for (int e = 0; e < NC; ++e) {
        w[j][e] = weight(j, e);
        x[j][e] = j > 0 ? tile[(r0 + j - 1) * DK + d + e] : 0.f;
      }
  }
#pragma unroll
  for (int r = 0; r < CK / 8; ++r) {
    float v[NC];
    if constexpr (TAPS > 0) {
#pragma unroll
      for (int e = 0; e < NC; ++e) {
#pragma unroll
        for (int j = 0; j + 1 < TAPS; ++j) x[j][e] = x[j + 1][e];
        x[TAPS - 1][e] = tile[(r0 + r + TAPS - 1) * DK + d + e];
        v[e] = 0.f;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) v[e] += w[j][e] * x[j][e];
        v[e] = silu_fast(v[e]);
      }
    } else {
#pragma unroll
      for (int e = 0; e < NC; ++e) {
        v[e] = 0.f;
        for (int j = 0; j < taps; ++j) v[e] += weight(j, e) * tile[(r0 + r + j) * DK + d + e];
        v[e] = silu_fast(v[e]);
      }
    }
    each(r0 + r, v);
  }
}
template <int DK, typename Each>
__device__ __forceinline__ void conv_dispatch(const LinearArgs& a, const float* tile, int r0, int d, int col, int width, Each each) {
  if (a.taps == 4) conv_tokens<DK, 4>(a, tile, r0, d, col, width, each);
  else if (a.taps == 3) conv_tokens<DK, 3>(a, tile, r0, d, col, width, each);
  else if (a.taps == 2) conv_tokens<DK, 2>(a, tile, r0, d, col, width, each);
  else conv_tokens<DK, 0>(a, tile, r0, d, col, width, each);
}

// grid (chunks, H)
template <int DK, bool DELTA>
__global__ void __launch_bounds__(NTHR, 2) linear_chunk_prepare_kernel(const __grid_constant__ LinearArgs a) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  PrepSmem<DK>& sm = *reinterpret_cast<PrepSmem<DK>*>(smem_raw);
  constexpr int LD = PrepSmem<DK>::LD, NC = DK / 32;
  pdl_wait();
  pdl_launch();
  const int chunk = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  int seg, t0;
  if (!find_chunk(a, chunk, seg, t0)) return;
  const int s0 = a.seg_start[seg], n = min(CK, a.seg_start[seg + 1] - t0), slot = a.seg_slot[seg];
  if (!HE_INDEX_OK(slot, a.n_slots, HE_SITE_STATE_SLOT)) return;
  const int grp = a.H / a.G, kh = h / grp;
  const bool own = h % grp == 0;                   // writes the query and key rows its group shares
  const size_t qk_plane = (size_t)a.T * a.G * DK;

  if constexpr (DELTA) {
    const int past = a.taps - 1, r0 = warp * (CK / 8), d = lane * NC;
#pragma unroll
    for (int which = 0; which < 2; ++which) {
      const int col = (which ? a.ck : 0) + kh * a.dim;
      if (which) __syncthreads();
      stage_tile<DK>(a, sm.tile, t0, n, s0, slot, past, col, a.dim);
      __syncthreads();
      const float scale = which ? a.kscale : a.qscale;
      __nv_bfloat16* p0 = which ? sm.k[0] : sm.q[0];
      __nv_bfloat16* p1 = which ? sm.k[1] : sm.q[1];
      conv_dispatch<DK>(a, sm.tile, r0, d, col, a.dim, [&](int r, float (&v)[NC]) {
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < NC; ++e) ss += v[e] * v[e];
        const float inv = r < n ? scale * rsqrtf(warp_sum(ss) + 1e-6f) : 0.f;
        __align__(8) __nv_bfloat16 hi[NC], lo[NC];
#pragma unroll
        for (int e = 0; e < NC; ++e) split(v[e] * inv, hi[e], lo[e]);
        __nv_bfloat16* g0 = a.qk + (size_t)(2 * which) * qk_plane + ((size_t)(t0 + r) * a.G + kh) * DK + d;
        if constexpr (NC == 4) {
          const uint2 wh = *reinterpret_cast<const uint2*>(hi), wl = *reinterpret_cast<const uint2*>(lo);
          *reinterpret_cast<uint2*>(p0 + r * LD + d) = wh;
          *reinterpret_cast<uint2*>(p1 + r * LD + d) = wl;
          if (own && r < n) {
            *reinterpret_cast<uint2*>(g0) = wh;
            *reinterpret_cast<uint2*>(g0 + qk_plane) = wl;
          }
        } else {
          const uint32_t wh = *reinterpret_cast<const uint32_t*>(hi), wl = *reinterpret_cast<const uint32_t*>(lo);
          *reinterpret_cast<uint32_t*>(p0 + r * LD + d) = wh;
          *reinterpret_cast<uint32_t*>(p1 + r * LD + d) = wl;
          if (own && r < n) {
            *reinterpret_cast<uint32_t*>(g0) = wh;
            *reinterpret_cast<uint32_t*>(g0 + qk_plane) = wl;
          }
        }
      });
    }
    for (int v0 = 0; v0 < a.vcols; v0 += DK) {
      const int col = a.cv + h * a.vdim + v0, width = max(0, min(DK, a.vdim - v0));
      __syncthreads();
      stage_tile<DK>(a, sm.tile, t0, n, s0, slot, past, col, width);
      __syncthreads();
      conv_dispatch<DK>(a, sm.tile, r0, d, col, width, [&](int r, float (&v)[NC]) {
        if (r >= n || v0 + d >= a.vcols) return;               // silu(0) = 0 in padded columns
        __align__(8) __nv_bfloat16 o[NC];
#pragma unroll
        for (int e = 0; e < NC; ++e) o[e] = f32_to_bf16(v[e]);
        __nv_bfloat16* dst = a.vb + ((size_t)(t0 + r) * a.H + h) * a.vcols + v0 + d;
        if constexpr (NC == 4) *reinterpret_cast<uint2*>(dst) = *reinterpret_cast<const uint2*>(o);
        else *reinterpret_cast<uint32_t*>(dst) = *reinterpret_cast<const uint32_t*>(o);
      });
    }
    __syncthreads();
  } else {
    // rows as they are into the planes (bf16 rows have no remainder), values on their way out; then a warp turns the queries and
    // keys of a token in place, a lane has pairs (i, i + half) of both
    const bool plain = a.row_dtype == 1 && ((a.stride | a.ck | a.cv | a.dim | a.vdim) & 7) == 0;
    const __nv_bfloat16* rows = reinterpret_cast<const __nv_bfloat16*>(a.rows);
    for (int i = tid; i < 2 * CK * (DK / 8); i += NTHR) {
      const int which = i / (CK * (DK / 8)), r = i / (DK / 8) % CK, dd = i % (DK / 8) * 8;
      const size_t o = (size_t)(t0 + r) * a.stride + (which ? a.ck : 0) + kh * a.dim + dd;
      __align__(16) __nv_bfloat16 hi[8], lo[8];
      uint4 wh = make_uint4(0u, 0u, 0u, 0u), wl = wh;
      if (r < n && dd < a.dim) {
        if (plain) {
          wh = *reinterpret_cast<const uint4*>(rows + o);
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e) split(dd + e < a.dim ? la_row(a, o + e) : 0.f, hi[e], lo[e]);
          wh = *reinterpret_cast<const uint4*>(hi);
          wl = *reinterpret_cast<const uint4*>(lo);
        }
      }
      *reinterpret_cast<uint4*>((which ? sm.k[0] : sm.q[0]) + r * LD + dd) = wh;
      *reinterpret_cast<uint4*>((which ? sm.k[1] : sm.q[1]) + r * LD + dd) = wl;
    }
    for (int i = tid; i < n * (a.vcols / 8); i += NTHR) {
      const int r = i / (a.vcols / 8), dd = i % (a.vcols / 8) * 8;
      const size_t o = (size_t)(t0 + r) * a.stride + a.cv + h * a.vdim + dd;
      uint4 w;
      if (plain) {
        w = *reinterpret_cast<const uint4*>(rows + o);
      } else {
        __align__(16) __nv_bfloat16 v[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = f32_to_bf16(dd + e < a.vdim ? la_row(a, o + e) : 0.f);
        w = *reinterpret_cast<const uint4*>(v);
      }
      *reinterpret_cast<uint4*>(a.vb + ((size_t)(t0 + r) * a.H + h) * a.vcols + dd) = w;
    }
    __syncthreads();
    const int half = a.rot_dims >> 1;
    for (int r = warp; r < n; r += NTHR / 32) {
      const int p = a.pos[t0 + r];
      const auto get = [&](const __nv_bfloat16 (&x)[2][CK * LD], int dd) { return bf16_to_f32(x[0][r * LD + dd]) + bf16_to_f32(x[1][r * LD + dd]); };
      for (int i = lane; i < half; i += 32) {
        float c, s;
        la_angle(a.freq[i], p, c, s);
        const float qu = get(sm.q, i), qv = get(sm.q, half + i), ku = get(sm.k, i) * a.kscale, kv = get(sm.k, half + i) * a.kscale;
        split(qu * c - qv * s, sm.q[0][r * LD + i], sm.q[1][r * LD + i]);
        split(qv * c + qu * s, sm.q[0][r * LD + half + i], sm.q[1][r * LD + half + i]);
        split(ku * c - kv * s, sm.k[0][r * LD + i], sm.k[1][r * LD + i]);
        split(kv * c + ku * s, sm.k[0][r * LD + half + i], sm.k[1][r * LD + half + i]);
      }
      for (int dd = a.rot_dims + lane; dd < a.dim; dd += 32) split(get(sm.k, dd) * a.kscale, sm.k[0][r * LD + dd], sm.k[1][r * LD + dd]);
    }
    __syncthreads();
    if (own)
      for (int i = tid; i < 4 * n * (DK / 8); i += NTHR) {
        const int pl = i / (n * (DK / 8)), r = i / (DK / 8) % n, dd = i % (DK / 8) * 8;
        const __nv_bfloat16* src = pl < 2 ? sm.q[pl] : sm.k[pl - 2];
        *reinterpret_cast<uint4*>(a.qk + pl * qk_plane + ((size_t)(t0 + r) * a.G + kh) * DK + dd) =
            *reinterpret_cast<const uint4*>(src + r * LD + dd);
      }
  }
  if (DELTA && warp == 0) {                        // log decays summed over the chunk, two tokens per lane
    float l0 = 2 * lane < n ? la_log_decay(a, t0 + 2 * lane, h) : 0.f, l1 = 2 * lane + 1 < n ? la_log_decay(a, t0 + 2 * lane + 1, h) : 0.f;
    float s = l0 + l1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, s, o);
      if (lane >= o) s += v;
    }
    float before = __shfl_up_sync(0xffffffffu, s, 1);
    if (lane == 0) before = 0.f;
    sm.b[2 * lane] = before + l0;
    sm.b[2 * lane + 1] = s;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = 2 * lane + e;
      const float be = r < n ? la_beta(a, t0 + r, h) : 0.f;
      sm.beta[r] = be;
      if (r < n) {
        a.lg[(size_t)(t0 + r) * a.H + h] = e == 0 ? before + l0 : s;
        a.beta[(size_t)(t0 + r) * a.H + h] = be;
      }
    }
  }
  __syncthreads();

  // rows mt * 16 .. of K K^T (delta rule: first four warps) and Q K^T; tiles above the diagonal are left out
  {
    const int mt = warp & 3;
    const bool kk = DELTA && warp < 4;
    const int nt0 = DELTA ? 0 : (warp >> 2) * 4, nt1 = min(DELTA ? 8 : nt0 + 4, 2 * mt + 2);
    const __nv_bfloat16* m0 = kk ? sm.k[0] : sm.q[0];
    const __nv_bfloat16* m1 = kk ? sm.k[1] : sm.q[1];
    constexpr int NT = DELTA ? 8 : 4;
    float acc[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    const int ao = mt * 16 * LD + a_off(lane, LD), bo = b_off(lane, LD);
#pragma unroll 2
    for (int ks = 0; ks < DK / 16; ++ks) {
      uint32_t ah[4], al[4];
      ldsm4(ah, m0 + ao + ks * 16);
      ldsm4(al, m1 + ao + ks * 16);
#pragma unroll
      for (int j = 0; j < NT; j += 2) {
        if (nt0 + j >= nt1) continue;
        uint32_t bh[4], bl[4];
        ldsm4(bh, sm.k[0] + (nt0 + j) * 8 * LD + bo + ks * 16);
        ldsm4(bl, sm.k[1] + (nt0 + j) * 8 * LD + bo + ks * 16);
        mma(acc[j], ah, bh[0], bh[1]);
        mma(acc[j + 1], ah, bh[2], bh[3]);
        mma(acc[j], ah, bl[0], bl[1]);
        mma(acc[j + 1], ah, bl[2], bl[3]);
        mma(acc[j], al, bh[0], bh[1]);
        mma(acc[j + 1], al, bh[2], bh[3]);
      }
    }
    const size_t plane = (size_t)a.chunks * a.H * CK * CK, base = ((size_t)chunk * a.H + h) * CK * CK;
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      if (nt0 + j >= nt1) continue;
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int i = mt * 16 + (lane >> 2) + hf * 8, c = (nt0 + j) * 8 + (lane & 3) * 2;
        float v[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int jj = c + e;
          const bool below = kk ? jj < i : jj <= i;
          const float ratio = !below ? 0.f : DELTA ? expf(sm.b[i] - sm.b[jj]) : a.pw[h * (CK + 1) + i - jj];
          v[e] = below ? acc[j][hf * 2 + e] * ratio : 0.f;
        }
        if (kk) {
          sm.A[i][c] = sm.beta[i] * v[0];
          sm.A[i][c + 1] = sm.beta[i] * v[1];
        } else {
          __align__(4) __nv_bfloat16 hi[2], lo[2];
          split(v[0], hi[0], lo[0]);
          split(v[1], hi[1], lo[1]);
          *reinterpret_cast<uint32_t*>(a.mats + base + i * CK + c) = *reinterpret_cast<uint32_t*>(hi);
          *reinterpret_cast<uint32_t*>(a.mats + plane + base + i * CK + c) = *reinterpret_cast<uint32_t*>(lo);
        }
      }
    }
    if constexpr (DELTA) {
      __syncthreads();
      // (I + A) X = I, a thread per column of X (zero above the diagonal)
      if (tid < CK) {
        float x[CK];
#pragma unroll
        for (int i = 0; i < CK; ++i) {
          float r = i == tid ? 1.f : 0.f, r1 = 0.f, r2 = 0.f, r3 = 0.f;
#pragma unroll
          for (int m = 0; m < (i & ~3); m += 4) {
            const float4 w = *reinterpret_cast<const float4*>(&sm.A[i][m]);
            r -= w.x * x[m];
            r1 -= w.y * x[m + 1];
            r2 -= w.z * x[m + 2];
            r3 -= w.w * x[m + 3];
          }
#pragma unroll
          for (int m = i & ~3; m < i; ++m) r -= sm.A[i][m] * x[m];
          x[i] = (r + r1) + (r2 + r3);
          __nv_bfloat16 hi, lo;
          split(x[i], hi, lo);
          a.mats[2 * plane + base + i * CK + tid] = hi;
          a.mats[3 * plane + base + i * CK + tid] = lo;
        }
      }
    }
  }
}

// ---------------------------------------------------------------- scan
template <int DK>
struct ScanSmem {
  static constexpr int LD = DK + 8;
  __nv_bfloat16 k[2][2][CK * LD];          // buffer, plane
  __nv_bfloat16 q[2][CK * LD];
  __nv_bfloat16 S[2][NV * LD];             // [column][row]
  __nv_bfloat16 X[2][CK * LDM], P[2][CK * LDM];
  __nv_bfloat16 v[CK * (NV + 8)];
  __nv_bfloat16 R[2][NV * LDM], D[2][NV * LDM], E[2][NV * LDM];      // [column][token]
  float b[2][CK], beta[2][CK];
};

// acc += A (16 rows, kt tiles of 16 columns, both planes) times B (NT blocks of 8 columns, both planes)
template <int NT, bool TRANS_A>
__device__ __forceinline__ void product(float (&acc)[NT][4], const __nv_bfloat16* a0, const __nv_bfloat16* a1, int a_step,
                                        const __nv_bfloat16* b0, const __nv_bfloat16* b1, int b_ld, int kt) {
#pragma unroll 4
  for (int ks = 0; ks < kt; ++ks) {
    uint32_t ah[4], al[4];
    if constexpr (TRANS_A) {
      ldsm4t(ah, a0 + ks * a_step);
      ldsm4t(al, a1 + ks * a_step);
    } else {
      ldsm4(ah, a0 + ks * a_step);
      ldsm4(al, a1 + ks * a_step);
    }
#pragma unroll
    for (int j = 0; j < NT; j += 2) {
      uint32_t bh[4], bl[4];
      ldsm4(bh, b0 + j * 8 * b_ld + ks * 16);
      ldsm4(bl, b1 + j * 8 * b_ld + ks * 16);
      mma(acc[j], ah, bh[0], bh[1]);
      mma(acc[j + 1], ah, bh[2], bh[3]);
      mma(acc[j], ah, bl[0], bl[1]);
      mma(acc[j + 1], ah, bl[2], bl[3]);
      mma(acc[j], al, bh[0], bh[1]);
      mma(acc[j + 1], al, bh[2], bh[3]);
    }
  }
}

template <int NT>
__device__ __forceinline__ void clear(float (&acc)[NT][4]) {
#pragma unroll
  for (int j = 0; j < NT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
}

// grid (n_seg, H, ceil(vcols / 32))
template <int DK, bool DELTA>
__global__ void __launch_bounds__(NTHR) linear_chunk_scan_kernel(const __grid_constant__ LinearArgs a) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  ScanSmem<DK>& sm = *reinterpret_cast<ScanSmem<DK>*>(smem_raw);
  constexpr int LD = ScanSmem<DK>::LD, NT = NV / 8;
  pdl_wait();
  pdl_launch();
  const int seg = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * NV, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int g = lane >> 2, c2 = (lane & 3) * 2;
  const int s0 = a.seg_start[seg], s1 = a.seg_start[seg + 1], slot = a.seg_slot[seg], kh = h / (a.H / a.G);
  if (!HE_INDEX_OK(slot, a.n_slots, HE_SITE_STATE_SLOT)) return;
  int chunk0 = 0;
  for (int s = 0; s < seg; ++s) chunk0 += (a.seg_start[s + 1] - a.seg_start[s] + CK - 1) / CK;
  const int n_chunks = (s1 - s0 + CK - 1) / CK;
  const float* pw = DELTA ? nullptr : a.pw + (size_t)h * (CK + 1);

  const auto load_rows = [&](int ch) {             // queries, keys, values, gates of chunk ch
    if (ch < n_chunks) {
      const int t0 = s0 + ch * CK, buf = ch & 1;
      const size_t plane = (size_t)a.T * a.G * DK;
      for (int i = tid; i < 4 * CK * (DK / 8); i += NTHR) {
        const int pl = i / (CK * (DK / 8)), r = i / (DK / 8) % CK, d = i % (DK / 8) * 8, t = t0 + r;
        const bool live = t < s1;
        const __nv_bfloat16* src = a.qk + pl * plane + ((size_t)(live ? t : s0) * a.G + kh) * DK + d;
        cp16((pl < 2 ? sm.q[pl] : sm.k[buf][pl - 2]) + r * LD + d, src, live);
      }
      for (int i = tid; i < CK * (NV / 8); i += NTHR) {
        const int r = i / (NV / 8), d = i % (NV / 8) * 8, t = t0 + r;
        const bool live = t < s1 && col0 + d < a.vcols;
        cp16(sm.v + r * (NV + 8) + d, a.vb + ((size_t)(t < s1 ? t : s0) * a.H + h) * a.vcols + (live ? col0 + d : 0), live);
      }
      if (DELTA && tid < CK) {
        const int t = t0 + tid;
        const bool live = t < s1;
        cp4(&sm.b[buf][tid], a.lg + (size_t)(live ? t : s0) * a.H + h, live);
        cp4(&sm.beta[buf][tid], a.beta + (size_t)(live ? t : s0) * a.H + h, live);
      }
    }
    cp_commit();
  };
  const auto load_matrix = [&](int ch, int which, __nv_bfloat16 (&dst)[2][CK * LDM]) {
    if (ch < n_chunks) {
      const size_t plane = (size_t)a.chunks * a.H * CK * CK, base = ((size_t)(chunk0 + ch) * a.H + h) * CK * CK;
      for (int i = tid; i < 2 * CK * (CK / 8); i += NTHR) {
        const int pl = i / (CK * (CK / 8)), r = i / (CK / 8) % CK, d = i % (CK / 8) * 8;
        cp16(dst[pl] + r * LDM + d, a.mats + (which + pl) * plane + base + r * CK + d, true);
      }
    }
    cp_commit();
  };

  // state: warp w keeps rows [16 w, 16 w + 16) of the CTA's columns
  float* Sg = a.S + ((size_t)slot * a.H + h) * a.dim * a.vcols + col0;
  const bool has_rows = warp < DK / 16;
  float S[NT][4];
  const auto publish = [&]() {
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int o = (j * 8 + c2 + (e & 1)) * LD + warp * 16 + g + (e >> 1) * 8;
        split(S[j][e], sm.S[0][o], sm.S[1][o]);
      }
  };
  load_rows(0);
  if constexpr (DELTA) load_matrix(0, 2, sm.X);
  else cp_commit();
  if (has_rows) {
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = warp * 16 + g + (e >> 1) * 8, c = j * 8 + c2 + (e & 1);
        S[j][e] = d < a.dim && col0 + c < a.vcols ? Sg[(size_t)d * a.vcols + c] : 0.f;
      }
    publish();
  }
  const int mt = warp & 3;                         // 16 tokens of the chunk: first four warps K S, the others Q S
  const int ao = mt * 16 * LD + a_off(lane, LD), am = mt * 16 * LDM + a_off(lane, LDM);
  for (int ch = 0; ch < n_chunks; ++ch) {
    const int buf = ch & 1, t0 = s0 + ch * CK, n = min(CK, s1 - t0);
    cp_wait<1>();
    __syncthreads();                               // rows of this chunk, and the state's planes
    load_matrix(ch, 0, sm.P);
    const float* b = sm.b[buf];
    const auto upto = [&](int i) { return DELTA ? expf(b[i]) : pw[min(i, n - 1) + 1]; };      // decay up to token i
    const auto rest = [&](int i) { return DELTA ? expf(b[n - 1] - b[i]) : pw[max(n - 1 - i, 0)]; };   // ... behind it
    float acc[NT][4];
    clear(acc);
    if (warp >= 4) {
      product<NT, false>(acc, sm.q[0] + ao, sm.q[1] + ao, 16, sm.S[0] + b_off(lane, LD), sm.S[1] + b_off(lane, LD), LD, DK / 16);
    } else if (DELTA) {
      product<NT, false>(acc, sm.k[buf][0] + ao, sm.k[buf][1] + ao, 16, sm.S[0] + b_off(lane, LD), sm.S[1] + b_off(lane, LD), LD,
                         DK / 16);
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int i = mt * 16 + g + hf * 8;
        const float up = upto(i), be = sm.beta[buf][i];
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int c = j * 8 + c2 + e;
            const float r = be * (bf16_to_f32(sm.v[i * (NV + 8) + c]) - up * acc[j][hf * 2 + e]);
            split(r, sm.R[0][c * LDM + i], sm.R[1][c * LDM + i]);
          }
      }
    } else {
      for (int k = tid; k < CK * NV; k += 128) {
        const int i = k / NV, c = k % NV;
        const __nv_bfloat16 v = sm.v[i * (NV + 8) + c];
        sm.D[0][c * LDM + i] = v;
        sm.D[1][c * LDM + i] = f32_to_bf16(0.f);
        split(bf16_to_f32(v) * rest(i), sm.E[0][c * LDM + i], sm.E[1][c * LDM + i]);
      }
    }
    if constexpr (DELTA) {
      cp_wait<1>();
      __syncthreads();                             // R, inverse
      load_rows(ch + 1);
      float d[2][4];
      clear(d);
      const int n0 = (warp >> 2) * 16;             // two column blocks per warp
      product<2, false>(d, sm.X[0] + am, sm.X[1] + am, 16, sm.R[0] + n0 * LDM + b_off(lane, LDM),
                        sm.R[1] + n0 * LDM + b_off(lane, LDM), LDM, mt + 1);
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int i = mt * 16 + g + hf * 8;
        const float re = rest(i);
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int o = (n0 + j * 8 + c2 + e) * LDM + i;
            split(d[j][hf * 2 + e], sm.D[0][o], sm.D[1][o]);
            split(d[j][hf * 2 + e] * re, sm.E[0][o], sm.E[1][o]);
          }
      }
      cp_wait<1>();
      __syncthreads();                             // D, E, P
      load_matrix(ch + 1, 2, sm.X);
    } else {
      cp_wait<0>();
      __syncthreads();                             // D, E, P
      load_rows(ch + 1);
      cp_commit();
    }
    if (warp >= 4) {
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const float up = upto(mt * 16 + g + hf * 8);
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          acc[j][hf * 2] *= up;
          acc[j][hf * 2 + 1] *= up;
        }
      }
      product<NT, false>(acc, sm.P[0] + am, sm.P[1] + am, 16, sm.D[0] + b_off(lane, LDM), sm.D[1] + b_off(lane, LDM), LDM, mt + 1);
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int i = mt * 16 + g + hf * 8;
        if (i < n) {
          float* o = a.o + ((size_t)(t0 + i) * a.H + h) * a.vcols + col0 + c2;
#pragma unroll
          for (int j = 0; j < NT; ++j)
            if (col0 + j * 8 < a.vcols) *reinterpret_cast<float2*>(o + j * 8) = make_float2(acc[j][hf * 2], acc[j][hf * 2 + 1]);
        }
      }
    }
    if (has_rows) {
      const float all = upto(n - 1);
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[j][e] *= all;
      const int ko = warp * 16 + at_off(lane, LD);
      product<NT, true>(S, sm.k[buf][0] + ko, sm.k[buf][1] + ko, 16 * LD, sm.E[0] + b_off(lane, LDM), sm.E[1] + b_off(lane, LDM), LDM,
                        CK / 16);
      publish();                                   // read again behind the next barrier
    }
  }
  cp_wait<0>();
  if (has_rows) {
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = warp * 16 + g + (e >> 1) * 8, c = j * 8 + c2 + (e & 1);
        if (d < a.dim && col0 + c < a.vcols) Sg[(size_t)d * a.vcols + c] = S[j][e];
      }
  }
  if (DELTA && a.taps > 1)                         // the CTAs of a segment share its ring's columns
    for (int c = (h * gridDim.z + blockIdx.z) * NTHR + tid; c < a.C; c += a.H * gridDim.z * NTHR) la_ring_update(a, slot, s0, s1, c);
}

int check(const LinearArgs& a) {
  return a.H < 1 || a.G < 1 || a.H % a.G != 0 || a.dim < 1 || a.dim > 128 || a.vdim < 1 || a.vcols < a.vdim || a.vcols % 8 != 0 ||
                 a.H > 65535 || a.n_seg < 1 || a.chunks < a.T / CK + (a.T % CK != 0) || a.jS != nullptr ||
                 (a.delta && a.taps > 1 && a.ring == nullptr) || (!a.delta && a.pw == nullptr)
             ? -HE_ERR_BAD_ARG : 0;
}

template <typename K>
int launch(K kernel, dim3 grid, size_t smem, const LinearArgs& a, cudaStream_t stream) {
  cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  return (int)launch_pdl(kernel, grid, dim3(NTHR), smem, stream, a);
}

}  // namespace

HE_API int he_linear_chunk_prepare(const LinearArgs* args, cudaStream_t stream) {
  const LinearArgs& a = *args;
  if (a.T <= 0) return 0;
  if (check(a) != 0) return -HE_ERR_BAD_ARG;
  const dim3 grid(a.chunks, a.H);
  if (a.dim <= 64)
    return a.delta ? launch(linear_chunk_prepare_kernel<64, true>, grid, sizeof(PrepSmem<64>), a, stream)
                   : launch(linear_chunk_prepare_kernel<64, false>, grid, sizeof(PrepSmem<64>), a, stream);
  return a.delta ? launch(linear_chunk_prepare_kernel<128, true>, grid, sizeof(PrepSmem<128>), a, stream)
                 : launch(linear_chunk_prepare_kernel<128, false>, grid, sizeof(PrepSmem<128>), a, stream);
}

HE_API int he_linear_chunk_scan(const LinearArgs* args, cudaStream_t stream) {
  const LinearArgs& a = *args;
  if (a.T <= 0) return 0;
  if (check(a) != 0) return -HE_ERR_BAD_ARG;
  const dim3 grid(a.n_seg, a.H, (a.vcols + NV - 1) / NV);
  if (a.dim <= 64)
    return a.delta ? launch(linear_chunk_scan_kernel<64, true>, grid, sizeof(ScanSmem<64>), a, stream)
                   : launch(linear_chunk_scan_kernel<64, false>, grid, sizeof(ScanSmem<64>), a, stream);
  return a.delta ? launch(linear_chunk_scan_kernel<128, true>, grid, sizeof(ScanSmem<128>), a, stream)
                 : launch(linear_chunk_scan_kernel<128, false>, grid, sizeof(ScanSmem<128>), a, stream);
}
