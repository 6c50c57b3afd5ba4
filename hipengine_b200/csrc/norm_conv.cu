// RMS norm over groups of channels for the two sublayers of a parallel layer, with the short causal convolution over time that
// precedes the mixer: n = norm(x) * w1, a[t] = n[t] + sum_j cw[j] n[t - taps + 1 + j], b = norm(x) * w2.
//
// Groups are independent, so a CTA owns one group of a tile of consecutive tokens of one segment.  A warp (or all warps, when
// there is one row) normalises a row into shared memory and writes the plain rows on the way; one barrier later the
// convolution runs from shared memory.  The taps - 1 rows ahead of a tile are normalised again; ahead of a segment they are the
// slot's state.  Only the CTA of a segment's first tile reads the state and only it replaces it, after that, with the
// segment's last rows (normalised again where they lie in another tile).  With a journal the state stays and the rows that
// would be the state after every token are recorded.
#include "common.cuh"

using namespace he;

struct NormConvArgs {
  const float* x;            // [T][ldx] residual rows, zero in padded columns
  long long ldx;
  const float* w1;           // [H] gains of the mixer's norm
  const float* w2;           // [H] gains of the other norm, or null
  const float* cw;           // [taps][H] oldest first, or null: no convolution
  float* state;              // [n_slots][taps - 1][H] normalised rows ahead of the segment, oldest first
  float* journal;            // [T][taps - 1][H] or null
  const int* seg_start;      // [n_seg + 1]; null: no convolution, rows are independent
  const int* seg_slot;       // [n_seg]
  void* a;                   // [T][H] bf16 or fp32
  void* b;                   // [T][H] or null
  int T, H, groups, gw;      // gw: real channels per group; H >= groups * gw
  int taps, n_seg, n_slots, out_bf16, tile;
  float eps;
};

namespace {

constexpr int NW = 8, NTHR = NW * 32;
constexpr int MAX_TILE = 32;
constexpr size_t SMEM_SOFT = 36 * 1024, SMEM_HARD = 200 * 1024;

template <int V> struct Vec;
template <> struct Vec<1> { float v[1]; };
template <> struct __align__(16) Vec<4> { float v[4]; };

template <int V>
__device__ __forceinline__ Vec<V> ldv(const float* p) { return *reinterpret_cast<const Vec<V>*>(p); }
template <int V>
__device__ __forceinline__ void stv(float* p, const Vec<V>& x) { *reinterpret_cast<Vec<V>*>(p) = x; }
template <int V>
__device__ __forceinline__ void stv(__nv_bfloat16* p, const Vec<V>& x) {
  if constexpr (V == 4) {
    __align__(8) __nv_bfloat162 o[2] = {__floats2bfloat162_rn(x.v[0], x.v[1]), __floats2bfloat162_rn(x.v[2], x.v[3])};
    *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(o);
  } else {
    *p = f32_to_bf16(x.v[0]);
  }
}

// V: channels per access (4 where a group is a multiple of four channels)
template <typename OutT, int V>
__global__ void __launch_bounds__(NTHR) norm_conv_kernel(const __grid_constant__ NormConvArgs a) {
  extern __shared__ __align__(16) float rows[];    // [past + tile][gw]: history, then the tile
  __shared__ float part[NW];
  pdl_wait();
  pdl_launch();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = blockIdx.y, gw = a.gw, c0 = g * gw, past = a.cw != nullptr ? a.taps - 1 : 0;
  int seg = 0, s0 = 0, s1 = a.T, tile = blockIdx.x, slot = 0;
  if (a.seg_start != nullptr) {
    if (a.n_seg == a.T) {
      seg = tile;
      tile = 0;
    } else {
      for (; seg < a.n_seg; ++seg) {
        const int n = (a.seg_start[seg + 1] - a.seg_start[seg] + a.tile - 1) / a.tile;
        if (tile < n) break;
        tile -= n;
      }
    }
    if (seg >= a.n_seg) return;
    s0 = a.seg_start[seg];
    s1 = a.seg_start[seg + 1];
    slot = a.seg_slot[seg];
    if (past > 0 && !HE_INDEX_OK(slot, a.n_slots, HE_SITE_STATE_SLOT)) return;
  }
  const int t0 = s0 + tile * a.tile, n = min(a.tile, s1 - t0);
  if (n <= 0) return;
  float* state = past > 0 ? a.state + (size_t)slot * past * a.H + c0 : nullptr;
  OutT* bo = reinterpret_cast<OutT*>(a.b);

  // rows[at ..] <- normalised rows t .. t + count - 1; the plain rows go out where `out` says so
  const auto normalise = [&](int t, int count, int at, bool out) {
    const int wpr = count == 1 ? NW : 1;                       // warps per row
    for (int r0 = 0; r0 < count; r0 += NW / wpr) {
      const int r = r0 + (wpr == 1 ? warp : 0), i0 = (wpr == 1 ? lane : (int)threadIdx.x) * V, step = wpr * 32 * V;
      float* dst = rows + (size_t)(at + r) * gw;
      const bool live = r < count;
      float ss = 0.f;
      if (live) {
        const float* src = a.x + (size_t)(t + r) * a.ldx + c0;
#pragma unroll 4
        for (int i = i0; i < gw; i += step) {
          const Vec<V> v = ldv<V>(src + i);
#pragma unroll
          for (int e = 0; e < V; ++e) ss += v.v[e] * v.v[e];
          stv<V>(dst + i, v);
        }
      }
      ss = warp_sum(ss);
      if (wpr > 1) {
        if (lane == 0) part[warp] = ss;
        __syncthreads();
        ss = 0.f;
#pragma unroll
        for (int w = 0; w < NW; ++w) ss += part[w];
      }
      if (!live) continue;
      const float inv = rsqrtf(ss / (float)gw + a.eps);
      const bool plain = out && bo != nullptr && t + r >= t0;
#pragma unroll 4
      for (int i = i0; i < gw; i += step) {
        Vec<V> v = ldv<V>(dst + i), w = ldv<V>(a.w1 + c0 + i), u = v;
#pragma unroll
        for (int e = 0; e < V; ++e) v.v[e] *= inv * w.v[e];
        stv<V>(dst + i, v);
        if (plain) {
          w = ldv<V>(a.w2 + c0 + i);
#pragma unroll
          for (int e = 0; e < V; ++e) u.v[e] *= inv * w.v[e];
          stv<V>(bo + (size_t)(t + r) * a.H + c0 + i, u);
        }
      }
    }
  };

  // history: state rows ahead of the segment, then rows of this segment ahead of the tile (recomputed with the tile)
  const int again = min(past, t0 - s0), old = past - again;    // rows of the segment / of the state among the history
  for (int i = threadIdx.x * V; i < old * gw; i += NTHR * V) {
    const int j = i / gw, c = i - j * gw;                      // history row j is state row j + again
    stv<V>(rows + i, ldv<V>(state + (size_t)(j + again) * a.H + c));
  }
  normalise(t0 - again, n + again, old, true);
  __syncthreads();
  OutT* ao = reinterpret_cast<OutT*>(a.a);
  for (int i = threadIdx.x * V; i < n * gw; i += NTHR * V) {
    const int r = i / gw, c = i - r * gw;
    const float* p = rows + (size_t)r * gw + c;                // row r of the window: the oldest tap
    Vec<V> acc = ldv<V>(p + (size_t)past * gw);
    if (a.cw != nullptr) {
      for (int j = 0; j <= past; ++j) {
        const Vec<V> w = ldv<V>(a.cw + (size_t)j * a.H + c0 + c), v = ldv<V>(p + (size_t)j * gw);
#pragma unroll
        for (int e = 0; e < V; ++e) acc.v[e] += w.v[e] * v.v[e];
        if (a.journal != nullptr && j > 0) stv<V>(a.journal + ((size_t)(t0 + r) * past + j - 1) * a.H + c0 + c, v);
      }
    }
    stv<V>(ao + (size_t)(t0 + r) * a.H + c0 + c, acc);
  }
  const int pad0 = a.groups * gw;
  if (g == a.groups - 1 && pad0 < a.H) {                       // padded columns
    const int np = a.H - pad0;
    for (int i = threadIdx.x; i < n * np; i += NTHR) {
      const size_t o = (size_t)(t0 + i / np) * a.H + pad0 + i % np;
      if constexpr (sizeof(OutT) == 2) {
        ao[o] = f32_to_bf16(0.f);
        if (bo != nullptr) bo[o] = f32_to_bf16(0.f);
      } else {
        ao[o] = 0.f;
        if (bo != nullptr) bo[o] = 0.f;
      }
    }
    if (a.journal != nullptr)
      for (int i = threadIdx.x; i < n * past * np; i += NTHR)
        a.journal[((size_t)t0 * past + i / np) * a.H + pad0 + i % np] = 0.f;
  }
  if (past == 0 || tile != 0 || a.journal != nullptr) return;
  const int len = s1 - s0;
  int first = n;                                               // row of `rows` that becomes state row 0
  if (len > n) {                                               // the last rows lie in another tile
    __syncthreads();
    normalise(s1 - past, past, 0, false);
    __syncthreads();
    first = 0;
  }
  for (int i = threadIdx.x * V; i < past * gw; i += NTHR * V) {
    const int j = i / gw, c = i - j * gw;
    stv<V>(state + (size_t)j * a.H + c, ldv<V>(rows + (size_t)first * gw + i));
  }
}

template <typename OutT, int V>
int launch(const NormConvArgs& a, dim3 grid, size_t smem, cudaStream_t stream) {
  // the attribute belongs to the (function, device) pair: set on every call that needs it
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(norm_conv_kernel<OutT, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return (int)launch_pdl(norm_conv_kernel<OutT, V>, grid, dim3(NTHR), smem, stream, a);
}

}  // namespace

HE_API int he_norm_conv(const NormConvArgs* args, cudaStream_t stream) {
  NormConvArgs a = *args;
  if (a.T <= 0) return 0;
  const int past = a.cw != nullptr ? a.taps - 1 : 0;
  if (a.groups < 1 || a.gw < 1 || a.groups > 65535 || a.groups * (long long)a.gw > a.H || (a.cw != nullptr && a.taps < 1) ||
      (a.cw != nullptr && a.seg_start == nullptr) || (past > 0 && (a.state == nullptr || a.seg_slot == nullptr)) ||
      (a.seg_start != nullptr && a.n_seg < 1) || ((a.b != nullptr) != (a.w2 != nullptr)))
    return -HE_ERR_BAD_ARG;
  const size_t row = (size_t)a.gw * sizeof(float);
  const int least = past > 1 ? past : 1;
  // tokens per tile: enough CTAs, a bounded share of shared memory, and never fewer than the history has rows
  long long t = (long long)a.T * a.groups / (4 * 148);
  const long long fit = (long long)(SMEM_SOFT / row) - past;
  if (t > fit) t = fit;
  if (t > MAX_TILE) t = MAX_TILE;
  if (t < least) t = least;
  a.tile = (int)t;
  size_t smem = (size_t)(past + a.tile) * row;
  if (smem > SMEM_HARD) return -HE_ERR_BAD_ARG;
  const bool v4 = a.gw % 4 == 0 && a.H % 4 == 0 && a.ldx % 4 == 0;
  const bool single = a.seg_start != nullptr && a.n_seg == a.T;          // one row per segment
  const dim3 g(single ? a.T : (a.T + a.tile - 1) / a.tile + (a.seg_start != nullptr ? a.n_seg : 0), a.groups);
  if (a.out_bf16) return v4 ? launch<__nv_bfloat16, 4>(a, g, smem, stream) : launch<__nv_bfloat16, 1>(a, g, smem, stream);
  return v4 ? launch<float, 4>(a, g, smem, stream) : launch<float, 1>(a, g, smem, stream);
}
HE_API int he_norm_conv_args_size() { return (int)sizeof(NormConvArgs); }
