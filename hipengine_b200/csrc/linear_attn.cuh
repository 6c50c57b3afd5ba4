// Linear attention with a matrix state per head: arguments and arithmetic shared by the serial kernels (linear_attn.cu) and the
// chunked prompt kernels (linear_chunk.cu).
//
// Per head, with a state S [dim][vdim] in fp32:
//   retention   q, k rotated (halves), k times kscale;          S <- g S + k v^T;                            o = S^T q
//   delta rule  q, k, v through a short causal convolution and silu, q and k brought to unit length, q times qscale;
//               S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// then o / rms(o) [* gain] * silu(z).  The decay is kept as g - 1: for memories of thousands of tokens that is what counts, and a
// number rounded next to one would be off to the same side every token.
//
// The convolution's past is a ring: the input of position p of a slot lies at p % taps.  A one-token step reads the other entries
// and writes its own, so the heads that share a query and key need no order among them.
#pragma once

#include "common.cuh"

struct LinearArgs {
  const void* rows;          // [T][stride] projected rows: q at 0, k at ck, v at cv (the convolution's C columns), z at cz
  long long stride;
  const float* ab;           // delta: [T][ab_stride] fp32, column h: logit of beta, column ca + h: input of the decay
  long long ab_stride;
  const float* gm;           // retention: [H] decay - 1
  const float* pw;           // retention, chunks: [H][65] powers of the decay
  const float* rate;         // delta: [H] exp(A_log)
  const float* dt;           // delta: [H]
  const float* cw;           // [taps][C] oldest first
  const double* freq;        // [rot_dims / 2]
  const float* gain;         // [vdim] or null
  float* S;                  // [n_slots][H][dim][vcols]
  float* ring;               // [n_slots][taps][C] or null (one tap)
  float* jS;                 // [T][H][dim][vcols]: the state after every token; the states stay as they are then.  Or null
  float* jring;              // [T][taps][C] or null
  const int* seg_start;      // [n_seg + 1]
  const int* seg_slot;       // [n_seg]
  const int* tok_seg;        // [T]
  const int* pos;            // [T]
  float* qf;                 // [T][G][dim] prepared rows
  float* kf;
  float* vf;                 // [T][H][vcols]
  float* g1;                 // [T][H] g - 1
  float* beta;               // [T][H]
  float* o;                  // [T][H][vcols]
  void* out;                 // [T][H * vcols]
  // chunks: planes of bf16 pairs (value, remainder)
  __nv_bfloat16* qk;         // [4][T][G][dk] q, q remainder, k, k remainder (dk: dim padded to 64 or 128)
  __nv_bfloat16* vb;         // [T][H][vcols]
  __nv_bfloat16* mats;       // [4][chunks][H][64][64] P, P remainder, inverse, inverse remainder
  float* lg;                 // [T][H] log decay summed from the chunk's start (inclusive)
  int T, n_seg, n_slots, H, G, dim, vdim, vcols, taps, C, ck, cv, cz, ca, rot_dims;
  int delta, row_dtype, out_f32;     // rows: 0 f32, 1 bf16
  int chunks;                // upper bound the matrices are laid out for
  float eps, kscale, qscale;
};

namespace he {

__device__ __forceinline__ float la_row(const LinearArgs& a, size_t i) {
  return a.row_dtype == 0 ? reinterpret_cast<const float*>(a.rows)[i]
                          : bf16_to_f32(reinterpret_cast<const __nv_bfloat16*>(a.rows)[i]);
}
__device__ __forceinline__ float la_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float la_silu(float x) { return x * la_sigmoid(x); }
__device__ __forceinline__ float la_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// log of head h's decay at token t (delta rule)
__device__ __forceinline__ float la_log_decay(const LinearArgs& a, int t, int h) {
  return -a.rate[h] * la_softplus(a.ab[(size_t)t * a.ab_stride + a.ca + h] + a.dt[h]);
}
__device__ __forceinline__ float la_beta(const LinearArgs& a, int t, int h) {
  return la_sigmoid(a.ab[(size_t)t * a.ab_stride + h]);
}

// silu of the convolution of column c at token t of a segment that starts at token s0
__device__ __forceinline__ float la_conv(const LinearArgs& a, int t, int s0, int slot, int p, int c) {
  float acc = 0.f;
  for (int j = 0; j < a.taps; ++j) {
    const int back = a.taps - 1 - j, q = p - back;              // position of the input
    float x = 0.f;
    if (t - back >= s0) x = la_row(a, (size_t)(t - back) * a.stride + c);
    else if (q >= 0) x = a.ring[((size_t)slot * a.taps + q % a.taps) * a.C + c];
    acc += a.cw[(size_t)j * a.C + c] * x;
    if (a.jring != nullptr && a.taps > 1) {
      const int e = q >= 0 ? q % a.taps : q + a.taps;           // q > -taps
      a.jring[((size_t)t * a.taps + e) * a.C + c] = x;
    }
  }
  return la_silu(acc);
}

// cosine and sine of pair i at position p, the angle reduced to one turn in double
__device__ __forceinline__ void la_angle(double freq, int p, float& c, float& s) {
  const double two_pi = 6.283185307179586476925286766559, per_turn = 0.15915494309189533576888376337251;
  const double ang = (double)p * freq;
  sincosf((float)(ang - two_pi * rint(ang * per_turn)), &s, &c);
}

// A warp prepares one query or key head of token t: dst[0 .. dim) (shared or global memory).  col: its first column
__device__ __forceinline__ void la_prepare_head(const LinearArgs& a, int t, int s0, int slot, int p, int col, float scale,
                                                float* dst, int lane) {
  if (a.delta) {
    float ss = 0.f;
    for (int d = lane; d < a.dim; d += 32) {
      const float x = la_conv(a, t, s0, slot, p, col + d);
      dst[d] = x;
      ss += x * x;
    }
    const float inv = scale / sqrtf(warp_sum(ss) + 1e-6f);
    for (int d = lane; d < a.dim; d += 32) dst[d] *= inv;
    return;
  }
  const int half = a.rot_dims >> 1;
  const size_t r = (size_t)t * a.stride + col;
  for (int i = lane; i < half; i += 32) {
    float c, s;
    la_angle(a.freq[i], p, c, s);
    const float u = la_row(a, r + i), v = la_row(a, r + half + i);
    dst[i] = (u * c - v * s) * scale;
    dst[half + i] = (v * c + u * s) * scale;
  }
  for (int d = a.rot_dims + lane; d < a.dim; d += 32) dst[d] = la_row(a, r + d) * scale;
}

// the ring after tokens [s0, s1) of a segment, column c
__device__ __forceinline__ void la_ring_update(const LinearArgs& a, int slot, int s0, int s1, int c) {
  for (int t = max(s0, s1 - a.taps); t < s1; ++t)
    a.ring[((size_t)slot * a.taps + a.pos[t] % a.taps) * a.C + c] = la_row(a, (size_t)t * a.stride + c);
}

}  // namespace he
