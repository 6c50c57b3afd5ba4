// Real-gated linear recurrence (RG-LRU): arguments and arithmetic shared by the scan (rglru.cu) and the one-token step
// (gemv_float.cu).
//
// Per channel: r = sigmoid(gate 0), i = sigmoid(gate 1), a = exp(decay * r) (decay = -8 softplus(lambda)),
// S <- a S + sqrt(1 - a^2) i u, output S * gelu(y).  All of it in fp32.
#pragma once

#include "common.cuh"

struct RglruArgs {
  const float* g;            // gate products: block b, token t at b * g_bs + t * g_ts: block_cols of gate 0, then of gate 1 (scan)
  long long g_ts, g_bs;
  const __nv_bfloat16* gw;   // [blocks][2 * block_cols][block_cols] gate maps (step)
  const float* gb;           // [blocks][2 * block_cols] biases
  const float* decay;        // [C]
  const void* u;             // block b, token t, channel c of the block at b * u_bs + t * u_ts + c
  long long u_ts, u_bs;
  const void* y;             // [T][row_stride] rows of the output gate, without bias
  const float* yb;           // [C]
  const void* x;             // [T][row_stride] inputs of the convolution, without bias: the last ones become its state
  const float* xb;           // [C]
  long long row_stride;
  float* S;                  // [n_slots][C]
  float* cstate;             // [n_slots][taps - 1][C] biased inputs, oldest first
  float* journal;            // [T][C] S after every token; the states stay as they are then.  Or null
  const int* seg_start;      // [n_seg + 1]
  const int* seg_slot;       // [n_seg]
  void* out;                 // [T][out_stride]
  long long out_stride;
  int C, block_cols, taps, n_slots, n_seg, T;
  int row_dtype, act_f32;    // x and y rows: 0 f32, 1 bf16; u and out in fp32
};

namespace he {

__device__ __forceinline__ float rg_sigmoid(float x) { return __fdividef(1.f, 1.f + __expf(fminf(-x, 80.f))); }

// e^x - 1 for x <= 0 with a small relative error: the power series (nested) near zero, the difference elsewhere
__device__ __forceinline__ float rg_expm1(float x) {
  const float s = x * (1.f + x * (1.f / 2.f) * (1.f + x * (1.f / 3.f) * (1.f + x * (1.f / 4.f) * (1.f + x * (1.f / 5.f) *
                  (1.f + x * (1.f / 6.f))))));
  return x > -0.25f ? s : __expf(x) - 1.f;
}

__device__ __forceinline__ float rg_sqrt(float x) {
  float y;
  asm("sqrt.approx.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// gelu_tanh(z) = z / 2 (1 + tanh w) = z sigmoid(2 w)
__device__ __forceinline__ float rg_gelu(float z) {
  return z * rg_sigmoid(1.5957691216057308f * (z + 0.044715f * z * z * z));
}

// decay and drive of one token and channel.  Memories of thousands of tokens hang on 1 - a, so it is what is computed: an
// exponential next to one that is off by an ulp is off to the same side token after token.
__device__ __forceinline__ void rg_gates(float gr, float gi, float decay, float u, float& a, float& d) {
  const float m = rg_expm1(decay * rg_sigmoid(gr));               // a - 1
  a = 1.f + m;
  d = rg_sqrt(-m * (2.f + m)) * rg_sigmoid(gi) * u;
}

__device__ __forceinline__ float rg_load(const void* p, bool f32, size_t i) {
  return f32 ? reinterpret_cast<const float*>(p)[i] : bf16_to_f32(reinterpret_cast<const __nv_bfloat16*>(p)[i]);
}

// the convolution's state of channel c after rows [s0, s0 + n) of a segment
__device__ __forceinline__ void rg_conv_state(const RglruArgs& a, int slot, int c, int s0, int n) {
  const int past = a.taps - 1;
  float* st = a.cstate + (size_t)slot * past * a.C + c;
  for (int j = 0; j < past; ++j) {
    const int idx = n + j;                       // of [state ++ segment]; never behind j
    st[(size_t)j * a.C] = idx < past ? st[(size_t)idx * a.C]
                                     : rg_load(a.x, a.row_dtype == 0, (size_t)(s0 + idx - past) * a.row_stride + c) + a.xb[c];
  }
}

}  // namespace he
