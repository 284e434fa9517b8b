// Real-gated linear recurrence with diagonal state (RG-LRU), the arithmetic shared by its kernels.
//
//   r = sigmoid(zr), i = sigmoid(zi)                 gates, from a block-diagonal product of u
//   log a = -c r softplus(lam)                       decay
//   S_t = a S_(t-1) + sqrt(1 - a^2) i u              state, fp32
//   out = S_t gelu(y)                                with the other branch of the block
#pragma once
#include "row_vec.cuh"

namespace ft {

struct RglruGateParams {
  const void* u;            // [rows, ldu]: the convolved branch
  const float* r_bias;      // [channels]
  const float* i_bias;
  const float* decay;       // [channels]: -c softplus(lam)
  float* a;                 // fp32 [rows, channels]: decay of the row
  float* x;                 // fp32 [rows, channels]: input term of the row
  long long ldu;
  int channels;
  // rows 0 .. n_single - 1 are the only new token of their sequence: their recurrence is one step, taken at once
  int n_single;
  const int* pos;
  const int* slots;
  float* state;             // fp32 [slots, channels]
  const void* y;            // [rows, ldy]: the other branch ahead of its activation
  void* out;                // [rows, ldo]
  long long ldy, ldo;
};

// Each function comes in two forms: for fp32 models with CUDA's accurate functions, ahead of bf16 operands and results
// with the approximate instructions (both work in 32-bit; the second is good to a few units in the last place).
__device__ __forceinline__ float sigmoid_row(float z, const float*) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float fast_rcp(float x) {
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
__device__ __forceinline__ float sigmoid_row(float z, const __nv_bfloat16*) {
  return fast_rcp(1.f + fast_exp2(-1.4426950408889634f * z));
}
__device__ __forceinline__ float gelu_row(float g, const float*) {
  const float k = 0.7978845608028654f * (g + 0.044715f * g * g * g);
  return 0.5f * g * (1.f + tanhf(k));
}
// 0.5 (1 + tanh k) = 1 / (1 + exp(-2 k))
__device__ __forceinline__ float gelu_row(float g, const __nv_bfloat16*) {
  return g * sigmoid_row(1.5957691216057308f * (g + 0.044715f * g * g * g), static_cast<const __nv_bfloat16*>(nullptr));
}

// a = exp(log_a) and sqrt(1 - a^2) from q = a - 1: decays are often within 1e-3 of one, where an error in the last place
// of exp would change the length of the memory, and the difference 1 - a^2 would cancel.
__device__ __forceinline__ void decay_and_gain(float log_a, float& a, float& gain, const float*) {
  const float q = expm1f(log_a);
  a = 1.f + q;
  gain = sqrtf(-q * (2.f + q));
}
// The same with q from the Taylor series of exp(z) - 1 near zero (seven terms: 3e-9 of q at 0.25) and a plain difference away from it.
__device__ __forceinline__ void decay_and_gain(float log_a, float& a, float& gain, const __nv_bfloat16*) {
  const float z = log_a;
  const float near = z * (1.f + z * (0.5f + z * (1.f / 6 + z * (1.f / 24 + z * (1.f / 120 + z * (1.f / 720 + z * (1.f / 5040)))))));
  const float q = z > -0.25f ? near : fast_exp2(1.4426950408889634f * z) - 1.f;
  a = 1.f + q;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(gain) : "f"(-q * (2.f + q)));
}

// Decay and input term of eight channels c .. c + 7 of one row from its gates' pre-activations zr, zi (without bias) and its
// convolved branch u.
template <typename T>
__device__ __forceinline__ void rglru_gates8(const RglruGateParams& p, int c, const float* zr, const float* zi, const float* u, float* a,
                                             float* x) {
  const T* kind = nullptr;
  float br[8], bi[8], dec[8];
  load8(p.r_bias + c, br);
  load8(p.i_bias + c, bi);
  load8(p.decay + c, dec);
#pragma unroll
  for (int e = 0; e < 8; ++e) {
    float gain;
    decay_and_gain(dec[e] * sigmoid_row(zr[e] + br[e], kind), a[e], gain, kind);
    x[e] = gain * sigmoid_row(zi[e] + bi[e], kind) * u[e];
  }
}

// One step of the recurrence for eight channels of a row that is its sequence's only token.
template <typename T>
__device__ __forceinline__ void rglru_step8(const RglruGateParams& p, long long row, int c, const float* a, const float* x) {
  float* st = p.state + static_cast<long long>(p.slots[row]) * p.channels + c;
  float s[8], y[8];
  load8(static_cast<const T*>(p.y) + row * p.ldy + c, y);
  load8(static_cast<const float*>(st), s);
  const bool fresh = p.pos[row] == 0;       // a sequence starts from zero, whatever the slot held before
#pragma unroll
  for (int e = 0; e < 8; ++e) {
    s[e] = fresh ? x[e] : a[e] * s[e] + x[e];
    y[e] = s[e] * gelu_row(y[e], static_cast<const T*>(nullptr));
  }
  store8(st, s);
  store8(static_cast<T*>(p.out) + row * p.ldo + c, y);
}

}  // namespace ft
