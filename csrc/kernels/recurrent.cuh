// What the kernels of recurrent mixers share: gates, output norm and gate, the inputs a convolution keeps.
//
// A sequence's portion is {first row, tokens, place of its state, position of the first token}.
#pragma once
#include "sm100_common.cuh"

namespace rb {

template <typename T>
__device__ __forceinline__ float rec_sigmoid(float z) {
  return sizeof(T) == 4 ? 1.0f / (1.0f + expf(-z)) : __fdividef(1.0f, 1.0f + __expf(-z));
}
// by the hardware tanh (relative error about 2^-11), for results that are rounded to 16 bits
__device__ __forceinline__ float sigmoid_tanh(float z) { return fmaf(fast_tanh(0.5f * z), 0.5f, 0.5f); }
// log(1 + e^x)
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }

// The output gate: sigmoid(z), or silu(z).
template <typename T>
__device__ __forceinline__ float rec_gate(float z, int silu) {
  const float s = rec_sigmoid<T>(z);
  return silu ? z * s : s;
}

// How a head's results leave the kernel: divided by their root mean square, times a weight, times a gate.
template <typename T>
struct RecOut {
  T* out;                        // row t, head h at out + t * ldo + h * vdim_p
  long long ldo;
  const T* gate;                 // the same layout, ldg apart
  long long ldg;
  const float* norm;             // norm + h * norm_step
  int norm_step;
  float* tmp;                    // [rows, heads * vdim_p], used when a head has several blocks of columns
  float eps;
  int silu;                      // gate: 0 sigmoid, 1 silu
};
template <typename T>
__device__ __forceinline__ void rec_write(const RecOut<T>& p, long long row, int h, int c, int vdim_p, float o, float r) {
  const long long col = (long long)h * vdim_p + c;
  p.out[row * p.ldo + col] = from_f32<T>(o * r * p.norm[h * p.norm_step + c] * rec_gate<T>(to_f32<T>(p.gate[row * p.ldg + col]), p.silu));
}
// log input and log forget gate from what the projection left
__device__ __forceinline__ float2 mlstm_gates(float zi, float zf, float cap) {
  return make_float2(cap * tanhf(zi / cap), -softplus_f(-cap * tanhf(zf / cap)));
}

// The inputs of a head's convolutions: query, key and value channels side by side, 2 dim_p + vdim_p of them.  Heads that
// share queries and keys keep a copy each.  Channel c of them among the channels of all heads:
__device__ __forceinline__ int delta_channel(int c, int h, int heads, int kv_heads, int dim_p, int vdim_p) {
  const int kh = h / (heads / kv_heads);
  return c < dim_p ? kh * dim_p + c : c < 2 * dim_p ? (kv_heads + kh) * dim_p + c - dim_p : 2 * kv_heads * dim_p + h * vdim_p + c - 2 * dim_p;
}
// The inputs that the next portion needs, after this one: conv [places, heads, taps - 1, 2 dim_p + vdim_p].
template <typename T>
__device__ __forceinline__ void delta_keep_inputs(const T* raw, long long ldr, T* conv, int4 seq, int h, int heads, int kv_heads, int dim_p,
                                                  int vdim_p, int taps, int tid, int threads) {
  const int own = 2 * dim_p + vdim_p, past = taps - 1;
  T* st = conv + ((long long)seq.z * heads + h) * past * own;
  for (int c = tid; c < own; c += threads) {
    const int ch = delta_channel(c, h, heads, kv_heads, dim_p, vdim_p);
    for (int j = 0; j < past; ++j) {           // upwards: an entry is read before it is overwritten
      const int at = seq.y - past + j;
      st[(long long)j * own + c] = at >= 0     ? raw[(long long)(seq.x + at) * ldr + ch]
                                   : seq.w > 0 ? st[(long long)(at + past) * own + c]
                                               : from_f32<T>(0.f);
    }
  }
}

}  // namespace rb
