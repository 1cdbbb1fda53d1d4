// Combines the partial results of attention whose keys were split over several CTAs.
#pragma once
#include "sm100_common.cuh"

namespace rb {

// Sigmoid gate on attention output: none, one number per output number, or one per head.
enum : int { ATTN_GATE_NONE = 0, ATTN_GATE_ELEMENT = 1, ATTN_GATE_HEAD = 2 };

// Soft cap of scores: cap tanh(score / cap).  `in` = 2 log2(e) / cap turns a score into the exponent of e^(2 score / cap);
// written with the exponential, whose absolute error in the result stays near 1e-6 of the cap.
__device__ __forceinline__ float soft_cap(float s, float in, float cap) {
  return cap - __fdividef(2.0f * cap, 1.0f + fast_exp2(s * in));
}

template <typename T>
__device__ __forceinline__ float sigmoid_f(float z) {
  return sizeof(T) == 4 ? 1.0f / (1.0f + expf(-z)) : __fdividef(1.0f, 1.0f + __expf(-z));
}

// part_o [rows, heads, splits, n] sums weighted by 2^(score - maximum), part_ml [rows, heads, splits, 2] (maximum in
// log2 units, sum of weights).  The sink adds exp(sink) to the denominator; the result is multiplied by out_scale.  Head h of row t goes to
// out[t * ldo + h * n]; gate rows are ldg apart.  A CTA takes 128 numbers of one (row, head): each warp every
// fourth split, four numbers a lane.
template <typename T>
__global__ void __launch_bounds__(128)
    attn_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                      const float* __restrict__ sink, const T* __restrict__ gate, long long ldg, int gate_kind,
                      T* __restrict__ out, long long ldo, int heads, int n, int splits, float out_scale) {
  __shared__ float s_o[4][128], s_l[4];
  const long long bh = blockIdx.x;
  const int h = (int)(bh % heads);
  const long long row = bh / heads;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int d = blockIdx.y * 128 + lane * 4;
  const float2* ml = reinterpret_cast<const float2*>(part_ml) + bh * splits;
  const float sk = sink ? sink[h] * 1.4426950408889634f : -INFINITY;
  float gm = sk;
  for (int s = lane; s < splits; s += 32) gm = fmaxf(gm, ml[s].x);
  gm = warp_max(gm);
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  float l = 0.f;
  if (gm != -INFINITY) {
#pragma unroll 4
    for (int s = warp; s < splits; s += 4) {
      const float2 v = ml[s];
      if (v.x != -INFINITY) {
        const float f = exp2f(v.x - gm);
        l += v.y * f;
        if (d < n) {
          const float4 q = *reinterpret_cast<const float4*>(part_o + (bh * splits + s) * n + d);
          o.x += q.x * f; o.y += q.y * f; o.z += q.z * f; o.w += q.w * f;
        }
      }
    }
  }
  *reinterpret_cast<float4*>(&s_o[warp][lane * 4]) = o;
  if (lane == 0) s_l[warp] = l;
  __syncthreads();
  float gl = s_l[0] + s_l[1] + s_l[2] + s_l[3];
  if (sink) gl += exp2f(sk - gm);
  const float inv = gl > 0.f ? out_scale / gl : 0.f;
  const int e = blockIdx.y * 128 + threadIdx.x;
  if (e < n) {
    float v = (s_o[0][threadIdx.x] + s_o[1][threadIdx.x] + s_o[2][threadIdx.x] + s_o[3][threadIdx.x]) * inv;
    if (gate_kind == ATTN_GATE_ELEMENT) v *= sigmoid_f<T>(to_f32<T>(gate[row * ldg + (long long)h * n + e]));
    else if (gate_kind == ATTN_GATE_HEAD) v *= sigmoid_f<T>(to_f32<T>(gate[row * ldg + h]));
    out[row * ldo + (long long)h * n + e] = from_f32<T>(v);
  }
}

template <typename T>
void launch_attn_merge(const float* part_o, const float* part_ml, const float* sink, const T* gate, long long ldg,
                       int gate_kind, T* out, long long ldo, int rows, int heads, int n, int splits, cudaStream_t st,
                       float out_scale = 1.0f) {
  attn_merge_kernel<T><<<dim3((unsigned)(rows * heads), (n + 127) / 128), 128, 0, st>>>(part_o, part_ml, sink, gate, ldg,
                                                                                       gate_kind, out, ldo, heads, n, splits, out_scale);
}

}  // namespace rb
