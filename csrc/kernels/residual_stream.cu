// A residual stream kept in fp32 for sm_100a: embedding rows scaled into it, and RMS norms that read it
// once and write one or two normed copies (two sub-layers that start from the same x, each with its own
// weight) in the type the following matrix product takes.  A norm can first add rows to x: what the chosen
// experts of a mixture left for each token.
//
// A residual may also be several parallel streams with learned connections (hyper-connections): a sub-layer reads a
// weighted sum of them, and afterwards the streams are mixed with one another and each gains a multiple of the
// sub-layer's result.  stream_mix_norm does all that lies between two sub-layers in one pass.
//
// Embeddings may be normed themselves, and a sub-layer's result scaled channel by channel before the sum (layer scale):
// embed_norm and scaled_add_norm, each up to the next sub-layer's input.
#include "sm100_common.cuh"

namespace rb {

// V numbers per thread and access (1: any width and alignment)
template <typename T, int V>
__global__ void __launch_bounds__(256)
    embed_scaled_kernel(const long long* __restrict__ ids, const T* __restrict__ table, float* __restrict__ x,
                        long long tokens, int D, int vocab, float scale) {
  const int groups = D / V;
  const long long n = tokens * groups;
  const long long stride = (long long)gridDim.x * blockDim.x;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += stride) {
    const int t = (int)(i / groups);
    const int c = (int)(i - (long long)t * groups) * V;
    const long long id = ids[t];
    const bool known = id >= 0 && id < vocab;
    if constexpr (V == 1) {
      x[(long long)t * D + c] = known ? to_f32<T>(table[id * D + c]) * scale : 0.f;
    } else {
      T e[V];
      if (known) {
        if constexpr (sizeof(T) == 2) *reinterpret_cast<uint2*>(e) = *reinterpret_cast<const uint2*>(table + id * D + c);
        else *reinterpret_cast<uint4*>(e) = *reinterpret_cast<const uint4*>(table + id * D + c);
      }
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
      if (known) o = make_float4(to_f32<T>(e[0]) * scale, to_f32<T>(e[1]) * scale, to_f32<T>(e[2]) * scale, to_f32<T>(e[3]) * scale);
      *reinterpret_cast<float4*>(x + (long long)t * D + c) = o;
    }
  }
}

// One CTA per row.  y1 / y2 have ldy columns per row; columns D .. ldy are written as zero (the product
// that follows may want a padded inner dimension).  The row is read twice, the second time from L1.
// ADD: x[t] += the rows add_rows[t, 0 .. n_add) of `add` (row stride lda) before the norm.
template <typename T, bool ADD>
__global__ void __launch_bounds__(256)
    rms_norm_stream_kernel(float* __restrict__ x, const float* __restrict__ w1, const float* __restrict__ w2,
                           T* __restrict__ y1, T* __restrict__ y2, int D, int ldy, float eps, const T* __restrict__ add,
                           long long lda, const int* __restrict__ add_rows, int n_add) {
  __shared__ float red[8];
  const long long row = blockIdx.x;
  float* xr = x + row * D;
  const int tid = threadIdx.x;
  float s = 0.f;
  const bool vec = (D & 3) == 0 && (!ADD || (lda & 3) == 0);
  const int* ar = ADD ? add_rows + row * n_add : nullptr;
  if (vec) {
    for (int c = tid * 4; c < D; c += 1024) {
      float4 v = *reinterpret_cast<const float4*>(xr + c);
      if constexpr (ADD) {
#pragma unroll 4
        for (int k = 0; k < n_add; ++k) {
          const T* a = add + ar[k] * lda + c;
          if constexpr (sizeof(T) == 4) {
            const float4 q = *reinterpret_cast<const float4*>(a);
            v.x += q.x; v.y += q.y; v.z += q.z; v.w += q.w;
          } else {
            const uint2 q = *reinterpret_cast<const uint2*>(a);
            const float2 lo = unpack2<T>(q.x), hi = unpack2<T>(q.y);
            v.x += lo.x; v.y += lo.y; v.z += hi.x; v.w += hi.y;
          }
        }
        *reinterpret_cast<float4*>(xr + c) = v;
      }
      s += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
  } else {
    for (int c = tid; c < D; c += 256) {
      float v = xr[c];
      if constexpr (ADD) {
        for (int k = 0; k < n_add; ++k) v += to_f32<T>(add[ar[k] * lda + c]);
        xr[c] = v;
      }
      s += v * v;
    }
  }
  s = warp_sum(s);
  if ((tid & 31) == 0) red[tid >> 5] = s;
  __syncthreads();
  s = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) s += red[i];
  const float r = 1.0f / sqrtf(s / D + eps);
  T* o1 = y1 + row * ldy;
  T* o2 = w2 ? y2 + row * ldy : nullptr;
  // a thread reads back only what it wrote itself
  if (vec && (ldy & 3) == 0) {
    for (int c = tid * 4; c < D; c += 1024) {
      const float4 v = *reinterpret_cast<const float4*>(xr + c);
      const float n[4] = {v.x * r, v.y * r, v.z * r, v.w * r};
      auto put = [&](const float* w, T* o) {
        const float4 g = *reinterpret_cast<const float4*>(w + c);
        if constexpr (sizeof(T) == 4) {
          *reinterpret_cast<float4*>(o + c) = make_float4(n[0] * g.x, n[1] * g.y, n[2] * g.z, n[3] * g.w);
        } else {
          *reinterpret_cast<uint2*>(o + c) =
              make_uint2(pack2<T>(n[0] * g.x, n[1] * g.y), pack2<T>(n[2] * g.z, n[3] * g.w));
        }
      };
      put(w1, o1);
      if (o2) put(w2, o2);
    }
  } else {
    if (ADD && vec) __syncthreads();       // columns were written in fours
    for (int c = tid; c < D; c += 256) {
      o1[c] = from_f32<T>(xr[c] * r * w1[c]);
      if (o2) o2[c] = from_f32<T>(xr[c] * r * w2[c]);
    }
  }
  for (int c = D + tid; c < ldy; c += 256) {
    o1[c] = from_f32<T>(0.f);
    if (o2) o2[c] = from_f32<T>(0.f);
  }
}

// One CTA per token.  From the old streams x_s and the last sub-layer's result y (fp32, plus rows of `add`):
//   x_t <- sum_s mix[s][t] x_s + w_out[t] y,   u = sum_s w_in[s] x_s,   h = u / sqrt(mean(u^2) + eps) * w
// y null: the streams stay as they are.  SN: streams, rounded up.  V numbers per thread and access.
struct StreamMixParams {
  const float* x;                // stream s of token t at x + t * ldx + s * sx (sx 0: all streams are equal)
  long long ldx, sx;
  float* xo;                     // [tokens, streams, D], may be x; null: the new streams are not kept
  const float* y;                // [tokens, D]
  const float *mix, *w_out, *w_in, *w;
  const int* add_rows;
  long long lda;
  int streams, D, ldh, n_add;
  float eps;
};
template <typename T, int SN, int V>
__global__ void __launch_bounds__(1024) stream_mix_norm_kernel(const StreamMixParams p, const T* __restrict__ add, T* __restrict__ h) {
  extern __shared__ __align__(16) float s_u[];
  __shared__ float red[32];
  const long long t = blockIdx.x;
  const int tid = threadIdx.x, S = p.streams, D = p.D, step = blockDim.x * V;
  float mix[SN][SN], wo[SN], wi[SN];
#pragma unroll
  for (int s = 0; s < SN; ++s) {
    wi[s] = s < S ? p.w_in[s] : 0.f;
    wo[s] = p.y && s < S ? p.w_out[s] : 0.f;
#pragma unroll
    for (int o = 0; o < SN; ++o) mix[s][o] = p.y && s < S && o < S ? p.mix[s * S + o] : 0.f;
  }
  const float* x = p.x + t * p.ldx;
  const int* ar = p.n_add ? p.add_rows + t * p.n_add : nullptr;
  float sq = 0.f;
  for (int c = tid * V; c < D; c += step) {
    float in[SN][V], y[V];
#pragma unroll
    for (int s = 0; s < SN; ++s) {
      if (s < S) {
        if constexpr (V == 4) *reinterpret_cast<float4*>(in[s]) = *reinterpret_cast<const float4*>(x + s * p.sx + c);
        else in[s][0] = x[s * p.sx + c];
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) in[s][e] = 0.f;
      }
    }
    float u[V];
#pragma unroll
    for (int e = 0; e < V; ++e) u[e] = 0.f;
    if (p.y) {
      if constexpr (V == 4) *reinterpret_cast<float4*>(y) = *reinterpret_cast<const float4*>(p.y + t * D + c);
      else y[0] = p.y[t * D + c];
#pragma unroll 4
      for (int k = 0; k < p.n_add; ++k) {
        const T* a = add + ar[k] * p.lda + c;
        if constexpr (V == 1) {
          y[0] += to_f32<T>(a[0]);
        } else if constexpr (sizeof(T) == 4) {
          const float4 q = *reinterpret_cast<const float4*>(a);
          y[0] += q.x; y[1] += q.y; y[2] += q.z; y[3] += q.w;
        } else {
          const uint2 q = *reinterpret_cast<const uint2*>(a);
          const float2 lo = unpack2<T>(q.x), hi = unpack2<T>(q.y);
          y[0] += lo.x; y[1] += lo.y; y[2] += hi.x; y[3] += hi.y;
        }
      }
#pragma unroll
      for (int o = 0; o < SN; ++o) {
        float v[V];
#pragma unroll
        for (int e = 0; e < V; ++e) {
          v[e] = wo[o] * y[e];
#pragma unroll
          for (int s = 0; s < SN; ++s) v[e] = fmaf(mix[s][o], in[s][e], v[e]);
          u[e] = fmaf(wi[o], v[e], u[e]);
        }
        if (p.xo && o < S) {
          if constexpr (V == 4) *reinterpret_cast<float4*>(p.xo + (t * S + o) * D + c) = *reinterpret_cast<float4*>(v);
          else p.xo[(t * S + o) * D + c] = v[0];
        }
      }
    } else {
#pragma unroll
      for (int s = 0; s < SN; ++s)
#pragma unroll
        for (int e = 0; e < V; ++e) u[e] = fmaf(wi[s], in[s][e], u[e]);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
      s_u[c + e] = u[e];
      sq += u[e] * u[e];
    }
  }
  sq = warp_sum(sq);
  if ((tid & 31) == 0) red[tid >> 5] = sq;
  __syncthreads();
  sq = 0.f;
  for (int i = 0; i < (int)blockDim.x / 32; ++i) sq += red[i];
  const float r = 1.0f / sqrtf(sq / D + p.eps);
  T* o = h + t * p.ldh;
  // a thread reads back what it wrote itself
  for (int c = tid * V; c < D; c += step) {
    float n[V];
#pragma unroll
    for (int e = 0; e < V; ++e) n[e] = s_u[c + e] * r * p.w[c + e];
    if constexpr (V == 1) o[c] = from_f32<T>(n[0]);
    else if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>(o + c) = make_float4(n[0], n[1], n[2], n[3]);
    else *reinterpret_cast<uint2*>(o + c) = make_uint2(pack2<T>(n[0], n[1]), pack2<T>(n[2], n[3]));
  }
  for (int c = D + tid; c < p.ldh; c += blockDim.x) o[c] = from_f32<T>(0.f);
}

template <typename T>
int launch_stream_mix_norm(const StreamMixParams& p, const void* add, void* h, long long tokens, bool vec, cudaStream_t st) {
  const int smem = p.D * 4, threads = tokens < 64 && p.D > 1024 ? 1024 : 256;
  auto go = [&](auto kern) {
    if (smem > 40 * 1024) {
      const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
      if (e != cudaSuccess) return 2000 + (int)e;
    }
    kern<<<(unsigned)tokens, threads, smem, st>>>(p, (const T*)add, (T*)h);
    const cudaError_t e = cudaGetLastError();
    return e == cudaSuccess ? 0 : 3000 + (int)e;
  };
  if (vec) {
    if (p.streams <= 2) return go(stream_mix_norm_kernel<T, 2, 4>);
    if (p.streams <= 4) return go(stream_mix_norm_kernel<T, 4, 4>);
    return go(stream_mix_norm_kernel<T, 8, 4>);
  }
  if (p.streams <= 4) return go(stream_mix_norm_kernel<T, 4, 1>);
  return go(stream_mix_norm_kernel<T, 8, 1>);
}

// One CTA per token: x = table[id] / sqrt(mean + eps) * g (g: one number), h = x / sqrt(mean(x^2) + eps) * w.  The weight w
// has w_step 1 (a number per channel) or 0 (one number).  V numbers per thread and access.
template <typename T, int V>
__global__ void __launch_bounds__(256)
    embed_norm_kernel(const long long* __restrict__ ids, const T* __restrict__ table, const float* __restrict__ g, const float* __restrict__ w,
                      int w_step, float* __restrict__ x, T* __restrict__ h, int D, int ldh, int vocab, float eps) {
  __shared__ float red[8];
  const long long t = blockIdx.x, id = ids[t];
  const bool known = id >= 0 && id < vocab;      // an id outside the vocabulary gives a row of zeros
  const T* e = table + (known ? id : 0) * D;
  const int tid = threadIdx.x;
  auto load = [&](int c, float (&v)[V]) {
    if constexpr (V == 1) {
      v[0] = to_f32<T>(e[c]);
    } else if constexpr (sizeof(T) == 4) {
      *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(e + c);
    } else {
      const uint2 q = *reinterpret_cast<const uint2*>(e + c);
      const float2 lo = unpack2<T>(q.x), hi = unpack2<T>(q.y);
      v[0] = lo.x; v[1] = lo.y; v[2] = hi.x; v[3] = hi.y;
    }
  };
  float sq = 0.f;
  for (int c = tid * V; c < D; c += 256 * V) {
    float v[V];
    load(c, v);
#pragma unroll
    for (int i = 0; i < V; ++i) sq += v[i] * v[i];
  }
  sq = warp_sum(sq);
  if ((tid & 31) == 0) red[tid >> 5] = sq;
  __syncthreads();
  sq = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) sq += red[i];
  const float mean = known ? sq / D : 0.f, rx = known ? *g / sqrtf(mean + eps) : 0.f, rh = 1.0f / sqrtf(mean * rx * rx + eps);
  for (int c = tid * V; c < D; c += 256 * V) {
    float v[V], n[V];
    load(c, v);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      v[i] *= rx;
      n[i] = v[i] * rh * w[(c + i) * w_step];
    }
    if constexpr (V == 1) {
      x[t * D + c] = v[0];
      h[t * ldh + c] = from_f32<T>(n[0]);
    } else {
      *reinterpret_cast<float4*>(x + t * D + c) = make_float4(v[0], v[1], v[2], v[3]);
      if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>(h + t * ldh + c) = make_float4(n[0], n[1], n[2], n[3]);
      else *reinterpret_cast<uint2*>(h + t * ldh + c) = make_uint2(pack2<T>(n[0], n[1]), pack2<T>(n[2], n[3]));
    }
  }
  for (int c = D + tid; c < ldh; c += 256) h[t * ldh + c] = from_f32<T>(0.f);
}

// One CTA per token: x <- x + scale * y (channel by channel; kept if `keep`), h = x / sqrt(mean(x^2) + eps) * w, w as above.
// A thread keeps its N pieces of V numbers in registers.
template <typename T, int V, int N>
__global__ void __launch_bounds__(256)
    scaled_add_norm_kernel(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ scale, const float* __restrict__ w,
                           int w_step, T* __restrict__ h, int D, int ldh, float eps, int keep) {
  __shared__ float red[8];
  const long long t = blockIdx.x;
  const int tid = threadIdx.x;
  float v[N][V];
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int c = (i * 256 + tid) * V;
    if (c >= D) continue;
    if constexpr (V == 4) {
      const float4 a = *reinterpret_cast<const float4*>(x + t * D + c), b = *reinterpret_cast<const float4*>(y + t * D + c),
                   s = *reinterpret_cast<const float4*>(scale + c);
      v[i][0] = fmaf(s.x, b.x, a.x); v[i][1] = fmaf(s.y, b.y, a.y); v[i][2] = fmaf(s.z, b.z, a.z); v[i][3] = fmaf(s.w, b.w, a.w);
    } else {
      v[i][0] = fmaf(scale[c], y[t * D + c], x[t * D + c]);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) sq += v[i][e] * v[i][e];
  }
  sq = warp_sum(sq);
  if ((tid & 31) == 0) red[tid >> 5] = sq;
  __syncthreads();
  sq = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) sq += red[i];
  const float r = 1.0f / sqrtf(sq / D + eps);
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int c = (i * 256 + tid) * V;
    if (c >= D) continue;
    float n[V];
#pragma unroll
    for (int e = 0; e < V; ++e) n[e] = v[i][e] * r * w[(c + e) * w_step];
    if constexpr (V == 4) {
      if (keep) *reinterpret_cast<float4*>(x + t * D + c) = make_float4(v[i][0], v[i][1], v[i][2], v[i][3]);
      if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>(h + t * ldh + c) = make_float4(n[0], n[1], n[2], n[3]);
      else *reinterpret_cast<uint2*>(h + t * ldh + c) = make_uint2(pack2<T>(n[0], n[1]), pack2<T>(n[2], n[3]));
    } else {
      if (keep) x[t * D + c] = v[i][0];
      h[t * ldh + c] = from_f32<T>(n[0]);
    }
  }
  for (int c = D + tid; c < ldh; c += 256) h[t * ldh + c] = from_f32<T>(0.f);
}
template <typename T, int V>
int launch_scaled_add_norm(float* x, const float* y, const float* scale, const float* w, int w_step, void* h, long long tokens, int D, int ldh,
                           float eps, int keep, cudaStream_t st) {
  const int pieces = (D + 256 * V - 1) / (256 * V);
  auto go = [&](auto kern) {
    kern<<<(unsigned)tokens, 256, 0, st>>>(x, y, scale, w, w_step, (T*)h, D, ldh, eps, keep);
    const cudaError_t e = cudaGetLastError();
    return e == cudaSuccess ? 0 : 3000 + (int)e;
  };
  if (pieces <= 1) return go(scaled_add_norm_kernel<T, V, 1>);
  if (pieces <= 2) return go(scaled_add_norm_kernel<T, V, 2>);
  if (pieces <= 4) return go(scaled_add_norm_kernel<T, V, 4>);
  if (pieces <= 8) return go(scaled_add_norm_kernel<T, V, 8>);
  if (pieces <= 16) return go(scaled_add_norm_kernel<T, V, 16>);
  return 22;
}

}  // namespace rb

#define RB_BY_DTYPE(CALL)                                       \
  if (dtype == rbh::DT_BF16) { using T = __nv_bfloat16; CALL; } \
  else if (dtype == rbh::DT_F16) { using T = __half; CALL; }    \
  else if (dtype == rbh::DT_F32) { using T = float; CALL; }     \
  else return 20;
#define RB_LAUNCH_STATUS()             \
  cudaError_t e_ = cudaGetLastError(); \
  return e_ == cudaSuccess ? 0 : 3000 + (int)e_

extern "C" {

// x[t, :] = table[ids[t], :] * scale; an id outside the vocabulary gives a row of zeros
int rb_embed_scaled(int dtype, const long long* ids, const void* table, float* x, long long tokens, int D, int vocab,
                    float scale, void* stream) {
  using namespace rb;
  if (tokens <= 0) return 0;
  const bool vec = D % 4 == 0 && ((reinterpret_cast<uintptr_t>(table) | reinterpret_cast<uintptr_t>(x)) & 15) == 0;
  const long long blocks = (tokens * (vec ? D / 4 : D) + 255) / 256;
  const unsigned g = (unsigned)(blocks < 148 * 64 ? blocks : 148 * 64);
  cudaStream_t st = (cudaStream_t)stream;
  if (vec) {
    RB_BY_DTYPE((embed_scaled_kernel<T, 4><<<g, 256, 0, st>>>(ids, (const T*)table, x, tokens, D, vocab, scale)))
  } else {
    RB_BY_DTYPE((embed_scaled_kernel<T, 1><<<g, 256, 0, st>>>(ids, (const T*)table, x, tokens, D, vocab, scale)))
  }
  RB_LAUNCH_STATUS();
}

// y1 = x / sqrt(mean(x^2) + eps) * w1, y2 the same with w2 (both null or both set); x, w1, w2 fp32.
// add (may be null): rows of the type of y1, lda apart; row t of x first gains rows add_rows[t * n_add + ...].
int rb_rms_norm_stream(int dtype, float* x, const float* w1, const float* w2, void* y1, void* y2, long long rows,
                       int D, int ldy, float eps, const void* add, long long lda, const int* add_rows, int n_add, void* stream) {
  using namespace rb;
  if (rows <= 0) return 0;
  if (ldy < D || (w2 == nullptr) != (y2 == nullptr)) return 21;
  if (add && ((reinterpret_cast<uintptr_t>(add) & 15) || lda < D)) return 21;
  if (add) {
    RB_BY_DTYPE((rms_norm_stream_kernel<T, true><<<(unsigned)rows, 256, 0, (cudaStream_t)stream>>>(x, w1, w2, (T*)y1, (T*)y2, D, ldy, eps, (const T*)add, lda, add_rows, n_add)))
  } else {
    RB_BY_DTYPE((rms_norm_stream_kernel<T, false><<<(unsigned)rows, 256, 0, (cudaStream_t)stream>>>(x, w1, w2, (T*)y1, (T*)y2, D, ldy, eps, nullptr, 0, nullptr, 0)))
  }
  RB_LAUNCH_STATUS();
}

// See StreamMixParams.  x, y, weights fp32; h [tokens, ldh] (zero beyond D); add: rows of h's type, lda apart, token t
// gains rows add_rows[t * n_add + ...] on top of y.  At most 8 streams.
int rb_stream_mix_norm(int dtype, const float* x, long long ldx, long long sx, float* xo, const float* y, const float* mix,
                       const float* w_out, const float* w_in, const float* w, void* h, long long tokens, int streams, int D,
                       int ldh, float eps, const void* add, long long lda, const int* add_rows, int n_add, void* stream) {
  using namespace rb;
  if (tokens <= 0) return 0;
  if (streams < 1 || streams > 8 || D > 50000) return 22;
  if (ldh < D || (add && (!y || lda < D)) || (y && (!mix || !w_out))) return 21;
  auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = D % 4 == 0 && ldx % 4 == 0 && sx % 4 == 0 && ldh % 4 == 0 && al(x) && al(xo) && al(y) && al(w) && al(h) &&
                   (!add || (al(add) && lda % 4 == 0));
  const StreamMixParams p{x, ldx, sx, xo, y, mix, w_out, w_in, w, add_rows, lda, streams, D, ldh, add ? n_add : 0, eps};
  RB_BY_DTYPE(return launch_stream_mix_norm<T>(p, add, h, tokens, vec, (cudaStream_t)stream))
}

// See embed_norm_kernel: x fp32 [tokens, D], h [tokens, ldh] of the table's type (zero beyond D).
int rb_embed_norm(int dtype, const long long* ids, const void* table, const float* g, const float* w, int w_step, float* x, void* h,
                  long long tokens, int D, int ldh, int vocab, float eps, void* stream) {
  using namespace rb;
  if (tokens <= 0) return 0;
  if (ldh < D) return 21;
  auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = D % 4 == 0 && ldh % 4 == 0 && al(table) && al(x) && al(h);
  cudaStream_t st = (cudaStream_t)stream;
  if (vec) {
    RB_BY_DTYPE((embed_norm_kernel<T, 4><<<(unsigned)tokens, 256, 0, st>>>(ids, (const T*)table, g, w, w_step, x, (T*)h, D, ldh, vocab, eps)))
  } else {
    RB_BY_DTYPE((embed_norm_kernel<T, 1><<<(unsigned)tokens, 256, 0, st>>>(ids, (const T*)table, g, w, w_step, x, (T*)h, D, ldh, vocab, eps)))
  }
  RB_LAUNCH_STATUS();
}

// See scaled_add_norm_kernel: x, y fp32 [tokens, D], h [tokens, ldh] of type dtype (zero beyond D).  D: up to 16384 (4096 if odd).
int rb_scaled_add_norm(int dtype, float* x, const float* y, const float* scale, const float* w, int w_step, void* h, long long tokens, int D,
                       int ldh, float eps, int keep, void* stream) {
  using namespace rb;
  if (tokens <= 0) return 0;
  if (ldh < D) return 21;
  auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = D % 4 == 0 && ldh % 4 == 0 && al(x) && al(y) && al(scale) && al(h);
  cudaStream_t st = (cudaStream_t)stream;
  if (vec) {
    RB_BY_DTYPE(return (launch_scaled_add_norm<T, 4>(x, y, scale, w, w_step, h, tokens, D, ldh, eps, keep, st)))
  } else {
    RB_BY_DTYPE(return (launch_scaled_add_norm<T, 1>(x, y, scale, w, w_step, h, tokens, D, ldh, eps, keep, st)))
  }
}
}
