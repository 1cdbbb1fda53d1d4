// Gated delta rule over prompt portions, sm_100a, 16-bit activations: chunks of 64 tokens instead of a loop over tokens.
//
// S <- diag(g_t) S, u_t = beta_t (v_t - S^T k_t), S <- S + k_t u_t^T, o_t = S^T q_t.  With products of decays inside a chunk,
// G(t, j) = g_(j+1) ... g_t per key channel, and S_0 what the chunk starts from,
//
//   u_t + beta_t sum over j < t of (k_t . G(t, j) k_j) u_j = beta_t (v_t - S_0^T (G(t, 0) k_t))
//
// is a unit lower triangular system (I + L) U = diag(beta) (V - K' S_0), so U = U_0 - W S_0 with U_0 = T V, W = T K',
// T = (I + L)^-1 diag(beta); then O = Q' S_0 + A U with A(t, j) = q_t . G(t, j) k_j for j <= t, and the state at the end is
// G(end, 0) S_0 + K''^T U with K''_j = G(end, j) k_j.
//
//   local    per chunk and head: convolutions, unit lengths, decays; L, A, T; W, U_0, K'', Q'
//   scan     per portion, head and 16 columns of the state: U and the next state, chunk by chunk
//   outputs  per chunk and head: O, output norm and gate
//
// No decay is ever divided by: within 16 neighbouring tokens G(t, j) grows factor by factor along t, and between groups of
// 16 it is (from the end of j's group to the start of t's group) times one part on either side, all at most one.
//
// Where a head's channels decay together (HEAD), G(t, j) is a number, 2^(c_t - c_j) with c the running sum of the logarithms, at
// most one again, and it comes out of the products over channels: the pairs of tokens are one product K K^T and one Q K^T.
// Convolved queries and keys are then 16-bit numbers whose unit lengths are a factor per token, so those products are exact.
//
// Values are 16-bit, everything else is fp32 and goes into tensor products as pairs of 16-bit numbers (see SplitPair), three
// products each (two where the other side is 16-bit).  The outputs run on tcgen05; the products before them are warp-level:
// small, with operands made in registers (local), or one behind the other with a change of form in between (scan).
#include "recurrent.cuh"
#include "warp_mma.cuh"

namespace rb {

constexpr int kDeltaCols = 16;
using bf16 = __nv_bfloat16;

struct DeltaChunkParams {
  const bf16* raw;               // row: kv_heads x dim_p queries, keys, heads x vdim_p values, before their convolutions
  long long ldr;
  const float* taps_w;           // [taps][channels]
  bf16* conv;                    // [places, heads, taps - 1, 2 dim_p + vdim_p]
  const float *a, *dt, *decay;   // steps as in DeltaRowsParams (row 0 = first row of the batch), [heads]
  long long lda;
  int per_head;
  const float* b;                // [tokens, ldb]
  long long ldb;
  int* status;
  const int4* items;             // chunks: {first row, tokens, portion}
  const int4* seqs;              // portions
  const int* first;              // [portions + 1] first chunk
  float* S;                      // [places, heads, dim_p, vdim_p]
  // by chunk and head, two planes each (high and low parts), as they lie in shared memory (tile_at), so that one bulk copy
  // brings them there; D: dim_p rounded up to 64
  uint8_t* wk;                   // W, K'': 4 planes [64][D]
  // operands of tcgen05: rows of 64 numbers (128 bytes, swizzled)
  uint8_t* qa;                   // Q' per 64 key numbers, then A: 128 rows, the high parts of 64 tokens and their low parts
  uint8_t* su;                   // per plane and 64 columns: S_0, D rows; then the same of U, 64 rows
  float *u0, *end;               // [64][vdim_p], [D]: G(end, 0)
  int heads, kv_heads, dim_p, vdim_p, vdim, taps, channels;
  float q_scale;
  RecOut<bf16> o;
};

// ---------------------------------------------------------------------------------------------------------
// local
// ---------------------------------------------------------------------------------------------------------
template <int KS, int VS, bool HEAD>      // 64-column sub-tiles of keys and of values; a decay per head
struct DeltaLocalCfg {
  static constexpr int D = KS * 64, LD = D + 4, LT = 68;
  static constexpr int VEC_BYTES = HEAD ? 0 : 64 * LD * 4, TRI_BYTES = 64 * LT * 4, PLANE = 64 * D * 2, V_BYTES = 64 * VS * 128;
  static constexpr int SMEM_BYTES = 3 * VEC_BYTES + (HEAD ? 2 : 3) * TRI_BYTES + 2 * PLANE + V_BYTES + (HEAD ? 0 : 4 * D * 4) + 128;
};

__device__ __forceinline__ float dot4(float4 a, float4 b, float s) {
  return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, s))));
}
// the exponential, unlike the hardware tanh, keeps small results exact to fp32 rounding
__device__ __forceinline__ float sigmoid_quick(float z) { return __fdividef(1.0f, 1.0f + __expf(-z)); }
__device__ __forceinline__ float4 mul4(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }

template <int KS, int VS, bool HEAD>
__global__ void __launch_bounds__(512, HEAD ? 2 : 1) delta_chunk_local_kernel(const DeltaChunkParams p) {
  using C = DeltaLocalCfg<KS, VS, HEAD>;
  constexpr int D = C::D, LD = C::LD, LT = C::LT;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 127) & ~static_cast<uintptr_t>(127));
  uint8_t* s_kb = smem;                                     // K' planes; HEAD: convolved keys, then queries
  uint8_t* s_v = s_kb + 2 * C::PLANE;
  float* s_k = reinterpret_cast<float*>(s_v + C::V_BYTES);  // keys, later times their decays since their group's start
  float* s_q = s_k + 64 * LD;                               // queries, the same
  float* s_g = s_q + 64 * LD;                               // decays, later keys times what decays up to their group's end
  float* s_L = HEAD ? s_k : s_g + 64 * LD;
  float* s_T = s_L + 64 * LT;
  float* s_A = s_T + 64 * LT;
  float* s_P = s_A + 64 * LT;                               // [4][D] a group's product of decays
  __shared__ float s_beta[64], s_M[3][16][17];
  // HEAD, per token: running sum of the logarithms of decays, factors of the convolved query and key, of the key in W
  __shared__ float s_c[HEAD ? 64 : 1], s_rq[HEAD ? 64 : 1], s_rk[HEAD ? 64 : 1], s_w[HEAD ? 64 : 1];
  const int4 it = p.items[blockIdx.x];
  const int4 seq = p.seqs[it.z];
  const int h = blockIdx.y, kh = h / (p.heads / p.kv_heads), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const long long ch = (long long)blockIdx.x * p.heads + h;
  const int channels = 2 * p.dim_p + p.vdim_p, past = p.taps - 1;      // inputs that a head keeps

  // ---- a warp brings four tokens, a lane four numbers of each vector
  {
    const bf16* conv = p.conv + (((long long)seq.z * p.heads + h) * past) * channels;
    const int c4 = lane * 4, t0 = warp * 4, off0 = it.x + t0 - seq.x;
    const bool kd = c4 < p.dim_p, vd = c4 < p.vdim_p;
    float4 x[4], step[4];
    const float* wp = p.taps_w + c4;
    const bf16* src = p.raw + (long long)(it.x + t0) * p.ldr + c4;
    const int cq = kh * p.dim_p, ck = (p.kv_heads + kh) * p.dim_p, cv = 2 * p.kv_heads * p.dim_p + h * p.vdim_p;
    auto input = [&](int i, int ch0, int own) {      // channels of token t0 + i; zeros before the sequence and past the chunk
      if (t0 + i >= it.y) return make_uint2(0, 0);
      if (off0 + i >= 0) return *reinterpret_cast<const uint2*>(src + i * p.ldr + ch0);
      return seq.w > 0 ? *reinterpret_cast<const uint2*>(conv + (long long)(past + off0 + i) * channels + own + c4) : make_uint2(0, 0);
    };
    auto add = [&](float4& o, float4 w, uint2 in2) {
      const float2 lo = unpack2<bf16>(in2.x), hi = unpack2<bf16>(in2.y);
      o.x = fmaf(w.x, lo.x, o.x); o.y = fmaf(w.y, lo.y, o.y); o.z = fmaf(w.z, hi.x, o.z); o.w = fmaf(w.w, hi.y, o.w);
    };
    auto activate = [&]() {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        if (t0 + i >= it.y) x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        x[i].x *= sigmoid_quick(x[i].x); x[i].y *= sigmoid_quick(x[i].y); x[i].z *= sigmoid_quick(x[i].z); x[i].w *= sigmoid_quick(x[i].w);
      }
    };
    // four taps, the usual number: inputs come ahead of their use
    auto convolved4 = [&](const uint2 (&in)[7], int ch0, bool live) {
#pragma unroll
      for (int i = 0; i < 4; ++i) x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!live) return;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float4 w = *reinterpret_cast<const float4*>(wp + (long long)j * p.channels + ch0);
#pragma unroll
        for (int i = 0; i < 4; ++i) add(x[i], w, in[i + j]);
      }
      activate();
    };
    auto convolved = [&](int ch0, int own, bool live) {
#pragma unroll
      for (int i = 0; i < 4; ++i) x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!live) return;
      for (int j = 0; j < p.taps; ++j) {
        const float4 w = *reinterpret_cast<const float4*>(wp + (long long)j * p.channels + ch0);
#pragma unroll
        for (int i = 0; i < 4; ++i) add(x[i], w, input(i + j - past, ch0, own));
      }
      activate();
    };
    auto unit = [&](float* dst, uint8_t* plane, float* factor, float scale) {
      float n[4];
      if constexpr (HEAD) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const uint2 v = make_uint2(pack2<bf16>(x[i].x, x[i].y), pack2<bf16>(x[i].z, x[i].w));
          if (c4 < D) *reinterpret_cast<uint2*>(plane + tile_at<KS * 8>(t0 + i, c4 >> 3) + (c4 & 4) * 2) = v;
          const float2 lo = unpack2<bf16>(v.x), hi = unpack2<bf16>(v.y);
          x[i] = make_float4(lo.x, lo.y, hi.x, hi.y);
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) n[i] = dot4(x[i], x[i], 0.f);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1)
#pragma unroll
        for (int i = 0; i < 4; ++i) n[i] += __shfl_xor_sync(0xffffffffu, n[i], o);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float f = scale / sqrtf(n[i] + 1e-6f);
        if constexpr (HEAD) {
          if (lane == 0) factor[t0 + i] = f;
        } else if (c4 < D) *reinterpret_cast<float4*>(dst + (t0 + i) * LD + c4) = make_float4(x[i].x * f, x[i].y * f, x[i].z * f, x[i].w * f);
      }
    };
    auto values = [&]() {
      if (c4 >= VS * 64) return;
#pragma unroll
      for (int i = 0; i < 4; ++i)
        *reinterpret_cast<uint2*>(s_v + tile_at<VS * 8>(t0 + i, c4 >> 3) + (c4 & 4) * 2) =
            make_uint2(pack2<bf16>(x[i].x, x[i].y), pack2<bf16>(x[i].z, x[i].w));
    };
    auto steps = [&]() {
      if constexpr (HEAD) return;
#pragma unroll
      for (int i = 0; i < 4; ++i)
        step[i] = kd && t0 + i < it.y ? *reinterpret_cast<const float4*>(p.a + (long long)(it.x + t0 + i) * p.lda + h * p.dim_p + c4)
                                      : make_float4(0.f, 0.f, 0.f, 0.f);
    };
    if (p.taps == 4) {
      uint2 iq[7], ik[7], iv[7];
#pragma unroll
      for (int i = 0; i < 7; ++i) {
        iq[i] = kd ? input(i - 3, cq, 0) : make_uint2(0, 0);
        ik[i] = kd ? input(i - 3, ck, p.dim_p) : make_uint2(0, 0);
        iv[i] = vd ? input(i - 3, cv, 2 * p.dim_p) : make_uint2(0, 0);
      }
      steps();
      convolved4(iq, cq, kd);
      unit(s_q, s_kb + C::PLANE, s_rq, p.q_scale);
      convolved4(ik, ck, kd);
      unit(s_k, s_kb, s_rk, 1.0f);
      convolved4(iv, cv, vd);
      values();
    } else {
      steps();
      convolved(cq, 0, kd);
      unit(s_q, s_kb + C::PLANE, s_rq, p.q_scale);
      convolved(ck, p.dim_p, kd);
      unit(s_k, s_kb, s_rk, 1.0f);
      convolved(cv, 2 * p.dim_p, vd);
      values();
    }
    if constexpr (!HEAD) {
      if (c4 < D) {
        const float4 d = kd ? *reinterpret_cast<const float4*>(p.dt + h * p.dim_p + c4) : make_float4(0.f, 0.f, 0.f, 0.f);
        const float f = -p.decay[h] * 1.4426950408889634f;
        // e^(-decay log(1 + e^z)), the logarithm in base two both ways
        auto one = [&](float z) { return fast_exp2(f * (fmaxf(z, 0.f) + 0.6931471805599453f * __log2f(1.0f + __expf(-fabsf(z))))); };
#pragma unroll
        for (int i = 0; i < 4; ++i)
          *reinterpret_cast<float4*>(s_g + (t0 + i) * LD + c4) =
              kd && t0 + i < it.y ? make_float4(one(step[i].x + d.x), one(step[i].y + d.y), one(step[i].z + d.z), one(step[i].w + d.w))
                                  : make_float4(1.f, 1.f, 1.f, 1.f);
      }
    }
    if (lane < 4)
      s_beta[t0 + lane] = t0 + lane < it.y ? 1.0f / (1.0f + expf(-p.b[(long long)(it.x + t0 + lane) * p.ldb + h])) : 0.f;
    if constexpr (HEAD) {
      if (lane < 4)
        s_c[t0 + lane] = t0 + lane < it.y ? -1.4426950408889634f * p.decay[h] *
                                                softplus_f(p.a[(long long)(it.x + t0 + lane) * p.lda + h] + p.dt[h]) : 0.f;
      for (int i = tid; i < 64 * LT; i += 512) s_T[i] = 0.f;
    } else {
      for (int i = tid; i < 64 * LT; i += 512) s_A[i] = 0.f;
    }
  }
  __syncthreads();
  const int r = lane >> 2, c2 = (lane & 3) * 2;
  uint8_t *wk = p.wk + ch * 4 * C::PLANE, *qa = p.qa + ch * (2 * C::PLANE + 2 * 64 * 128);
  // 16-byte chunk c of token t's high (0) or low (1) parts among 128 rows of 64 numbers
  auto stacked = [](int plane, int t, int c) { return (c >> 3) * (128 * 128) + (plane * 64 + t) * 128 + (((c & 7) ^ (t & 7)) << 4); };
  auto split4 = [](float4 v, uint2& hi, uint2& lo) {
    const SplitPair a = split2(v.x, v.y), b = split2(v.z, v.w);
    hi = make_uint2(a.hi, b.hi);
    lo = make_uint2(a.lo, b.lo);
  };

  if constexpr (HEAD) {
    // ---- running sums; then pairs: a warp has 16 later tokens, 32 earlier ones, and keys or queries of the later ones
    if (warp == 0) {
      const float a = s_c[2 * lane], b = a + s_c[2 * lane + 1];
      float sum = b;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += up;
      }
      const float c0 = sum - b + a;
      s_c[2 * lane] = c0;
      s_c[2 * lane + 1] = sum;
      s_w[2 * lane] = s_beta[2 * lane] * s_rk[2 * lane] * fast_exp2(c0);
      s_w[2 * lane + 1] = s_beta[2 * lane + 1] * s_rk[2 * lane + 1] * fast_exp2(sum);
    }
    const int mt = warp & 3, query = (warp >> 2) & 1, half = warp >> 3;
    float acc[4][4];
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[n][e] = 0.f;
    if (half == 0 || mt >= 2) {
      const uint32_t left = smem_u32(s_kb) + query * C::PLANE, right = smem_u32(s_kb);
      const int lr = mt * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), rr = half * 32 + (lane >> 4) * 8 + (lane & 7);
#pragma unroll
      for (int ks = 0; ks < KS * 4; ++ks) {
        uint32_t x[4], y[4];
        ldmatrix_x4(left + tile_at<KS * 8>(lr, ks * 2 + (lane >> 4)), x);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          ldmatrix_x4(right + tile_at<KS * 8>(rr + n * 16, ks * 2 + ((lane >> 3) & 1)), y);
          mma_bf16(acc[2 * n], x, y[0], y[1]);
          mma_bf16(acc[2 * n + 1], x, y[2], y[3]);
        }
      }
    }
    __syncthreads();
    {
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int t = mt * 16 + r + 8 * x;
        const float ct = s_c[t], f = query ? s_rq[t] : s_rk[t] * s_beta[t];
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          const int j = half * 32 + n * 8 + c2;
          float v[2];
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const bool see = query ? j + e <= t : j + e < t;
            v[e] = see ? acc[n][2 * x + e] * f * s_rk[j + e] * fast_exp2(ct - s_c[j + e]) : 0.f;
          }
          if (query) {
            const SplitPair a = split2(v[0], v[1]);
            *reinterpret_cast<uint32_t*>(qa + 2 * C::PLANE + stacked(0, t, j >> 3) + (j & 7) * 2) = a.hi;
            *reinterpret_cast<uint32_t*>(qa + 2 * C::PLANE + stacked(1, t, j >> 3) + (j & 7) * 2) = a.lo;
          } else {
            *reinterpret_cast<float2*>(s_L + t * LT + j) = make_float2(v[0], v[1]);
          }
        }
      }
    }
    __syncthreads();
  } else {

    // ---- pairs inside a group of 16: a thread takes keys jj and 15 - jj, together 15 later tokens, and a few channels
    {
      const int grp = warp >> 2, jj = lane & 7, dg = (warp & 3) * 4 + (lane >> 3);
      float aL[15], aA[15], aD[2] = {0.f, 0.f};
#pragma unroll
      for (int s = 0; s < 15; ++s) aL[s] = aA[s] = 0.f;
      const float *gk = s_k + grp * 16 * LD, *gq = s_q + grp * 16 * LD, *gg = s_g + grp * 16 * LD;
#pragma unroll
      for (int x = 0; x < KS; ++x) {
        const int c = x * 64 + dg * 4;
        float4 pr = *reinterpret_cast<const float4*>(gk + jj * LD + c);
        const float4 k2 = *reinterpret_cast<const float4*>(gk + (15 - jj) * LD + c);
        aD[0] = dot4(pr, *reinterpret_cast<const float4*>(gq + jj * LD + c), aD[0]);
        aD[1] = dot4(k2, *reinterpret_cast<const float4*>(gq + (15 - jj) * LD + c), aD[1]);
#pragma unroll
        for (int s = 1; s <= 15; ++s) {
          if (s == 16 - jj) pr = k2;
          const int t = s <= 15 - jj ? jj + s : s;
          pr = mul4(pr, *reinterpret_cast<const float4*>(gg + t * LD + c));
          aL[s - 1] = dot4(pr, *reinterpret_cast<const float4*>(gk + t * LD + c), aL[s - 1]);
          aA[s - 1] = dot4(pr, *reinterpret_cast<const float4*>(gq + t * LD + c), aA[s - 1]);
        }
      }
      float* part = s_T + ((warp & 3) * 32 + grp * 8 + jj) * 33;      // [4 quarters][group, jj][32]
      auto put = [&](float v, int i) {
        v += __shfl_xor_sync(0xffffffffu, v, 8);
        v += __shfl_xor_sync(0xffffffffu, v, 16);
        if (lane < 8) part[i] = v;
      };
#pragma unroll
      for (int s = 0; s < 15; ++s) {
        put(aL[s], s);
        put(aA[s], 15 + s);
      }
      put(aD[0], 30);
      put(aD[1], 31);
    }
    __syncthreads();
    for (int i = tid; i < 1024; i += 512) {
      const int gj = i >> 5, e = i & 31, jj = gj & 7, base = (gj >> 3) * 16;
      float v = 0.f;
#pragma unroll
      for (int w = 0; w < 4; ++w) v += s_T[(w * 32 + gj) * 33 + e];
      if (e >= 30) {
        const int j = base + (e == 30 ? jj : 15 - jj);
        s_A[j * LT + j] = v;
      } else {
        const int s = e % 15 + 1;
        const bool lo = s <= 15 - jj;
        const int t = base + (lo ? jj + s : s), j = base + (lo ? jj : 15 - jj);
        if (e < 15) s_L[t * LT + j] = v * s_beta[t];
        else s_A[t * LT + j] = v;
      }
    }

    // ---- decays since the group's start and up to its end, channel by channel
    if (tid < 4 * D) {
      const int d = tid % D, base = tid / D * 16;
      float g[16], k[16], e = 1.f;
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        g[i] = s_g[(base + i) * LD + d];
        k[i] = s_k[(base + i) * LD + d];
        e *= g[i];
        s_k[(base + i) * LD + d] = k[i] * e;
        s_q[(base + i) * LD + d] *= e;
      }
      s_P[tid] = e;
      e = 1.f;
#pragma unroll
      for (int i = 15; i >= 0; --i) {
        s_g[(base + i) * LD + d] = k[i] * e;
        e *= g[i];
      }
    }
    __syncthreads();
    for (int i = tid; i < 64 * LT; i += 512) s_T[i] = 0.f;
    if (warp < 6) {
      // ---- pairs between groups: warp = (later group, earlier group)
      const int b = warp < 1 ? 1 : warp < 3 ? 2 : 3, a = warp - (b == 1 ? 0 : b == 2 ? 1 : 3);
      float accL[2][4], accA[2][4];
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) accL[n][e] = accA[n][e] = 0.f;
#pragma unroll 1
      for (int ks = 0; ks < D / 16; ++ks) {
        uint32_t kh_[4], kl[4], qh[4], ql[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int at = (b * 16 + r + (e & 1) * 8) * LD + ks * 16 + (e >> 1) * 8 + c2;
          const float2 kv = *reinterpret_cast<const float2*>(s_k + at), qv = *reinterpret_cast<const float2*>(s_q + at);
          const SplitPair sk = split2(kv.x, kv.y), sq = split2(qv.x, qv.y);
          kh_[e] = sk.hi; kl[e] = sk.lo; qh[e] = sq.hi; ql[e] = sq.lo;
        }
        float2 f[2] = {make_float2(1.f, 1.f), make_float2(1.f, 1.f)};      // whole groups in between
        for (int m = a + 1; m < b; ++m)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const float2 x = *reinterpret_cast<const float2*>(s_P + m * D + ks * 16 + e * 8 + c2);
            f[e].x *= x.x;
            f[e].y *= x.y;
          }
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          SplitPair x[2];
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const float2 v = *reinterpret_cast<const float2*>(s_g + (a * 16 + n * 8 + r) * LD + ks * 16 + e * 8 + c2);
            x[e] = split2(v.x * f[e].x, v.y * f[e].y);
          }
          mma_bf16(accL[n], kh_, x[0].hi, x[1].hi);
          mma_bf16(accL[n], kh_, x[0].lo, x[1].lo);
          mma_bf16(accL[n], kl, x[0].hi, x[1].hi);
          mma_bf16(accA[n], qh, x[0].hi, x[1].hi);
          mma_bf16(accA[n], qh, x[0].lo, x[1].lo);
          mma_bf16(accA[n], ql, x[0].hi, x[1].hi);
        }
      }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int t = b * 16 + r + (e >> 1) * 8, j = a * 16 + n * 8 + c2 + (e & 1);
          s_L[t * LT + j] = accL[n][e] * s_beta[t];
          s_A[t * LT + j] = accA[n][e];
        }
    } else {
      // ---- what leaves with the decays since the chunk's start (queries, keys of the system) or up to its end (keys)
      const int c4 = lane * 4;
      if (c4 < D) {
        float4 P[4];
#pragma unroll
        for (int m = 0; m < 4; ++m) P[m] = *reinterpret_cast<const float4*>(s_P + m * D + c4);
        for (int t = warp - 6; t < 64; t += 10) {
          const int grp = t >> 4;
          float4 before = make_float4(1.f, 1.f, 1.f, 1.f), after = before;
#pragma unroll
          for (int m = 0; m < 4; ++m) {
            if (m < grp) before = mul4(before, P[m]);
            if (m > grp) after = mul4(after, P[m]);
          }
          uint2 hi, lo;
          split4(mul4(*reinterpret_cast<const float4*>(s_k + t * LD + c4), before), hi, lo);
          const uint32_t at = tile_at<KS * 8>(t, c4 >> 3) + (c4 & 4) * 2;
          *reinterpret_cast<uint2*>(s_kb + at) = hi;
          *reinterpret_cast<uint2*>(s_kb + C::PLANE + at) = lo;
          split4(mul4(*reinterpret_cast<const float4*>(s_q + t * LD + c4), before), hi, lo);
          *reinterpret_cast<uint2*>(qa + stacked(0, t, c4 >> 3) + (c4 & 4) * 2) = hi;
          *reinterpret_cast<uint2*>(qa + stacked(1, t, c4 >> 3) + (c4 & 4) * 2) = lo;
          split4(mul4(*reinterpret_cast<const float4*>(s_g + t * LD + c4), after), hi, lo);
          *reinterpret_cast<uint2*>(wk + 2 * C::PLANE + at) = hi;
          *reinterpret_cast<uint2*>(wk + 3 * C::PLANE + at) = lo;
        }
        if (warp == 6) *reinterpret_cast<float4*>(p.end + ch * D + c4) = mul4(mul4(P[0], P[1]), mul4(P[2], P[3]));
      }
    }
    __syncthreads();
  }

  // ---- inverse of I + L: groups of 16 by substitution (one column per thread), then the blocks below them
  if (warp < 2) {
    const int base = tid >> 4 << 4, cc = tid & 15;
    float x[16];
#pragma unroll
    for (int t = 0; t < 16; ++t) x[t] = t == cc ? 1.f : 0.f;
#pragma unroll
    for (int j = 0; j < 15; ++j)               // column by column: a new x goes into all later sums
#pragma unroll
      for (int t = j + 1; t < 16; ++t) x[t] = fmaf(-s_L[(base + t) * LT + base + j], x[j], x[t]);
#pragma unroll
    for (int t = 0; t < 16; ++t) s_T[(base + t) * LT + base + cc] = x[t];
  } else if constexpr (HEAD) {
    // what leaves with the decays since the chunk's start (queries) or up to its end (keys)
    const int c4 = lane * 4;
    if (c4 < D) {
      const float last = s_c[63];
      for (int t = warp - 2; t < 64; t += 14) {
        const uint32_t at = tile_at<KS * 8>(t, c4 >> 3) + (c4 & 4) * 2;
        auto scaled = [&](const uint8_t* plane, float f) {
          const uint2 v = *reinterpret_cast<const uint2*>(plane + at);
          const float2 lo = unpack2<bf16>(v.x), hi = unpack2<bf16>(v.y);
          return make_float4(lo.x * f, lo.y * f, hi.x * f, hi.y * f);
        };
        uint2 hi, lo;
        split4(scaled(s_kb + C::PLANE, s_rq[t] * fast_exp2(s_c[t])), hi, lo);
        *reinterpret_cast<uint2*>(qa + stacked(0, t, c4 >> 3) + (c4 & 4) * 2) = hi;
        *reinterpret_cast<uint2*>(qa + stacked(1, t, c4 >> 3) + (c4 & 4) * 2) = lo;
        split4(scaled(s_kb, s_rk[t] * fast_exp2(last - s_c[t])), hi, lo);
        *reinterpret_cast<uint2*>(wk + 2 * C::PLANE + at) = hi;
        *reinterpret_cast<uint2*>(wk + 3 * C::PLANE + at) = lo;
      }
      const float e = fast_exp2(last);
      if (warp == 2) *reinterpret_cast<float4*>(p.end + ch * D + c4) = make_float4(e, e, e, e);
    }
  } else {
    for (int i = tid - 64; i < 64 * 16; i += 448) {         // A in planes, four numbers at a time
      const int t = i >> 4, c = (i & 15) * 4;
      const float4 v = *reinterpret_cast<const float4*>(s_A + t * LT + c);
      const SplitPair x = split2(v.x, v.y), y = split2(v.z, v.w);
      *reinterpret_cast<uint2*>(qa + 2 * C::PLANE + stacked(0, t, c >> 3) + (c & 4) * 2) = make_uint2(x.hi, y.hi);
      *reinterpret_cast<uint2*>(qa + 2 * C::PLANE + stacked(1, t, c >> 3) + (c & 4) * 2) = make_uint2(x.lo, y.lo);
    }
  }
  __syncthreads();
  // T_ba = -T_bb (sum over a <= m < b of L_bm T_ma): a warp takes 8 columns of a block
#pragma unroll 1
  for (int dist = 1; dist < 4; ++dist) {
    if (warp < 2 * (4 - dist)) {
      const int a = warp >> 1, b = a + dist, col = a * 16 + (warp & 1) * 8;
      float* m = &s_M[a][0][0] + (warp & 1) * 8;
      // c += L or T rows 16 b .., columns k .. k + 16, times the 16 x 8 numbers at x (row stride ld)
      auto product = [&](const float* left, int k, const float* x, int ld, float (&c)[3][4]) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 v = *reinterpret_cast<const float2*>(left + (b * 16 + r + (e & 1) * 8) * LT + k + (e >> 1) * 8 + c2);
          const SplitPair s = split2(v.x, v.y);
          hi[e] = s.hi;
          lo[e] = s.lo;
        }
        const SplitPair x0 = split2(x[c2 * ld + r], x[(c2 + 1) * ld + r]), x1 = split2(x[(c2 + 8) * ld + r], x[(c2 + 9) * ld + r]);
        mma_bf16(c[0], hi, x0.hi, x1.hi);
        mma_bf16(c[1], lo, x0.hi, x1.hi);
        mma_bf16(c[2], hi, x0.lo, x1.lo);
      };
      float c[3][4] = {};
      for (int k = a; k < b; ++k) product(s_L, k * 16, s_T + k * 16 * LT + col, LT, c);
#pragma unroll
      for (int e = 0; e < 4; ++e) m[(r + (e >> 1) * 8) * 17 + c2 + (e & 1)] = c[0][e] + (c[1][e] + c[2][e]);
      __syncwarp();
      float d[3][4] = {};
      product(s_T, b * 16, m, 17, d);
#pragma unroll
      for (int e = 0; e < 4; ++e) s_T[(b * 16 + r + (e >> 1) * 8) * LT + col + c2 + (e & 1)] = -(d[0][e] + (d[1][e] + d[2][e]));
    }
    __syncthreads();
  }

  // ---- W = T K', U_0 = T V
  {
    constexpr int NK = KS * 2, NV = VS * 2;                  // 8-column tiles per warp (a quarter of the columns)
    const int mt = warp & 3, cg = warp >> 2;
    float aw[NK][4], au[NV][4];
#pragma unroll
    for (int n = 0; n < NK; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) aw[n][e] = 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) au[n][e] = 0.f;
    const uint32_t kb = smem_u32(s_kb), vb = smem_u32(s_v);
#pragma unroll 1
    for (int ks = 0; ks <= mt; ++ks) {
      uint32_t hi[4], lo[4], wh[4], wl[4];       // times write strengths; HEAD: for W also times the keys' factors
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = mt * 16 + r + (e & 1) * 8, j = ks * 16 + (e >> 1) * 8 + c2;
        const float2 v = *reinterpret_cast<const float2*>(s_T + t * LT + j);
        const SplitPair s = split2(v.x * s_beta[j], v.y * s_beta[j + 1]);
        hi[e] = s.hi;
        lo[e] = s.lo;
        if constexpr (HEAD) {
          const SplitPair w = split2(v.x * s_w[j], v.y * s_w[j + 1]);
          wh[e] = w.hi;
          wl[e] = w.lo;
        } else {
          wh[e] = s.hi;
          wl[e] = s.lo;
        }
      }
      const int row = ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7);
#pragma unroll
      for (int n = 0; n < NK / 2; ++n) {
        const uint32_t at = kb + tile_at<KS * 8>(row, cg * NK + 2 * n + (lane >> 4));
        uint32_t x[4];
        ldmatrix_x4_trans(at, x);
        mma_bf16(aw[2 * n], wh, x[0], x[1]);
        mma_bf16(aw[2 * n + 1], wh, x[2], x[3]);
        mma_bf16(aw[2 * n], wl, x[0], x[1]);
        mma_bf16(aw[2 * n + 1], wl, x[2], x[3]);
        if constexpr (!HEAD) {
          ldmatrix_x4_trans(at + C::PLANE, x);
          mma_bf16(aw[2 * n], wh, x[0], x[1]);
          mma_bf16(aw[2 * n + 1], wh, x[2], x[3]);
        }
      }
#pragma unroll
      for (int n = 0; n < NV / 2; ++n) {
        uint32_t x[4];
        ldmatrix_x4_trans(vb + tile_at<VS * 8>(row, cg * NV + 2 * n + (lane >> 4)), x);
        mma_bf16(au[2 * n], hi, x[0], x[1]);
        mma_bf16(au[2 * n + 1], hi, x[2], x[3]);
        mma_bf16(au[2 * n], lo, x[0], x[1]);
        mma_bf16(au[2 * n + 1], lo, x[2], x[3]);
      }
    }
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int t = mt * 16 + r + 8 * x;
#pragma unroll
      for (int n = 0; n < NK; ++n) {
        const int c = (cg * NK + n) * 8 + c2;
        const SplitPair s = split2(aw[n][2 * x], aw[n][2 * x + 1]);
        const uint32_t at = tile_at<KS * 8>(t, c >> 3) + (c & 7) * 2;
        *reinterpret_cast<uint32_t*>(wk + at) = s.hi;
        *reinterpret_cast<uint32_t*>(wk + C::PLANE + at) = s.lo;
      }
#pragma unroll
      for (int n = 0; n < NV; ++n) {
        const int c = (cg * NV + n) * 8 + c2;
        if (c < p.vdim_p) *reinterpret_cast<float2*>(p.u0 + (ch * 64 + t) * p.vdim_p + c) = make_float2(au[n][2 * x], au[n][2 * x + 1]);
      }
    }
  }
}

// ---------------------------------------------------------------------------------------------------------
// scan: a CTA has 16 columns of one head's state, in registers (16 rows a warp) and, as planes, in shared memory.  It is
// bound by the length of a chunk's chain of products, so a product's three parts run in accumulators of their own, and
// its operands come a chunk ahead by bulk copies.  When there are more heads and columns than SMs, two groups of eight
// warps, 16 columns each, share the operands.
// ---------------------------------------------------------------------------------------------------------
template <int KS, int GROUPS>
struct DeltaScanCfg {
  static constexpr int D = KS * 64, PLANE = 64 * D * 2, STAGE = 4 * PLANE;           // W and K'', two planes each
  static constexpr int S_PLANE = D * 32, U_PLANE = 64 * 32, BLOCK = 2 * (S_PLANE + U_PLANE);
  static constexpr int SMEM_BYTES = 2 * STAGE + GROUPS * BLOCK + 128;
};

template <int KS, int GROUPS>
__global__ void __launch_bounds__(256 * GROUPS, 1) delta_chunk_scan_kernel(const DeltaChunkParams p, int* status) {
  using C = DeltaScanCfg<KS, GROUPS>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 127) & ~static_cast<uintptr_t>(127));
  __shared__ uint64_t full[2];
  __shared__ int s_abort;
  const int grp = GROUPS == 1 ? 0 : threadIdx.x >> 8, tid = threadIdx.x & 255, warp = tid >> 5, lane = tid & 31;
  uint8_t *s_s = smem + 2 * C::STAGE + grp * C::BLOCK, *s_u = s_s + 2 * C::S_PLANE;
  const uint32_t ring = smem_u32(smem), ss = smem_u32(s_s), su = smem_u32(s_u);
  const int blocks = (p.vdim_p + kDeltaCols - 1) / kDeltaCols, wide = (p.vdim_p + 63) / 64, cb = blockIdx.x * GROUPS + grp, col0 = cb * kDeltaCols, h = blockIdx.y;
  const bool mine = cb < blocks;                             // the last CTA's second group may have nothing to do
  const int r = lane >> 2, c2 = (lane & 3) * 2;
  const int4 seq = p.seqs[blockIdx.z];
  const int c0 = p.first[blockIdx.z], c1 = p.first[blockIdx.z + 1];
  const long long size = (long long)p.dim_p * p.vdim_p;
  float* state = p.S + ((long long)seq.z * p.heads + h) * size;
  if (threadIdx.x == 0) {
    mbar_init(smem_u32(&full[0]), 1);
    mbar_init(smem_u32(&full[1]), 1);
    s_abort = 0;
    fence_barrier_init();
  }
  __syncthreads();
  auto bring = [&](int c) {                                  // one thread
    const uint32_t bar = smem_u32(&full[(c - c0) & 1]);
    mbar_arrive_expect_tx(bar, C::STAGE);
    bulk_load_1d(ring + ((c - c0) & 1) * C::STAGE, p.wk + ((long long)c * p.heads + h) * C::STAGE, C::STAGE, bar);
  };
  if (threadIdx.x == 0) bring(c0);
  // rows of the state: warp % (4 KS); both 8-column tiles, or one when there are warps for each
  constexpr int MT = KS * 4, NT = KS == 2 ? 2 : 1;
  const int m0 = warp % MT * 16, n0 = warp / MT * NT;
  float S[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int d = m0 + r + 8 * x, c = col0 + (n0 + n) * 8 + c2;
      const bool live = seq.w != 0 && d < p.dim_p && c < p.vdim_p;
      const float2 v = live ? *reinterpret_cast<const float2*>(state + (long long)d * p.vdim_p + c) : make_float2(0.f, 0.f);
      S[n][2 * x] = v.x;
      S[n][2 * x + 1] = v.y;
    }
  // of chunk c: where 8 columns (tile n of the 16) of row x of S_0's or U's high plane go; the low plane's are `wide` blocks on
  auto state_at = [&](int c, int x, int n) {
    return p.su + ((long long)c * p.heads + h) * (2 * wide * (C::D + 64) * 128) + (cb >> 2) * (C::D * 128) + x * 128 +
           ((((cb & 3) * 2 + n) ^ (x & 7)) << 4);
  };
  auto u_at = [&](int c, int x, int n) {
    return p.su + ((long long)c * p.heads + h) * (2 * wide * (C::D + 64) * 128) + 2 * wide * (C::D * 128) + (cb >> 2) * (64 * 128) + x * 128 +
           ((((cb & 3) * 2 + n) ^ (x & 7)) << 4);
  };
  // planes of the state, for the products and for the outputs of chunk c
  auto publish = [&](int c) {
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const SplitPair s = split2(S[n][2 * x], S[n][2 * x + 1]);
        const uint32_t at = tile_at<2>(m0 + r + 8 * x, n0 + n) + c2 * 2;
        *reinterpret_cast<uint32_t*>(s_s + at) = s.hi;
        *reinterpret_cast<uint32_t*>(s_s + C::S_PLANE + at) = s.lo;
        if (c < c1 && mine) {
          uint8_t* g = state_at(c, m0 + r + 8 * x, n0 + n) + c2 * 2;
          *reinterpret_cast<uint32_t*>(g) = s.hi;
          *reinterpret_cast<uint32_t*>(g + wide * (C::D * 128)) = s.lo;
        }
      }
  };
  const int mt = warp & 3, nh = warp >> 2;                   // of U: 16 tokens, 8 columns
  const int ucol = col0 + nh * 8 + c2;
  float2 u0[2];
  float end[2];
  auto fetch = [&](int c) {
    const long long ch = (long long)c * p.heads + h;
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      u0[x] = ucol < p.vdim_p ? *reinterpret_cast<const float2*>(p.u0 + (ch * 64 + mt * 16 + r + 8 * x) * p.vdim_p + ucol) : make_float2(0.f, 0.f);
      end[x] = p.end[ch * C::D + m0 + r + 8 * x];
    }
  };
  fetch(c0);
  publish(c0);
  const int ar = ((lane >> 3) & 1) * 8 + (lane & 7), ac = lane >> 4;          // this lane's row and chunk for ldmatrix
#pragma unroll 1
  for (int c = c0; c < c1; ++c) {
    const int i = c - c0;
    const bool ok = mbar_wait(smem_u32(&full[i & 1]), (i >> 1) & 1, &s_abort, status, RB_ERR_TIMEOUT_FULL);
    if (!__syncthreads_and(ok)) break;                       // also: the planes of the state are there, the other stage is free
    if (threadIdx.x == 0 && c + 1 < c1) bring(c + 1);
    const uint32_t w = ring + (i & 1) * C::STAGE, kk = w + 2 * C::PLANE;
    float acc[3][4];
#pragma unroll
    for (int n = 0; n < 3; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[n][e] = 0.f;
#pragma unroll
    for (int ks = 0; ks < KS * 4; ++ks) {
      uint32_t hi[4], lo[4], x[4];                           // x: high plane's two fragments, then the low plane's
      const uint32_t aw = w + tile_at<KS * 8>(mt * 16 + ar, ks * 2 + ac);
      ldmatrix_x4(aw, hi);
      ldmatrix_x4(aw + C::PLANE, lo);
      ldmatrix_x4_trans(ss + ac * C::S_PLANE + tile_at<2>(ks * 16 + ar, nh), x);
      mma_bf16(acc[0], hi, x[0], x[1]);
      mma_bf16(acc[1], lo, x[0], x[1]);
      mma_bf16(acc[2], hi, x[2], x[3]);
    }
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const SplitPair s = split2(u0[x].x - (acc[0][2 * x] + (acc[1][2 * x] + acc[2][2 * x])),
                                 u0[x].y - (acc[0][2 * x + 1] + (acc[1][2 * x + 1] + acc[2][2 * x + 1])));
      const uint32_t at = tile_at<2>(mt * 16 + r + 8 * x, nh) + c2 * 2;
      *reinterpret_cast<uint32_t*>(s_u + at) = s.hi;
      *reinterpret_cast<uint32_t*>(s_u + C::U_PLANE + at) = s.lo;
      if (mine) {
        uint8_t* g = u_at(c, mt * 16 + r + 8 * x, nh) + c2 * 2;
        *reinterpret_cast<uint32_t*>(g) = s.hi;
        *reinterpret_cast<uint32_t*>(g + wide * (64 * 128)) = s.lo;
      }
    }
    const float e0 = end[0], e1 = end[1];
    if (c + 1 < c1) fetch(c + 1);
    __syncthreads();
    float add[NT][2][4];
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      S[n][0] *= e0; S[n][1] *= e0; S[n][2] *= e1; S[n][3] *= e1;
#pragma unroll
      for (int e = 0; e < 4; ++e) add[n][0][e] = add[n][1][e] = 0.f;
    }
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t hi[4], lo[4];
      const uint32_t ak = kk + tile_at<KS * 8>(ks * 16 + ac * 8 + (lane & 7), (m0 >> 3) + ((lane >> 3) & 1));
      ldmatrix_x4_trans(ak, hi);
      ldmatrix_x4_trans(ak + C::PLANE, lo);
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        uint32_t x[4];
        ldmatrix_x4_trans(su + ac * C::U_PLANE + tile_at<2>(ks * 16 + ar, n0 + n), x);
        mma_bf16(S[n], hi, x[0], x[1]);
        mma_bf16(add[n][0], lo, x[0], x[1]);
        mma_bf16(add[n][1], hi, x[2], x[3]);
      }
    }
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[n][e] += add[n][0][e] + add[n][1][e];
    publish(c + 1);
  }
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int d = m0 + r + 8 * x, c = col0 + (n0 + n) * 8 + c2;
      if (d < p.dim_p && c < p.vdim_p) *reinterpret_cast<float2*>(state + (long long)d * p.vdim_p + c) = make_float2(S[n][2 * x], S[n][2 * x + 1]);
    }
  if (cb == 0) delta_keep_inputs<bf16>(p.raw, p.ldr, p.conv, seq, h, p.heads, p.kv_heads, p.dim_p, p.vdim_p, p.taps, tid, 256);
}

// ---------------------------------------------------------------------------------------------------------
// outputs on tcgen05.  64 tokens would fill half of a 128-row tile, so the high and the low parts of the left operands are its
// two halves: rows 0 .. 63 of the product with both planes of the right operand and rows 64 .. 127 add up to the result.
// Threads of warps 0-3: (token, half of the columns); warp 4 brings operands, warp 5 issues.
//   room 0   Q', then A, then what the halves exchange        room 1   S_0, high plane, then U        room 2   S_0, low plane,
//   then the output gates, then the results on their way out
// ---------------------------------------------------------------------------------------------------------
struct DeltaMaps {
  CUtensorMap gate;              // [head][row][number], boxes of 64 rows x 64 numbers
};

template <int KS, int VS>
struct DeltaOutCfg {
  static constexpr int D = KS * 64, Q_BYTES = KS * 128 * 128, A_BYTES = 128 * 128, QA = Q_BYTES + A_BYTES;
  static constexpr int S_PLANE = VS * D * 128, U_PLANE = VS * 64 * 128, SU = 2 * (S_PLANE + U_PLANE);
  static constexpr int most(int a, int b) { return a > b ? a : b; }
  static constexpr int ROOM0 = most(most(Q_BYTES, A_BYTES), VS * 128 * 128), ROOM1 = most(S_PLANE, 2 * U_PLANE), ROOM2 = most(S_PLANE, VS * 64 * 128);
  static constexpr int SMEM_BYTES = ROOM0 + ROOM1 + ROOM2 + 1024;
};

template <int KS, int VS>
__global__ void __launch_bounds__(192, 2) delta_chunk_out_kernel(const __grid_constant__ DeltaMaps maps, const DeltaChunkParams p) {
  using C = DeltaOutCfg<KS, VS>;
  constexpr int N = VS * 64, HALF = N / 2;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  __shared__ __align__(16) float s_norm[N];
  __shared__ float s_sum[2][64];
  __shared__ uint64_t bars[5];
  __shared__ uint32_t tmem_ptr;
  __shared__ int s_abort;
  uint64_t *s_full = bars, *s_done = bars + 1, *u_full = bars + 2, *o_done = bars + 3, *gate_full = bars + 4;
  const int4 it = p.items[blockIdx.x];
  const int h = blockIdx.y, tid = threadIdx.x, warp = uniform_warp_idx(), lane = tid & 31;
  const long long ch = (long long)blockIdx.x * p.heads + h;
  const uint32_t r0 = smem_u32(smem), r1 = r0 + C::ROOM0, r2 = r1 + C::ROOM1;
  uint8_t* s_gate = smem + C::ROOM0 + C::ROOM1;
  if (tid == 0) {
    for (int b = 0; b < 5; ++b) mbar_init(smem_u32(&bars[b]), 1);
    s_abort = 0;
    fence_barrier_init();
  }
  if (warp == 5) {
    tmem_alloc(smem_u32(&tmem_ptr), N);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_ptr;
  auto wait = [&](uint64_t* bar, int code) {
    const bool ok = mbar_wait(smem_u32(bar), 0, &s_abort, p.status, code);
    return __all_sync(0xffffffffu, ok) != 0;
  };
  if (warp == 4) {
    const uint8_t *qa = p.qa + ch * C::QA, *su = p.su + ch * C::SU;
    if (lane == 0) {
      const uint32_t bar = smem_u32(s_full);
      mbar_arrive_expect_tx(bar, C::Q_BYTES + 2 * C::S_PLANE);
      bulk_load_1d(r0, qa, C::Q_BYTES, bar);
      bulk_load_1d(r1, su, C::S_PLANE, bar);
      bulk_load_1d(r2, su + C::S_PLANE, C::S_PLANE, bar);
    }
    __syncwarp();
    const bool ok = wait(s_done, RB_ERR_TIMEOUT_EMPTY);
    if (ok && lane == 0) {
      const uint32_t bar = smem_u32(u_full);
      mbar_arrive_expect_tx(bar, C::A_BYTES + 2 * C::U_PLANE);
      bulk_load_1d(r0, qa + C::Q_BYTES, C::A_BYTES, bar);
      bulk_load_1d(r1, su + 2 * C::S_PLANE, 2 * C::U_PLANE, bar);
      mbar_arrive_expect_tx(smem_u32(gate_full), VS * 64 * 128);
#pragma unroll
      for (int x = 0; x < VS; ++x) tma_load_3d(r2 + x * 64 * 128, &maps.gate, smem_u32(gate_full), x * 64, it.x, h);
    }
    __syncwarp();
    if (!ok)
      for (int i = 0; i < 64; ++i) __nanosleep(10000);
  } else if (warp == 5) {
    constexpr uint32_t idesc = make_idesc(UmmaFormat<bf16>::value, 0, 1, 128, N);
    bool ok = wait(s_full, RB_ERR_TIMEOUT_FULL);
    if (ok) {
      tc_fence_after();
#pragma unroll
      for (int plane = 0; plane < 2; ++plane)
#pragma unroll
        for (int x = 0; x < KS; ++x)                    // 64 key numbers
          umma_f16_w4<2, 128>(tmem, make_smem_desc_sw128(r0 + x * 128 * 128, 16, 1024),
                              make_smem_desc_sw128((plane ? r2 : r1) + x * 64 * 128, C::D * 128, 1024), idesc, plane + x != 0);
      umma_commit_w(smem_u32(s_done));
      ok = wait(u_full, RB_ERR_TIMEOUT_FULL);
    }
    if (ok) {
      tc_fence_after();
#pragma unroll
      for (int plane = 0; plane < 2; ++plane)
        umma_f16_w4<2, 128>(tmem, make_smem_desc_sw128(r0, 16, 1024), make_smem_desc_sw128(r1 + plane * C::U_PLANE, 64 * 128, 1024), idesc, 1u);
      umma_commit_w(smem_u32(o_done));
    }
  } else {
    // lanes 0-63 of tensor memory have the sums with high parts, 64-127 those with low parts; a thread of the first keeps the
    // first half of its token's columns, one of the second the second half, and they hand the rest to each other
    const int t = tid & 63, upper = tid >> 6;
    const uint32_t lane_addr = tmem + (static_cast<uint32_t>(warp * 32) << 16);
    if (tid < N) s_norm[tid] = tid < p.vdim_p ? p.o.norm[h * p.o.norm_step + tid] : 0.f;
    bool ok = wait(o_done, RB_ERR_TIMEOUT_TMEM_FULL) && wait(gate_full, RB_ERR_TIMEOUT_FULL);
    float o[HALF];
    auto swap_at = [&](int half, int c) {               // four numbers of a token's half; c: 16-byte chunk
      return reinterpret_cast<float4*>(smem + half * (64 * HALF * 4) + t * (HALF * 4) + ((c ^ (t & (HALF / 4 - 1))) << 4));
    };
    if (ok) {
      tc_fence_after();
#pragma unroll
      for (int x = 0; x < HALF; x += 32) {
        uint32_t r[32];
        tmem_ld_32x32b_x32(lane_addr + (upper ? 0 : HALF) + x, r);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; i += 4)
          *swap_at(upper ? 0 : 1, (x + i) / 4) =
              make_float4(__uint_as_float(r[i]), __uint_as_float(r[i + 1]), __uint_as_float(r[i + 2]), __uint_as_float(r[i + 3]));
      }
#pragma unroll
      for (int x = 0; x < HALF; x += 32) {
        uint32_t r[32];
        tmem_ld_32x32b_x32(lane_addr + (upper ? HALF : 0) + x, r);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) o[x + i] = __uint_as_float(r[i]);
      }
    }
    asm volatile("bar.sync 1, 128;" ::: "memory");
    float sum = 0.f;
    if (ok) {
#pragma unroll
      for (int c = 0; c < HALF / 4; ++c) {
        const float4 v = *swap_at(upper, c);
        o[4 * c] += v.x; o[4 * c + 1] += v.y; o[4 * c + 2] += v.z; o[4 * c + 3] += v.w;
#pragma unroll
        for (int e = 0; e < 4; ++e) {                   // columns past the value size may hold anything
          if (upper * HALF + 4 * c + e >= p.vdim_p) o[4 * c + e] = 0.f;
          sum = fmaf(o[4 * c + e], o[4 * c + e], sum);
        }
      }
    }
    s_sum[upper][t] = sum;
    asm volatile("bar.sync 1, 128;" ::: "memory");
    const float scale = 1.0f / sqrtf((s_sum[0][t] + s_sum[1][t]) / p.vdim + p.o.eps);
    auto gate_at = [&](int row, int c) {                // 16-byte chunk c of a row
      return reinterpret_cast<uint4*>(s_gate + (c >> 3) * (64 * 128) + row * 128 + (((c & 7) ^ (row & 7)) << 4));
    };
    if (ok) {
#pragma unroll
      for (int x = 0; x < HALF / 8; ++x) {              // a thread's gates give way to its results
        uint4* at = gate_at(t, upper * (HALF / 8) + x);
        uint4 g = *at;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 gate = unpack2<bf16>(reinterpret_cast<const uint32_t*>(&g)[e]);
          const float2 n = *reinterpret_cast<const float2*>(s_norm + upper * HALF + x * 8 + e * 2);
          const float gx = sigmoid_tanh(gate.x) * (p.o.silu ? gate.x : 1.0f), gy = sigmoid_tanh(gate.y) * (p.o.silu ? gate.y : 1.0f);
          reinterpret_cast<uint32_t*>(&g)[e] = pack2<bf16>(o[x * 8 + 2 * e] * scale * n.x * gx, o[x * 8 + 2 * e + 1] * scale * n.y * gy);
        }
        *at = g;
      }
    }
    asm volatile("bar.sync 1, 128;" ::: "memory");
    const int x = tid % (VS * 8);
    if (ok && x * 8 < p.vdim_p) {
#pragma unroll 4
      for (int row = tid / (VS * 8); row < 64; row += 128 / (VS * 8))
        if (row < it.y) *reinterpret_cast<uint4*>(p.o.out + (long long)(it.x + row) * p.o.ldo + (long long)h * p.vdim_p + x * 8) = *gate_at(row, x);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 5) {
    tc_fence_after();
    tmem_dealloc(tmem, N);
  }
}

template <int KS, int VS>
int launch_delta_chunk(const DeltaChunkParams& p, int tokens, int n_items, int portions, cudaStream_t st) {
  DeltaMaps maps;
  {
    uint64_t dims[3] = {(uint64_t)p.vdim_p, (uint64_t)tokens, (uint64_t)p.heads};
    uint64_t strides[3] = {2, (uint64_t)p.o.ldg * 2, (uint64_t)p.vdim_p * 2};
    uint32_t box[3] = {64, 64, 1};
    const int rc = rbh::encode_tensor_map(&maps.gate, rbh::DT_BF16, 3, const_cast<bf16*>(p.o.gate), dims, strides, box, 1);
    if (rc) return 1000 + rc;
  }
  auto local = p.per_head ? delta_chunk_local_kernel<KS, VS, true> : delta_chunk_local_kernel<KS, VS, false>;
  const int blocks = (p.vdim_p + kDeltaCols - 1) / kDeltaCols, groups = blocks > 1 && (long long)blocks * p.heads * portions > rbh::sm_count() ? 2 : 1;
  auto scan = groups == 2 ? delta_chunk_scan_kernel<KS, 2> : delta_chunk_scan_kernel<KS, 1>;
  auto outputs = delta_chunk_out_kernel<KS, VS>;
  const int sl = p.per_head ? DeltaLocalCfg<KS, VS, true>::SMEM_BYTES : DeltaLocalCfg<KS, VS, false>::SMEM_BYTES;
  const int ss = groups == 2 ? DeltaScanCfg<KS, 2>::SMEM_BYTES : DeltaScanCfg<KS, 1>::SMEM_BYTES, so = DeltaOutCfg<KS, VS>::SMEM_BYTES;
  cudaError_t e = cudaFuncSetAttribute(local, cudaFuncAttributeMaxDynamicSharedMemorySize, sl);
  if (e == cudaSuccess) e = cudaFuncSetAttribute(scan, cudaFuncAttributeMaxDynamicSharedMemorySize, ss);
  if (e == cudaSuccess) e = cudaFuncSetAttribute(outputs, cudaFuncAttributeMaxDynamicSharedMemorySize, so);
  if (e != cudaSuccess) return 2000 + (int)e;
  local<<<dim3(n_items, p.heads), 512, sl, st>>>(p);
  scan<<<dim3((blocks + groups - 1) / groups, p.heads, portions), 256 * groups, ss, st>>>(p, p.status);
  outputs<<<dim3(n_items, p.heads), 192, so, st>>>(maps, p);
  e = cudaGetLastError();
  return e == cudaSuccess ? 0 : 3000 + (int)e;
}

}  // namespace rb

extern "C" {

// Whether the kernels cover these sizes (others run token by token).
int rb_delta_chunk_ok(int dtype, int dim_p, int vdim_p) {
  return dtype == rbh::DT_BF16 && dim_p <= 128 && vdim_p <= 128 && dim_p % 8 == 0 && vdim_p % 8 == 0;
}

// Bytes of scratch per chunk and head: planes of W and K'', of Q' and A, blocks of S_0 and U, U_0, decays of the chunk.
struct DeltaScratch {
  long long wk, qa, su, u0, end;
};
static DeltaScratch delta_scratch(int dim_p, int vdim_p) {
  const long long D = dim_p <= 64 ? 64 : 128, wide = (vdim_p + 63) / 64;
  return {4 * 64 * D * 2, 2 * 64 * D * 2 + 2 * 64 * 128, wide * 2 * (D + 64) * 128, 64LL * vdim_p * 4, D * 4};
}
long long rb_delta_chunk_scratch(int dim_p, int vdim_p) {
  const DeltaScratch n = delta_scratch(dim_p, vdim_p);
  return n.wk + n.qa + n.su + n.u0 + n.end;
}

// raw, a, b, gate: `tokens` rows, the whole batch's (items count from row 0); items: chunks of up to 64 tokens; first: [portions + 1];
// scratch: rb_delta_chunk_scratch bytes per chunk and head.  Otherwise as rb_delta_prep and rb_delta_rows.
int rb_delta_chunk(int dtype, const void* raw, long long ldr, int tokens, const float* taps_w, void* conv, const float* a, long long lda,
                   int per_head, const float* dt, const float* decay, const float* b, long long ldb, const int* items, int n_items, const int* seqs, const int* first,
                   int portions, float* S, const void* gate, long long ldg, const float* norm, void* out, long long ldo, void* scratch,
                   int heads, int kv_heads, int dim_p, int vdim_p, int vdim, int taps, float q_scale, float eps, int silu, void* stream) {
  using namespace rb;
  if (n_items <= 0) return 0;
  if (!rb_delta_chunk_ok(dtype, dim_p, vdim_p) || heads % kv_heads || heads > 65535 || portions > 65535 || taps < 1) return 22;
  auto al = [](const void* x, int to) { return (reinterpret_cast<uintptr_t>(x) & (to - 1)) == 0; };
  if (!al(raw, 8) || !al(conv, 8) || !al(taps_w, 16) || (!per_head && (!al(a, 16) || !al(dt, 16) || lda % 4)) || !al(S, 16) || !al(gate, 16) || !al(out, 16) || !al(norm, 4) ||
      !al(scratch, 256) || ldr % 4 || ldg % 8 || ldo % 8)
    return 21;
  DeltaChunkParams p{};
  p.raw = (const bf16*)raw; p.ldr = ldr; p.taps_w = taps_w; p.conv = (bf16*)conv; p.a = a; p.lda = lda; p.per_head = per_head; p.dt = dt; p.decay = decay; p.b = b; p.ldb = ldb;
  p.items = (const int4*)items; p.seqs = (const int4*)seqs; p.first = first; p.S = S; p.heads = heads; p.kv_heads = kv_heads; p.dim_p = dim_p;
  p.vdim_p = vdim_p; p.vdim = vdim; p.taps = taps; p.q_scale = q_scale;
  p.channels = 2 * kv_heads * dim_p + heads * vdim_p;
  p.status = rbh::device_status_word();
  p.o = RecOut<bf16>{(bf16*)out, ldo, (const bf16*)gate, ldg, norm, 0, nullptr, eps, silu};
  const long long N = (long long)n_items * heads;
  char* at = (char*)scratch;
  auto take = [&](long long bytes) {
    char* x = at;
    at += N * bytes;
    return x;
  };
  const DeltaScratch sz = delta_scratch(dim_p, vdim_p);
  p.wk = (uint8_t*)take(sz.wk);
  p.qa = (uint8_t*)take(sz.qa);
  p.su = (uint8_t*)take(sz.su);
  p.u0 = (float*)take(sz.u0);
  p.end = (float*)take(sz.end);
  cudaStream_t st = (cudaStream_t)stream;
  if (dim_p <= 64) return vdim_p <= 64 ? launch_delta_chunk<1, 1>(p, tokens, n_items, portions, st) : launch_delta_chunk<1, 2>(p, tokens, n_items, portions, st);
  return vdim_p <= 64 ? launch_delta_chunk<2, 1>(p, tokens, n_items, portions, st) : launch_delta_chunk<2, 2>(p, tokens, n_items, portions, st);
}
}
