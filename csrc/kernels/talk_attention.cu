// Attention whose heads talk, sm_100a: the scores of a pair (query, key) in all heads are mixed by a matrix before the
// softmax, s'_h = sum over g of M[h, g] (q_g . k_g'), with g' the key/value head of query head g.  Here: what follows the
// input projection, and single query rows of any size and type (32-bit runs, large heads).  16-bit rows are in
// talk_decode.cu, prompt tiles in talk_prefill.cu.
//
// Values may be the keys as they were projected, before their rotation; the cache then keeps both forms.
// Cache layout: pool [num_blocks, kv_heads, block_size, dim], as for the other windows (window_attention.cu).
#include <type_traits>

#include "attn_merge.cuh"

namespace rb {

template <typename T>
__device__ __forceinline__ float4 talk_load4(const T* p) {
  if constexpr (sizeof(T) == 4) {
    return *reinterpret_cast<const float4*>(p);
  } else {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    const float2 lo = unpack2<T>(a.x), hi = unpack2<T>(a.y);
    return make_float4(lo.x, lo.y, hi.x, hi.y);
  }
}

// ---------------------------------------------------------------------------------------------------------
// after the input projection [q | k | ...]: rotation of every query and key head (element i with i + half); keys go to
// their cache rows rotated, and as they are to the values' rows.  Queries of single rows change in place.  Queries of
// prompt tiles leave mixed: s'_h is one product of keys of all key/value heads side by side with
//   q'_h = (sum over g of group c of M[h, g] q_g) for every key/value head c,
// so the tile kernel never sees more than one head's scores.
// REP: query heads per key/value head, rounded up; the queries of a group stay in registers.  QUAD: heads of up to 128 numbers
// whose rotation is made of whole groups of four: a warp has a head, a lane four neighbouring numbers, their partners come from
// another lane.  A CTA takes per_cta tokens.
// ---------------------------------------------------------------------------------------------------------
template <typename T>
struct TalkPostParams {
  T* proj;
  long long ldp;
  const float2* tab;          // [tokens, half] (cos, sin)
  const long long* slots;     // cache slot (block * block_size + offset) of every token, -1: keep nothing
  T *k_pool, *v_pool;
  const float* mix;           // [heads, heads]
  T* qmix;                    // [tokens - rows, heads, kv_heads, dim_p]
  long long tokens;
  int rows;                   // tokens whose queries change in place
  int per_cta;
  int heads, kv_heads, dim_p, half, block_size;
};

template <typename T>
__device__ __forceinline__ void talk_store4(T* p, float4 v) {
  if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>(p) = v;
  else *reinterpret_cast<uint2*>(p) = make_uint2(pack2<T>(v.x, v.y), pack2<T>(v.z, v.w));
}

template <typename T, int REP, bool QUAD>
__global__ void __launch_bounds__(256) talk_post_kernel(const TalkPostParams<T> p) {
  extern __shared__ __align__(16) float s_q[];             // [heads][dim_p], then [heads][kv_heads * REP]: M by groups
  const int tid = threadIdx.x, D = p.dim_p, rep = p.heads / p.kv_heads;
  float* s_m = s_q + p.heads * D;
  const long long first = (long long)blockIdx.x * p.per_cta, end = first + p.per_cta < p.tokens ? first + p.per_cta : p.tokens;
  if (end > p.rows)
    for (int i = tid; i < p.heads * p.kv_heads * REP; i += 256) {
      const int h = i / (p.kv_heads * REP), x = i - h * p.kv_heads * REP, c = x / REP, r = x - c * REP;
      s_m[i] = r < rep ? p.mix[h * p.heads + c * rep + r] : 0.f;
    }
  for (long long t = first; t < end; ++t) {
    T* row = p.proj + t * p.ldp;
    const float2* tab = p.tab + t * p.half;
    const bool tile = t >= p.rows;
    const long long slot = p.slots[t], blk = slot / p.block_size;
    const int off = (int)(slot - blk * p.block_size);
    auto cache_at = [&](int g) { return ((blk * p.kv_heads + g) * p.block_size + off) * D; };
    if constexpr (QUAD) {
      const int lane = tid & 31, c = lane * 4, reach = p.half >> 2;      // lanes between the two halves of a pair
      const bool low = lane < reach, high = !low && lane < 2 * reach;
      float2 cs[4];
      if (low || high) {
#pragma unroll
        for (int e = 0; e < 4; ++e) cs[e] = tab[(low ? c : c - p.half) + e];
      }
      for (int head = tid >> 5; head < p.heads + p.kv_heads; head += 8) {
        const bool is_q = head < p.heads;
        if (!is_q && slot < 0) break;
        T* src = row + head * D + c;
        const float4 v = c < D ? talk_load4<T>(src) : make_float4(0.f, 0.f, 0.f, 0.f);
        float x[4] = {v.x, v.y, v.z, v.w}, other[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) other[e] = __shfl_sync(0xffffffffu, x[e], low ? lane + reach : high ? lane - reach : lane);
        if (low || high) {
#pragma unroll
          for (int e = 0; e < 4; ++e) x[e] = low ? x[e] * cs[e].x - other[e] * cs[e].y : x[e] * cs[e].x + other[e] * cs[e].y;
        }
        if (c >= D) continue;
        const float4 o = make_float4(x[0], x[1], x[2], x[3]);
        if (is_q) {
          if (tile) *reinterpret_cast<float4*>(s_q + head * D + c) = o;
          else talk_store4<T>(src, o);
        } else {
          talk_store4<T>(p.k_pool + cache_at(head - p.heads) + c, o);
          talk_store4<T>(p.v_pool + cache_at(head - p.heads) + c, v);
        }
      }
    } else {
      for (int i = tid; i < (p.heads + p.kv_heads) * D; i += 256) {
        const int head = i / D, c = i - head * D;
        const bool is_q = head < p.heads;
        if (!is_q && slot < 0) break;
        const float x = to_f32<T>(row[i]);
        // a pair belongs to the thread of its lower element, so writing in place is safe
        if (is_q && !tile) {
          if (c < p.half) {
            const float2 cs = tab[c];
            const float v = to_f32<T>(row[i + p.half]);
            row[i] = from_f32<T>(x * cs.x - v * cs.y);
            row[i + p.half] = from_f32<T>(v * cs.x + x * cs.y);
          }
          continue;
        }
        float r = x;
        if (c < p.half) {
          const float2 cs = tab[c];
          r = x * cs.x - to_f32<T>(row[i + p.half]) * cs.y;
        } else if (c < 2 * p.half) {
          const float2 cs = tab[c - p.half];
          r = x * cs.x + to_f32<T>(row[i - p.half]) * cs.y;
        }
        if (is_q) {
          s_q[i] = r;
        } else {
          p.k_pool[cache_at(head - p.heads) + c] = from_f32<T>(r);
          p.v_pool[cache_at(head - p.heads) + c] = row[i];
        }
      }
    }
    if (!tile) continue;                                   // the same for all threads
    __syncthreads();
    // a thread has eight numbers of a group's queries and a share of the heads
    const int pieces = p.kv_heads * (D >> 3), shares = max(1, 256 / pieces);
    T* out = p.qmix + (t - p.rows) * (long long)p.heads * p.kv_heads * D;
    for (int x = tid; x < pieces * shares; x += 256) {
      const int share = x / pieces, y = x - share * pieces, c = y / (D >> 3), d = (y - c * (D >> 3)) * 8;
      float q[REP][8];
#pragma unroll
      for (int r = 0; r < REP; ++r)
#pragma unroll
        for (int e = 0; e < 8; e += 4) {
          const float4 v = r < rep ? *reinterpret_cast<const float4*>(s_q + (c * rep + r) * D + d + e) : make_float4(0.f, 0.f, 0.f, 0.f);
          q[r][e] = v.x; q[r][e + 1] = v.y; q[r][e + 2] = v.z; q[r][e + 3] = v.w;
        }
      for (int h = share; h < p.heads; h += shares) {
        float m[REP];
        const float* mp = s_m + (h * p.kv_heads + c) * REP;
        if constexpr (REP % 4 == 0) {
#pragma unroll
          for (int r = 0; r < REP; r += 4) *reinterpret_cast<float4*>(m + r) = *reinterpret_cast<const float4*>(mp + r);
        } else {
#pragma unroll
          for (int r = 0; r < REP; ++r) m[r] = mp[r];
        }
        float o[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int r = 0; r < REP; ++r)
#pragma unroll
          for (int e = 0; e < 8; ++e) o[e] = fmaf(m[r], q[r][e], o[e]);
        T* dst = out + ((long long)h * p.kv_heads + c) * D + d;
        if constexpr (sizeof(T) == 4) {
          reinterpret_cast<float4*>(dst)[0] = make_float4(o[0], o[1], o[2], o[3]);
          reinterpret_cast<float4*>(dst)[1] = make_float4(o[4], o[5], o[6], o[7]);
        } else {
          *reinterpret_cast<uint4*>(dst) = make_uint4(pack2<T>(o[0], o[1]), pack2<T>(o[2], o[3]), pack2<T>(o[4], o[5]), pack2<T>(o[6], o[7]));
        }
      }
    }
    __syncthreads();
  }
}

// ---------------------------------------------------------------------------------------------------------
// single query rows, any size.  A CTA takes a slice of one row's visible keys for all heads, 32 keys at a time: a lane
// has a key and a warp a few heads of a group for the raw scores, which all heads then read from shared memory.
// ---------------------------------------------------------------------------------------------------------
struct TalkRowsParams {
  const void *q, *k_pool, *v_pool;
  long long ldq;                 // query row stride; head h at h * dim
  const int *tables, *ctx;       // [rows, max_blocks], [rows]: keys up to and with the row's own
  const float *mix, *sink;       // [heads, heads]; [heads] or null
  const void* gate;
  long long ldg, ldo;
  void* out;
  float *part_o, *part_ml;       // used when splits > 1
  int heads, kv_heads, dim, vdim, window, block_size, max_blocks, splits, gate_kind;
  float scale_log2;
};
constexpr int kTalkKeys = 32, kTalkLd = 33;

template <typename T>
__global__ void __launch_bounds__(256) talk_rows_kernel(const TalkRowsParams p) {
  extern __shared__ __align__(16) float s_q[];             // [heads][dim]
  float* s_acc = s_q + p.heads * p.dim;                    // [heads][vdim]
  float* s_raw = s_acc + p.heads * p.vdim;                 // [heads][kTalkLd]
  float* s_p = s_raw + p.heads * kTalkLd;                  // the same: weights
  float* s_ml = s_p + p.heads * kTalkLd;                   // [heads] maxima, sums, factors on what was summed so far
  __shared__ long long s_row[kTalkKeys];                   // pool row of every key, of key/value head 0
  const int H = p.heads, D = p.dim, V = p.vdim, rep = H / p.kv_heads, b = blockIdx.x, sp = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int ctx = p.ctx[b], lo = max(0, ctx - p.window), n = ctx - lo, per = (n + p.splits - 1) / p.splits;
  const int t0 = lo + sp * per, t1 = min(ctx, t0 + per);
  const T *kp = reinterpret_cast<const T*>(p.k_pool), *vp = reinterpret_cast<const T*>(p.v_pool);
  const int* table = p.tables + (long long)b * p.max_blocks;
  auto ex2 = [](float x) { return sizeof(T) == 4 ? exp2f(x) : fast_exp2(x); };
  for (int i = threadIdx.x; i < H * D; i += 256) s_q[i] = to_f32<T>(reinterpret_cast<const T*>(p.q)[b * p.ldq + i]) * p.scale_log2;
  for (int i = threadIdx.x; i < H * V; i += 256) s_acc[i] = 0.f;
  for (int h = threadIdx.x; h < H; h += 256) {
    s_ml[h] = -INFINITY;
    s_ml[H + h] = 0.f;
  }
  for (int base = t0; base < t1; base += kTalkKeys) {
    __syncthreads();
    const int key = base + lane;
    if (warp == 0) {
      const int t = min(key, t1 - 1);
      s_row[lane] = (long long)table[min(t / p.block_size, p.max_blocks - 1)] * p.kv_heads * p.block_size + t % p.block_size;
    }
    __syncthreads();
    // raw scores: four heads of a group at a time
    const int quads = (rep + 3) / 4;
    for (int i = warp; i < p.kv_heads * quads; i += 8) {
      const int c = i / quads, r0 = (i - c * quads) * 4, h0 = c * rep + r0, nh = min(4, rep - r0);
      const T* kr = kp + (s_row[lane] + (long long)c * p.block_size) * D;
      float s[4] = {0.f, 0.f, 0.f, 0.f};
      for (int d = 0; d < D; d += 4) {
        const float4 k = talk_load4<T>(kr + d);
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const float4 q = *reinterpret_cast<const float4*>(s_q + (h0 + min(x, nh - 1)) * D + d);
          s[x] = fmaf(q.x, k.x, fmaf(q.y, k.y, fmaf(q.z, k.z, fmaf(q.w, k.w, s[x]))));
        }
      }
#pragma unroll
      for (int x = 0; x < 4; ++x)
        if (x < nh) s_raw[(h0 + x) * kTalkLd + lane] = s[x];
    }
    __syncthreads();
    for (int h = warp; h < H; h += 8) {
      float s = 0.f;
      for (int g = 0; g < H; ++g) s = fmaf(p.mix[h * H + g], s_raw[g * kTalkLd + lane], s);
      if (key >= t1) s = -INFINITY;
      const float m = s_ml[h], mx = fmaxf(m, warp_max(s));           // at least one key is live
      const float w = key < t1 ? ex2(s - mx) : 0.f, l = warp_sum(w);
      s_p[h * kTalkLd + lane] = w;
      __syncwarp();
      if (lane == 0) {
        const float f = m == -INFINITY ? 0.f : ex2(m - mx);
        s_ml[h] = mx;
        s_ml[H + h] = s_ml[H + h] * f + l;
        s_ml[2 * H + h] = f;
      }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < H * (V >> 2); i += 256) {
      const int h = i / (V >> 2), d = (i - h * (V >> 2)) * 4, c = h / rep;
      float4 o = *reinterpret_cast<float4*>(s_acc + h * V + d);
      const float f = s_ml[2 * H + h];
      o.x *= f; o.y *= f; o.z *= f; o.w *= f;
      const int live = min(kTalkKeys, t1 - base);
      for (int j = 0; j < live; ++j) {
        const float w = s_p[h * kTalkLd + j];
        const float4 v = talk_load4<T>(vp + (s_row[j] + (long long)c * p.block_size) * V + d);
        o.x = fmaf(w, v.x, o.x); o.y = fmaf(w, v.y, o.y); o.z = fmaf(w, v.z, o.z); o.w = fmaf(w, v.w, o.w);
      }
      *reinterpret_cast<float4*>(s_acc + h * V + d) = o;
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < H * V; i += 256) {
    const int h = i / V, d = i - h * V;
    if (p.splits > 1) {
      const long long pi = ((long long)b * H + h) * p.splits + sp;
      p.part_o[pi * V + d] = s_acc[i];
      if (d == 0) {
        p.part_ml[pi * 2] = s_ml[h];
        p.part_ml[pi * 2 + 1] = s_ml[H + h];
      }
      continue;
    }
    const float sk = p.sink ? p.sink[h] * 1.4426950408889634f : -INFINITY, m = s_ml[h], gm = fmaxf(m, sk);
    const float f = ex2(m - gm);
    float l = s_ml[H + h] * f;
    if (p.sink) l += ex2(sk - gm);
    float v = s_acc[i] * f / l;
    if (p.gate_kind == ATTN_GATE_ELEMENT) v *= sigmoid_f<T>(to_f32<T>(reinterpret_cast<const T*>(p.gate)[b * p.ldg + (long long)h * V + d]));
    else if (p.gate_kind == ATTN_GATE_HEAD) v *= sigmoid_f<T>(to_f32<T>(reinterpret_cast<const T*>(p.gate)[b * p.ldg + h]));
    reinterpret_cast<T*>(p.out)[b * p.ldo + (long long)h * V + d] = from_f32<T>(v);
  }
}

}  // namespace rb

#define RB_BY_DTYPE(...)                                               \
  if (dtype == rbh::DT_BF16) { using T = __nv_bfloat16; __VA_ARGS__; } \
  else if (dtype == rbh::DT_F32) { using T = float; __VA_ARGS__; }     \
  else return 20;
#define RB_LAUNCH_STATUS()             \
  cudaError_t e_ = cudaGetLastError(); \
  return e_ == cudaSuccess ? 0 : 3000 + (int)e_

extern "C" {

// proj row: heads x dim_p queries, kv_heads x dim_p keys.  The first `rows` tokens' queries change in place; the others'
// go to qmix [tokens - rows, heads, kv_heads, dim_p] (at most 8 query heads per key/value head), see TalkPostParams.
int rb_talk_post(int dtype, void* proj, long long ldp, const float* tab, const long long* slots, void* k_pool, void* v_pool, const float* mix,
                 void* qmix, long long tokens, int rows, int heads, int kv_heads, int dim_p, int rot, int block_size, void* stream) {
  using namespace rb;
  if (tokens <= 0) return 0;
  const int rep = heads / kv_heads;
  if ((rot & 1) || rot > dim_p || dim_p % 8 || ldp % 8 || heads % kv_heads || (rot && !tab)) return 21;
  if (rows < tokens && (rep > 8 || !qmix || !mix)) return 22;
  // tokens share a CTA's copy of the mixing matrix where there are many
  const int per_cta = rows < tokens && tokens >= 16LL * rbh::sm_count() ? 4 : 1;
  const bool quad = dim_p <= 128 && rot % 8 == 0;
  RB_BY_DTYPE({
    const TalkPostParams<T> p{(T*)proj, ldp, (const float2*)tab, slots, (T*)k_pool, (T*)v_pool, mix, (T*)qmix, tokens, rows, per_cta, heads,
                              kv_heads, dim_p, rot / 2, block_size};
    auto go = [&](auto kern, int REP) {
      const int smem = rows < tokens ? heads * (dim_p + kv_heads * REP) * 4 : 0;
      if (smem > 40 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return 2000 + (int)e;
      }
      kern<<<(unsigned)((tokens + per_cta - 1) / per_cta), 256, smem, (cudaStream_t)stream>>>(p);
      return 0;
    };
    auto by_rep = [&](auto q) {
      constexpr bool Q = decltype(q)::value;
      if (rep <= 1) return go(talk_post_kernel<T, 1, Q>, 1);
      if (rep <= 2) return go(talk_post_kernel<T, 2, Q>, 2);
      if (rep <= 4 || rows == tokens) return go(talk_post_kernel<T, 4, Q>, 4);
      return go(talk_post_kernel<T, 8, Q>, 8);
    };
    const int rc = quad ? by_rep(std::true_type{}) : by_rep(std::false_type{});
    if (rc) return rc;
  })
  RB_LAUNCH_STATUS();
}

// Bytes of shared memory that a CTA of the rows kernel takes; more than 227 KB: too large.
int rb_talk_rows_smem(int heads, int dim_p, int vdim_p) { return (heads * (dim_p + vdim_p + 2 * rb::kTalkLd + 3)) * 4; }

// q: row t, head h at q[t * ldq + h * dim_p]; out the same with ldo and vdim_p.  gate_kind: see attn_merge.cuh.
// Every row sees the last `window` of its keys.  Scratch for splits > 1: part_o rows*heads*splits*vdim_p floats, part_ml rows*heads*splits*2.
int rb_talk_rows(int dtype, const void* q, long long ldq, const void* k_pool, const void* v_pool, const int* tables, const int* ctx,
                 const float* mix, const float* sink, const void* gate, long long ldg, int gate_kind, void* out, long long ldo, float* part_o,
                 float* part_ml, int rows, int heads, int kv_heads, int dim_p, int vdim_p, int window, int block_size, int max_blocks,
                 int splits, float scale, void* stream) {
  using namespace rb;
  if (rows <= 0) return 0;
  const int smem = rb_talk_rows_smem(heads, dim_p, vdim_p);
  if (splits < 1 || splits > 1024 || heads % kv_heads || window < 1 || block_size < 1 || smem > 227 * 1024) return 22;
  auto al = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
  if (!al(q) || !al(k_pool) || !al(v_pool) || ldq % 8 || dim_p % 8 || vdim_p % 8) return 21;
  const TalkRowsParams p{q, k_pool, v_pool, ldq, tables, ctx, mix, sink, gate, ldg, ldo, out, part_o, part_ml, heads, kv_heads, dim_p, vdim_p,
                         window, block_size, max_blocks, splits, gate ? gate_kind : ATTN_GATE_NONE, scale * 1.4426950408889634f};
  cudaStream_t st = (cudaStream_t)stream;
  RB_BY_DTYPE({
    const cudaError_t e = cudaFuncSetAttribute(talk_rows_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return 2000 + (int)e;
    talk_rows_kernel<T><<<dim3(rows, splits), 256, smem, st>>>(p);
    if (splits > 1)
      launch_attn_merge<T>(part_o, part_ml, sink, (const T*)gate, ldg, p.gate_kind, (T*)out, ldo, rows, heads, vdim_p, splits, st);
  })
  RB_LAUNCH_STATUS();
}
}
