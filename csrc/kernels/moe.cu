// Mixture of experts, sm_100a: routing, the bookkeeping that groups tokens by expert, and a plain grouped product
// for every size and type.  The tensor-core grouped products are in moe_gemm.cu.
//
// Everything stays on the device and has launch shapes that do not depend on the routing, so a step can be captured
// in a CUDA graph.  A (token, choice) pair gets a slot; the slots of an expert are neighbours:
//
//   route     per token: logits, the top-k choices and their weights (softmax over the chosen logits; or the logits'
//             sigmoids, chosen with a correction added and only from the best groups), rank among the expert's tokens
//             (an atomic counter); the last CTA turns the counts into first slots per expert and work items
//             {expert, first slot, slots} of at most `tile` slots, and re-arms the counters
//   place     slot -> token and weight, (token, choice) -> slot; done by the last CTA itself when there are few pairs.
//             For large batches it also copies every token's row to its slots; for products in the largest tiles an
//             expert's slots start at a multiple of the tile, so that item i is rows i * tile .. of the sorted rows
//
// The weights of the gates and ups of an expert are stored in turns, 32 rows of each.  The routing weight goes onto
// gated unit, where it is still in 32 bits; the product behind it is linear.
//
// The order of tokens inside an expert depends on the atomics, the result does not: every slot is computed on its
// own.
#include "sm100_common.cuh"

namespace rb {

constexpr int kMoeMaxExperts = 1024;
constexpr int kMoeMaxGroups = 64;
enum : int { MOE_SOFTMAX = 0, MOE_SIGMOID = 1 };

struct MoeRouteParams {
  const float* bias;             // [experts]; softmax: part of the logits, sigmoid: added to the scores for the choice only
  int score, groups, keep;       // sigmoid: groups of neighbouring experts, of which the best `keep` are open
  int tokens, experts, top, tile, align;
  int* counts;                   // [experts] + finished CTAs, zero between launches
  int* idx;                      // [tokens, top] expert of every choice
  float* weight;                 // [tokens, top]
  int* rank;                     // [tokens, top] place among the expert's slots
  int* first;                    // [experts] first slot
  int4* items;                   // work items
  int* n_items;
  int* slot_token;               // [tokens * top]
  float* slot_weight;
  int* slot_of;                  // [tokens, top]
  int place;                     // the last CTA also places the pairs
};

__device__ __forceinline__ void moe_place(const MoeRouteParams& p, int i) {
  const int slot = __ldcg(&p.first[__ldcg(&p.idx[i])]) + __ldcg(&p.rank[i]);
  p.slot_token[slot] = i / p.top;
  p.slot_weight[slot] = __ldcg(&p.weight[i]);
  p.slot_of[i] = slot;
}

__device__ __forceinline__ float moe_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }

// One warp: closes (-infinity) the experts of all but the best groups; a group's score is the sum of its two largest.
__device__ __forceinline__ void moe_close_groups(const MoeRouteParams& p, float* z) {
  const int lane = threadIdx.x & 31, size = p.experts / p.groups;
  float score[kMoeMaxGroups / 32];
#pragma unroll
  for (int i = 0; i < kMoeMaxGroups / 32; ++i) {
    const int g = i * 32 + lane;
    float a = -INFINITY, b = -INFINITY;
    if (g < p.groups)
      for (int e = g * size; e < (g + 1) * size; ++e) {
        b = fmaxf(b, fminf(a, z[e]));
        a = fmaxf(a, z[e]);
      }
    score[i] = size > 1 ? a + b : a;
  }
  // a group's rank: how many are better (the lower index wins a tie)
  int rank[kMoeMaxGroups / 32] = {};
  for (int o = 0; o < p.groups; ++o) {
    const float s = __shfl_sync(0xffffffffu, o < 32 ? score[0] : score[1], o & 31);
#pragma unroll
    for (int i = 0; i < kMoeMaxGroups / 32; ++i) {
      const int g = i * 32 + lane;
      rank[i] += s > score[i] || (s == score[i] && o < g);
    }
  }
  __syncwarp();
#pragma unroll
  for (int i = 0; i < kMoeMaxGroups / 32; ++i) {
    const int g = i * 32 + lane;
    if (g < p.groups && rank[i] >= p.keep)
      for (int e = g * size; e < (g + 1) * size; ++e) z[e] = -INFINITY;
  }
  __syncwarp();
}

// One warp: the `top` largest of z[0 .. experts) (the lower index wins a tie), overwritten as they are taken.
// `raw`: the logits themselves (sigmoid).
__device__ __forceinline__ void moe_select(const MoeRouteParams& p, float* z, const float* raw, int token) {
  const int lane = threadIdx.x & 31;
  const bool soft = p.score == MOE_SOFTMAX;
  if (!soft && p.keep < p.groups) moe_close_groups(p, z);
  float vals = 0.f, sum = 0.f, best0 = 0.f;
  int mine = 0;
  for (int k = 0; k < p.top; ++k) {
    float best = -INFINITY;
    int at = kMoeMaxExperts;
    for (int e = lane; e < p.experts; e += 32)
      if (z[e] > best) {
        best = z[e];
        at = e;
      }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oa = __shfl_xor_sync(0xffffffffu, at, o);
      if (ov > best || (ov == best && oa < at)) {
        best = ov;
        at = oa;
      }
    }
    if (at >= p.experts) at = 0;           // nothing left to compare (logits that are not numbers)
    if (k == 0) best0 = best;
    const float ex = soft ? expf(best - best0) : 0.f;
    sum += ex;
    if (lane == (k & 31)) {
      vals = ex;
      mine = at;
    }
    if (lane == 0) z[at] = -INFINITY;
    __syncwarp();
    if ((k & 31) == 31 || k == p.top - 1) {
      const int c = (k & ~31) + lane;
      if (c <= k) {
        const int i = token * p.top + c;
        p.idx[i] = mine;
        p.weight[i] = soft ? vals : moe_sigmoid(raw[mine]);
        p.rank[i] = atomicAdd(&p.counts[mine], 1);
      }
    }
  }
  if (!soft) return;
  __syncwarp();
  for (int c = lane; c < p.top; c += 32) p.weight[token * p.top + c] /= sum;
}

// DOT: one CTA per token computes its logits from h and the router's rows; else logits are given and a warp takes
// a token.
template <typename T, bool DOT>
__global__ void __launch_bounds__(DOT ? 1024 : 256)
    moe_route_kernel(const T* __restrict__ h, long long ldh, const T* __restrict__ router, int dim,
                     const float* __restrict__ logits, long long ldz, const MoeRouteParams p) {
  __shared__ float z[DOT ? 1 : 8][kMoeMaxExperts];
  __shared__ float z_raw[DOT ? kMoeMaxExperts : 1];
  auto choice = [&](float logit, int e) { return p.score == MOE_SOFTMAX ? logit + p.bias[e] : moe_sigmoid(logit) + p.bias[e]; };
  __shared__ int s_last;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if constexpr (DOT) {
    constexpr int V = 16 / sizeof(T);
    const T* x = h + (long long)blockIdx.x * ldh;
    for (int e = warp; e < p.experts; e += 32) {
      const T* w = router + (long long)e * dim;
      float s = 0.f;
#pragma unroll 4
      for (int c = lane * V; c < dim; c += 32 * V) {
        const uint4 a = *reinterpret_cast<const uint4*>(x + c), b = *reinterpret_cast<const uint4*>(w + c);
#pragma unroll
        for (int j = 0; j < V; ++j) s = fmaf(to_f32<T>(reinterpret_cast<const T*>(&a)[j]), to_f32<T>(reinterpret_cast<const T*>(&b)[j]), s);
      }
      s = warp_sum(s);
      if (lane == 0) {
        z[0][e] = choice(s, e);
        z_raw[e] = s;
      }
    }
    __syncthreads();
    if (warp == 0) moe_select(p, z[0], z_raw, blockIdx.x);
  } else {
    const int t = blockIdx.x * 8 + warp;
    if (t < p.tokens) {
      for (int e = lane; e < p.experts; e += 32) z[warp][e] = choice(logits[t * ldz + e], e);
      __syncwarp();
      moe_select(p, z[warp], logits + t * ldz, t);
    }
  }
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) s_last = atomicAdd(&p.counts[p.experts], 1) == (int)gridDim.x - 1;
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  if (warp == 0) {
    int slot = 0, item = 0;
    for (int e0 = 0; e0 < p.experts; e0 += 32) {
      const int e = e0 + lane;
      const int n = e < p.experts ? __ldcg(&p.counts[e]) : 0;
      const int tiles = (n + p.tile - 1) / p.tile;
      const int room = (n + p.align - 1) / p.align * p.align;
      int ns = room, nt = tiles;                    // inclusive sums over the lanes
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int a = __shfl_up_sync(0xffffffffu, ns, o), b = __shfl_up_sync(0xffffffffu, nt, o);
        if (lane >= o) {
          ns += a;
          nt += b;
        }
      }
      const int s0 = slot + ns - room, i0 = item + nt - tiles;
      if (e < p.experts) {
        p.first[e] = s0;
        p.counts[e] = 0;
        for (int i = 0; i < tiles; ++i) p.items[i0 + i] = make_int4(e, s0 + i * p.tile, min(p.tile, n - i * p.tile), 0);
      }
      slot += __shfl_sync(0xffffffffu, ns, 31);
      item += __shfl_sync(0xffffffffu, nt, 31);
    }
    if (lane == 0) {
      *p.n_items = item;
      p.counts[p.experts] = 0;
    }
  }
  if (!p.place) return;
  __threadfence();
  __syncthreads();
  for (int i = threadIdx.x; i < p.tokens * p.top; i += blockDim.x) moe_place(p, i);
}

__global__ void __launch_bounds__(256) moe_place_kernel(const MoeRouteParams p) {
  const int i = blockIdx.x * 256 + threadIdx.x;
  if (i < p.tokens * p.top) moe_place(p, i);
}

// places a token's pairs and copies its row to their slots: one warp per token, 16-byte pieces
__global__ void __launch_bounds__(256)
    moe_sort_kernel(const uint4* __restrict__ h, long long ldh, uint4* __restrict__ sorted, int vecs, const MoeRouteParams p) {
  const int t = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (t >= p.tokens) return;
  for (int k0 = 0; k0 < p.top; k0 += 32) {
    int slot = 0;
    if (k0 + lane < p.top) {
      const int i = t * p.top + k0 + lane;
      moe_place(p, i);
      slot = p.slot_of[i];
    }
    const int n = min(32, p.top - k0);
    for (int c0 = 0; c0 < vecs; c0 += 128) {
      const int c = c0 + lane;
      uint4 v[4];
#pragma unroll
      for (int u = 0; u < 4; ++u)
        if (c + 32 * u < vecs) v[u] = h[t * ldh + c + 32 * u];
      for (int k = 0; k < n; ++k) {
        const long long s = __shfl_sync(0xffffffffu, slot, k);
#pragma unroll
        for (int u = 0; u < 4; ++u)
          if (c + 32 * u < vecs) sorted[s * vecs + c + 32 * u] = v[u];
      }
    }
  }
}

// ---------------------------------------------------------------------------------------------------------
// plain grouped product: 64 outputs x up to 16 slots of one expert per CTA.
//   GLU:  out[slot] = weight[slot] * clamped_unit(gate[e][m] . x[token], up[e][m] . x[token])
//   else: out[slot] = W[e][m] . x[slot]
// ---------------------------------------------------------------------------------------------------------
template <typename T, bool GLU>
__global__ void __launch_bounds__(256)
    moe_plain_kernel(const T* __restrict__ x, long long ldx, const T* __restrict__ w, T* __restrict__ out, long long ldo,
                     const int4* __restrict__ items, const int* __restrict__ n_items, const int* __restrict__ slot_token,
                     const float* __restrict__ slot_weight, int n_in, int n_out, const GluParams glu) {
  constexpr int KT = 32;
  __shared__ float sx[KT][17], sw[GLU ? 2 : 1][KT][65];
  __shared__ long long s_row[16];
  if ((int)blockIdx.y >= *n_items) return;
  const int4 it = items[blockIdx.y];
  const int m0 = blockIdx.x * 64, tid = threadIdx.x;
  if (tid < 16) {
    const int s = it.y + min(tid, it.z - 1);
    s_row[tid] = (long long)(GLU ? slot_token[s] : s) * ldx;
  }
  __syncthreads();
  const T* we = w + (long long)it.x * (GLU ? 2 : 1) * n_out * n_in;
  const int m = tid & 63, q = tid >> 6;      // output, slots q, q + 4, q + 8, q + 12
  float acc[GLU ? 2 : 1][4] = {};
  for (int k0 = 0; k0 < n_in; k0 += KT) {
    for (int i = tid; i < 16 * KT; i += 256) {
      const int k = i % KT, s = i / KT;
      sx[k][s] = k0 + k < n_in ? to_f32<T>(x[s_row[s] + k0 + k]) : 0.f;
    }
    for (int i = tid; i < 64 * KT; i += 256) {
      const int k = i % KT, r = i / KT;
      const bool in = k0 + k < n_in && m0 + r < n_out;
#pragma unroll
      for (int g = 0; g < (GLU ? 2 : 1); ++g)
        sw[g][k][r] = in ? to_f32<T>(we[(GLU ? (long long)((m0 + r) / 32) * 64 + g * 32 + (m0 + r) % 32 : m0 + r) * n_in + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < KT; ++k)
#pragma unroll
      for (int g = 0; g < (GLU ? 2 : 1); ++g)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[g][j] = fmaf(sw[g][k][m], sx[k][q + 4 * j], acc[g][j]);
    __syncthreads();
  }
  if (m0 + m >= n_out) return;
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int s = q + 4 * j;
    if (s >= it.z) continue;
    float v;
    if constexpr (GLU) v = clamped_unit<true>(acc[0][j], acc[1][j], glu) * slot_weight[it.y + s];
    else v = acc[0][j];
    out[(long long)(it.y + s) * ldo + m0 + m] = from_f32<T>(v);
  }
}

}  // namespace rb

#define RB_BY_DTYPE(CALL)                                       \
  if (dtype == rbh::DT_BF16) { using T = __nv_bfloat16; CALL; } \
  else if (dtype == rbh::DT_F32) { using T = float; CALL; }     \
  else return 20;
#define RB_LAUNCH_STATUS()             \
  cudaError_t e_ = cudaGetLastError(); \
  return e_ == cudaSuccess ? 0 : 3000 + (int)e_

extern "C" {

// logits null: they are computed here from h [tokens, dim] and router [experts, dim] (dim a multiple of 8, rows
// 16-byte aligned).  counts: experts + 1 ints, zero before the first call.  items: room for
// min(experts, pairs) + pairs / tile entries of four ints.  An expert's first slot is a multiple of align.  sorted (may
// be null): receives the rows of h by slot (row stride dim).  score 0: softmax over the chosen of logits + bias; 1:
// sigmoid of the logits, chosen by score + bias among the `keep` best of `groups` groups.
int rb_moe_route(int dtype, const void* h, long long ldh, const void* router, int dim, const float* logits, long long ldz,
                 const float* bias, int* counts, int* idx, float* weight, int* rank, int* first, int* items, int* n_items,
                 int* slot_token, float* slot_weight, int* slot_of, void* sorted, int tokens, int experts, int top, int score,
                 int groups, int keep, int tile, int align, void* stream) {
  using namespace rb;
  if (tokens <= 0) return 0;
  if (experts > kMoeMaxExperts || top < 1 || top > experts || tile < 1 || align < 1) return 22;
  if (score != MOE_SOFTMAX && (score != MOE_SIGMOID || groups < 1 || groups > kMoeMaxGroups || experts % groups || keep < 1 ||
                               keep > groups || top > experts / groups * keep))
    return 22;
  if ((!logits || sorted) &&
      (dim % 8 || ldh % 8 || ((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(router) | reinterpret_cast<uintptr_t>(sorted)) & 15)))
    return 21;
  cudaStream_t st = (cudaStream_t)stream;
  const int pairs = tokens * top;
  MoeRouteParams p{bias, score, groups, keep, tokens, experts, top, tile, align, counts, idx, weight, rank, first, (int4*)items, n_items,
                   slot_token, slot_weight, slot_of, pairs <= 4096 && !sorted};
  if (logits) {
    moe_route_kernel<float, false><<<(tokens + 7) / 8, 256, 0, st>>>(nullptr, 0, nullptr, 0, logits, ldz, p);
  } else {
    RB_BY_DTYPE((moe_route_kernel<T, true><<<tokens, 1024, 0, st>>>((const T*)h, ldh, (const T*)router, dim, nullptr, 0, p)))
  }
  if (sorted) {
    const int per = dtype == rbh::DT_F32 ? 4 : 8;
    moe_sort_kernel<<<(tokens + 7) / 8, 256, 0, st>>>((const uint4*)h, ldh / per, (uint4*)sorted, dim / per, p);
  } else if (!p.place) {
    moe_place_kernel<<<(pairs + 255) / 256, 256, 0, st>>>(p);
  }
  RB_LAUNCH_STATUS();
}

// items of at most 16 slots; max_items bounds *n_items.  w: [experts][(2) n_out][n_in]; glu: n_out a multiple of 32
int rb_moe_plain(int dtype, int glu, const void* x, long long ldx, const void* w, void* out, long long ldo, const int* items,
                 const int* n_items, int max_items, const int* slot_token, const float* slot_weight, int n_in, int n_out,
                 float limit, float slope, float shift, void* stream) {
  using namespace rb;
  if (max_items <= 0) return 0;
  if (max_items > 65535 || (glu && n_out % 32)) return 22;
  const dim3 grid((n_out + 63) / 64, max_items);
  const GluParams g{limit, slope, shift};
  cudaStream_t st = (cudaStream_t)stream;
  if (glu) {
    RB_BY_DTYPE((moe_plain_kernel<T, true><<<grid, 256, 0, st>>>((const T*)x, ldx, (const T*)w, (T*)out, ldo, (const int4*)items, n_items, slot_token, slot_weight, n_in, n_out, g)))
  } else {
    RB_BY_DTYPE((moe_plain_kernel<T, false><<<grid, 256, 0, st>>>((const T*)x, ldx, (const T*)w, (T*)out, ldo, (const int4*)items, n_items, slot_token, slot_weight, n_in, n_out, g)))
  }
  RB_LAUNCH_STATUS();
}
}
