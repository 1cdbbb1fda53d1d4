// Softmax and output of prompt attention in tiles of 128 query rows x 64 or 128 keys (tcgen05): what the warps that own the
// rows do between the products.  A thread owns one row, its lane of the tensor memory, which holds scores, weights and sums of
// weighted values in one of three arrangements:
//
//   TILE_TWO    scores of tile j in buffer j & 1, weights over the scores they come from
//   TILE_ONE    one buffer of scores, weights over them
//   TILE_APART  one buffer of scores, which is free again as soon as they are in registers, and one of weights
//
// P never leaves the tensor memory: a thread reads its row of S, exponentiates it and writes it back packed, and the second
// product takes it as its A operand.  O is rescaled in place when a row's
// maximum grows by more than 8 (in log2 units), which waits for the products issued so far; otherwise nothing does.
// At the end the head's sink (a number that only enters the denominator) joins and the rows are multiplied by the
// sigmoid of the output gate.
#pragma once
#include "attn_merge.cuh"
#include "pair_common.cuh"

namespace rb {

enum : int { TILE_TWO = 0, TILE_ONE = 1, TILE_APART = 2 };
// columns: scores from 0 on, then weights (TILE_APART), then sums
template <int KEYS, int MODE>
struct AttnTileCols {
  static constexpr int P = MODE == TILE_APART ? KEYS : 0, O = MODE == TILE_TWO ? 2 * KEYS : MODE == TILE_APART ? KEYS + KEYS / 2 : KEYS, END = O + 128;
};

struct AttnTile {
  uint32_t lane_addr;            // tensor memory of this warp's lanes
  int n_tiles, pos0, n_q, q_row0;      // key tiles; position of the first query, queries, row of the first query
  int window, keep;              // a row sees keys (pos - window, pos] and the sequence's first `keep`
  float scale_log2;
  // Barriers (shared-memory addresses; in a pair of CTAs p_ready and s_free are the issuing CTA's): scores are there, weights are
  // there ([2] each with TILE_TWO); products with values of even and odd tiles are through; scores are in registers (TILE_APART)
  uint32_t s_full, p_ready, pv_done, s_free;
  volatile int* abort_flag;
  int* status;
};
struct AttnRow {
  float m = -INFINITY, l = 0.f;  // reference of the exponents (log2 units), sum of weights
};
struct AttnOut {
  const float* sink;             // [heads] or null
  const void* gate;              // row t at gate + t * ldg; one number per output number or per head
  int gate_kind;
  void* out;                     // row t, column h * vdim + d
  long long ldg, ldo;
  int vdim;                      // padded to a multiple of 8
  float out_scale;
};

// A row's thread is through with something (tensor memory, after a fence): 128 arrivals a CTA, four in a pair.
template <bool PAIR>
__device__ __forceinline__ void attn_arrive(uint32_t bar) {
  if constexpr (PAIR) {
    __syncwarp();
    if ((threadIdx.x & 31) == 0) mbar_arrive_tmem_pair(bar);
  } else {
    mbar_arrive(bar);
  }
}

// All tiles of row t (thread t of 128).  key_of(j): first key of tile j; score(s): what becomes of a product before the mask.
// False: a wait ran out.
template <typename T, int VS, int KEYS, int MODE, bool PAIR = false, typename KeyOf, typename Score>
__device__ __forceinline__ bool attn_tile_softmax(const AttnTile& a, int t, KeyOf key_of, Score score, AttnRow& r) {
  using C = AttnTileCols<KEYS, MODE>;
  const int pos = a.pos0 + t;
#pragma unroll 1
  for (int j = 0; j < a.n_tiles; ++j) {
    const int buf = MODE == TILE_TWO ? j & 1 : 0, parity = MODE == TILE_TWO ? (j >> 1) & 1 : j & 1;
    const uint32_t s_addr = a.lane_addr + buf * KEYS;
    bool ok = mbar_wait(a.s_full + buf * 8, parity, a.abort_flag, a.status, RB_ERR_TIMEOUT_TMEM_FULL);
    ok = __all_sync(0xffffffffu, ok);
    if (!ok) return false;
    tc_fence_after();
    uint32_t sreg[KEYS];
#pragma unroll
    for (int i = 0; i < KEYS; i += 32) tmem_ld_32x32b_x32(s_addr + i, sreg + i);
    tmem_ld_wait();
    if constexpr (MODE == TILE_APART) {
      tc_fence_before();
      attn_arrive<PAIR>(a.s_free);
    }
#pragma unroll
    for (int i = 0; i < KEYS; ++i) sreg[i] = __float_as_uint(score(__uint_as_float(sreg[i])));
    const int kv0 = key_of(j);
    // a row sees keys (pos - window, pos] and kept ones; in the middle of a long window no row of the tile has to mask
    if (kv0 + KEYS - 1 > a.pos0 || (kv0 <= a.pos0 + a.n_q - 1 - a.window && kv0 + KEYS > a.keep)) {
      const int first = pos - a.window + 1 - kv0, last = pos - kv0, kept = a.keep - kv0;   // columns the row sees
#pragma unroll
      for (int i = 0; i < KEYS; ++i)
        if ((i < first && i >= kept) || i > last) sreg[i] = 0xff800000u;                   // -infinity
    }
    float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
    for (int i = 0; i < KEYS; ++i) mx[i & 3] = fmaxf(mx[i & 3], __uint_as_float(sreg[i]));
    const float m_new = fmaxf(r.m, fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * a.scale_log2);
    const bool need = m_new > r.m + 8.0f;
    if (__any_sync(0xffffffffu, need)) {         // the TMEM accesses below are warp-wide: uniform branch
      float alpha = 1.0f;
      if (need) {
        alpha = (r.m == -INFINITY) ? 0.0f : fast_exp2(r.m - m_new);
        r.m = m_new;
        r.l *= alpha;
      }
      if (j > 0) {
        ok = mbar_wait(a.pv_done + ((j - 1) & 1) * 8, ((j - 1) >> 1) & 1, a.abort_flag, a.status, RB_ERR_TIMEOUT_TMEM_EMPTY);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) return false;
        tc_fence_after();
#pragma unroll 1
        for (int c = 0; c < VS * 4; ++c) {
          uint32_t x[16];
          tmem_ld_32x32b_x16(a.lane_addr + C::O + c * 16, x);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 16; ++i) x[i] = __float_as_uint(__uint_as_float(x[i]) * alpha);
          tmem_st_32x32b_x16(a.lane_addr + C::O + c * 16, x);
        }
        tmem_st_wait();
      }
    }
    const float neg_m = (r.m == -INFINITY) ? 0.f : -r.m;
    float l4[4] = {0.f, 0.f, 0.f, 0.f};
    uint32_t packed[KEYS / 2];
#pragma unroll
    for (int i = 0; i < KEYS; i += 2) {
      const float p0 = fast_exp2(fmaf(__uint_as_float(sreg[i]), a.scale_log2, neg_m));
      const float p1 = fast_exp2(fmaf(__uint_as_float(sreg[i + 1]), a.scale_log2, neg_m));
      l4[(i >> 1) & 3] += p0 + p1;
      packed[i >> 1] = pack2<T>(p0, p1);
    }
    if constexpr (MODE == TILE_APART) {          // the product with the last weights has read them
      if (j > 0) {
        ok = mbar_wait(a.pv_done + ((j - 1) & 1) * 8, ((j - 1) >> 1) & 1, a.abort_flag, a.status, RB_ERR_TIMEOUT_TMEM_EMPTY);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) return false;
        tc_fence_after();
      }
    }
#pragma unroll
    for (int i = 0; i < KEYS / 2; i += 32) tmem_st_32x32b_x32(s_addr + C::P + i, packed + i);
    tmem_st_wait();
    r.l += (l4[0] + l4[1]) + (l4[2] + l4[3]);
    tc_fence_before();
    attn_arrive<PAIR>(a.p_ready + buf * 8);
  }
  return true;
}

// The row's result; `ok`: every wait so far ended.
template <typename T, int VS, int KEYS, int MODE>
__device__ __forceinline__ void attn_tile_out(const AttnTile& a, const AttnOut& o, int h, int t, const AttnRow& r, bool ok) {
  const float sk = o.sink ? o.sink[h] * 1.4426950408889634f : -INFINITY;
  const long long row = a.q_row0 + t;
  const bool each = o.gate_kind == ATTN_GATE_ELEMENT;
  const T* gate = reinterpret_cast<const T*>(o.gate) + row * o.ldg + (o.gate_kind == ATTN_GATE_HEAD ? h : (long long)h * o.vdim);
  // the gates are on their way while the last product runs
  uint4 gv[VS * 8];
  float head_gate = 1.0f;
  if (t < a.n_q) {
    if (each) {
#pragma unroll
      for (int q = 0; q < VS * 8; ++q)
        if (q * 8 < o.vdim) gv[q] = *reinterpret_cast<const uint4*>(gate + q * 8);
    } else if (o.gate_kind == ATTN_GATE_HEAD) {
      head_gate = sigmoid_f<T>(to_f32<T>(*gate));
    }
  }
  if (ok) ok = mbar_wait(a.pv_done + ((a.n_tiles - 1) & 1) * 8, ((a.n_tiles - 1) >> 1) & 1, a.abort_flag, a.status, RB_ERR_TIMEOUT_TMEM_EMPTY);
  ok = __all_sync(0xffffffffu, ok);
  if (ok) {
    tc_fence_after();
    const float m_all = fmaxf(r.m, sk);
    const float f_me = (r.m == -INFINITY) ? 0.f : fast_exp2(r.m - m_all);
    float l_all = r.l * f_me;
    if (o.sink) l_all += fast_exp2(sk - m_all);
    const float w = l_all > 0.f ? f_me / l_all * head_gate * o.out_scale : 0.f;
    T* dst = reinterpret_cast<T*>(o.out) + row * o.ldo + (long long)h * o.vdim;
#pragma unroll
    for (int c = 0; c < VS * 2; ++c) {
      uint32_t x[32];
      tmem_ld_32x32b_x32(a.lane_addr + AttnTileCols<KEYS, MODE>::O + c * 32, x);
      tmem_ld_wait();
      if (t < a.n_q) {
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          if (c * 32 + q * 8 < o.vdim) {
            uint4 v;
            T* e = reinterpret_cast<T*>(&v);
            const T* ge = reinterpret_cast<const T*>(&gv[c * 4 + q]);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
              float val = __uint_as_float(x[q * 8 + i]) * w;
              if (each) val *= sigmoid_f<T>(to_f32<T>(ge[i]));
              e[i] = from_f32<T>(val);
            }
            *reinterpret_cast<uint4*>(dst + c * 32 + q * 8) = v;
          }
        }
      }
    }
  }
}

}  // namespace rb
