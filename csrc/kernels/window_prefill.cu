// Prompt attention with a sliding window for sm_100a (tcgen05 + TMEM + TMA): keys and values are read straight from
// the pages of the cache, where this step's tokens have been put before; query heads share key/value heads.
//
// The batch is ragged: a work item is a tile of up to 128 query rows of one prompt portion; it sees the keys of its
// own sequence from its first row's window on up to its last row.  One CTA per (item, query head):
//
//   warp 8      TMA producer: Q once, K and V tiles of 128 keys (one page or several) through two-stage rings
//   warp 9      tcgen05 issuer: S = Q K^T into one of two TMEM buffers, O += P V
//   warps 0-3   softmax of the even key tiles, warps 4-7 of the odd ones; a thread owns one query row
//
// P never leaves the tensor memory: a thread reads its row of S, exponentiates it and writes it back packed over the
// columns it came from, where the second product takes it as its A operand.  Even and odd tiles keep separate
// maxima, sums and accumulators that meet at the end, where the head's sink (a number that only enters the
// denominator) joins and the rows are multiplied by the sigmoid of the output gate.
#include "attn_merge.cuh"

namespace rb {

struct WindowPrefillParams {
  int heads, rep;             // query heads, query heads per key/value head
  int kv_heads, vdim;         // vdim: padded to a multiple of 8
  int k_steps;                // 16-wide steps of a key
  int window, block_size, box_rows, max_blocks;
  float scale_log2;
  const int4* items;          // {first query row, query rows, row of the block table, position of the first query}
  const int* tables;
  const float* sink;          // [heads] or null
  const void* gate;           // row t at gate + t * ldg; one number per output number or per head
  int gate_kind;
  void* out;                  // row t, column h * vdim + d
  long long ldg, ldo;
  int* status;
};

template <int KS, int VS>     // 64-column sub-tiles of keys and of values
struct WindowPrefillCfg {
  static constexpr int SUB_BYTES = 128 * 128;
  static constexpr int QK_BYTES = KS * SUB_BYTES;
  static constexpr int V_BYTES = VS * SUB_BYTES;
  static constexpr int SMEM_BYTES = 3 * QK_BYTES + 2 * V_BYTES + 1024 + 256;
  static constexpr int S_COL = 0, O_COL = 256, TMEM_COLS = 512;
};

template <typename T, int KS, int VS>
__global__ void __launch_bounds__(320, 1)
    window_prefill_kernel(const __grid_constant__ CUtensorMap tq, const __grid_constant__ CUtensorMap tk,
                          const __grid_constant__ CUtensorMap tv, const WindowPrefillParams p) {
  using C = WindowPrefillCfg<KS, VS>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~static_cast<uintptr_t>(1023));
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + C::QK_BYTES;            // [2]
  uint8_t* sV = sK + 2 * C::QK_BYTES;        // [2]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sV + 2 * C::V_BYTES);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;     // [2]
  uint64_t* k_empty = bars + 3;    // [2]
  uint64_t* v_full = bars + 5;     // [2]
  uint64_t* v_empty = bars + 7;    // [2]
  uint64_t* s_full = bars + 9;     // [2]
  uint64_t* p_ready = bars + 11;   // [2]
  uint64_t* pv_done = bars + 13;   // [2]
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(bars + 15);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_ptr + 1);

  const int warp_idx = uniform_warp_idx();
  const int lane = threadIdx.x & 31;
  const int h = blockIdx.x;
  const int4 it = p.items[blockIdx.y];
  const int q_row0 = it.x, n_q = it.y, pos0 = it.w;
  // keys from the box that holds the first row's oldest key up to the last row's own; at least one tile
  const int key0 = max(0, pos0 - p.window + 1) / p.box_rows * p.box_rows;
  const int n_tiles = (pos0 + n_q - key0 + 127) / 128;

  if (threadIdx.x == 0) {
    prefetch_tensormap(&tq);
    prefetch_tensormap(&tk);
    prefetch_tensormap(&tv);
    mbar_init(smem_u32(q_full), 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(smem_u32(&k_full[s]), 1);
      mbar_init(smem_u32(&k_empty[s]), 1);
      mbar_init(smem_u32(&v_full[s]), 1);
      mbar_init(smem_u32(&v_empty[s]), 1);
      mbar_init(smem_u32(&s_full[s]), 1);
      mbar_init(smem_u32(&p_ready[s]), 128);
      mbar_init(smem_u32(&pv_done[s]), 1);
    }
    *abort_flag = 0;
    fence_barrier_init();
  }
  if (warp_idx == 9) {
    tmem_alloc(smem_u32(tmem_ptr), C::TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_ptr;

  if (warp_idx == 8) {
    if (lane == 0) {
      mbar_arrive_expect_tx(smem_u32(q_full), C::QK_BYTES);
#pragma unroll
      for (int s = 0; s < KS; ++s)
        tma_load_3d(smem_u32(sQ + s * C::SUB_BYTES), &tq, smem_u32(q_full), s * 64, q_row0, h);
    }
    const int* table = p.tables + (long long)it.z * p.max_blocks;
    const int g = h / p.rep, boxes = 128 / p.box_rows;          // at most 16
    // lane x looks up where box x of a tile starts, one tile ahead of its loads.  Boxes past the last key are
    // masked later; they are read from its page.
    const int last_box = (pos0 + n_q - 1) / p.box_rows * p.box_rows;
    auto lookup = [&](int j) -> int {
      const int t = min(key0 + j * 128 + min(lane, boxes - 1) * p.box_rows, last_box);
      return (table[min(t / p.block_size, p.max_blocks - 1)] * p.kv_heads + g) * p.block_size + t % p.block_size;
    };
    bool ok = true;
    int next_row = lookup(0);
    for (int j = 0; j < n_tiles; ++j) {
      const int st = j & 1;
      const uint32_t ph = (j >> 1) & 1;
      const int my_row = next_row;
      if (j + 1 < n_tiles) next_row = lookup(j + 1);
      ok = mbar_wait(smem_u32(&k_empty[st]), ph ^ 1, abort_flag, p.status, RB_ERR_TIMEOUT_EMPTY);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      const uint32_t kbar = smem_u32(&k_full[st]), vbar = smem_u32(&v_full[st]);
      if (lane == 0) mbar_arrive_expect_tx(kbar, C::QK_BYTES);
      for (int x = 0; x < boxes; ++x) {
        const int row = __shfl_sync(0xffffffffu, my_row, x);
        if (lane == 0)
#pragma unroll
          for (int s = 0; s < KS; ++s)
            tma_load_2d(smem_u32(sK + st * C::QK_BYTES + s * C::SUB_BYTES) + x * p.box_rows * 128, &tk, kbar, s * 64, row);
      }
      ok = mbar_wait(smem_u32(&v_empty[st]), ph ^ 1, abort_flag, p.status, RB_ERR_TIMEOUT_EMPTY);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      if (lane == 0) mbar_arrive_expect_tx(vbar, C::V_BYTES);
      for (int x = 0; x < boxes; ++x) {
        const int row = __shfl_sync(0xffffffffu, my_row, x);
        if (lane == 0)
#pragma unroll
          for (int s = 0; s < VS; ++s)
            tma_load_2d(smem_u32(sV + st * C::V_BYTES + s * C::SUB_BYTES) + x * p.box_rows * 128, &tv, vbar, s * 64, row);
      }
    }
    if (!ok)
      for (int i = 0; i < 64; ++i) __nanosleep(10000);
  } else if (warp_idx == 9) {
    constexpr uint32_t idesc_s = make_idesc(UmmaFormat<T>::value, 0, 0, 128, 128);
    constexpr uint32_t idesc_o = make_idesc(UmmaFormat<T>::value, 0, 1, 128, VS * 64);
    bool ok = mbar_wait(smem_u32(q_full), 0, abort_flag, p.status, RB_ERR_TIMEOUT_FULL);
    auto issue_s = [&](int j) {
      const int st = j & 1;
      const uint32_t q = smem_u32(sQ), k = smem_u32(sK + st * C::QK_BYTES);
      const uint32_t d = tmem_base + C::S_COL + st * 128;
#pragma unroll
      for (int i = 0; i < KS * 4; ++i)
        if (i < p.k_steps) {
          const uint32_t o = (i >> 2) * C::SUB_BYTES + (i & 3) * 32;
          umma_f16_w(d, make_smem_desc_sw128(q + o, 16, 1024), make_smem_desc_sw128(k + o, 16, 1024), idesc_s, i != 0);
        }
      umma_commit_w(smem_u32(&s_full[st]));
      umma_commit_w(smem_u32(&k_empty[st]));
    };
    if (ok) ok = mbar_wait(smem_u32(&k_full[0]), 0, abort_flag, p.status, RB_ERR_TIMEOUT_FULL);
    if (ok) {
      tc_fence_after();
      issue_s(0);
    }
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int st = j & 1;
      if (j + 1 < n_tiles) {
        // S(j+1) goes over P(j-1), whose product was issued before it and runs before it
        ok = mbar_wait(smem_u32(&k_full[st ^ 1]), ((j + 1) >> 1) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_FULL);
        if (!ok) break;
        tc_fence_after();
        issue_s(j + 1);
      }
      ok = mbar_wait(smem_u32(&p_ready[st]), (j >> 1) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_FLAG);
      if (!ok) break;
      ok = mbar_wait(smem_u32(&v_full[st]), (j >> 1) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_FULL);
      if (!ok) break;
      tc_fence_after();
      const uint32_t v = smem_u32(sV + st * C::V_BYTES);
      const uint32_t pt = tmem_base + C::S_COL + st * 128;
      const uint32_t d = tmem_base + C::O_COL + st * 128;
#pragma unroll
      for (int i = 0; i < 8; ++i)
        umma_f16_ts_w(d, pt + i * 8, make_smem_desc_sw128(v + i * 2048, C::SUB_BYTES, 1024), idesc_o,
                      (j >= 2 || i != 0) ? 1u : 0u);
      umma_commit_w(smem_u32(&v_empty[st]));
      umma_commit_w(smem_u32(&pv_done[st]));
    }
  } else {
    const int wg = warp_idx >> 2;
    const int t = (warp_idx & 3) * 32 + lane;      // query row of the tile == TMEM lane
    const int pos = pos0 + t;
    const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>((warp_idx & 3) * 32) << 16);
    const uint32_t s_addr = lane_addr + C::S_COL + wg * 128;
    const uint32_t o_mine = lane_addr + C::O_COL + wg * 128;
    float m_used = -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = wg; j < n_tiles; j += 2) {
      ok = mbar_wait(smem_u32(&s_full[wg]), (j >> 1) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_TMEM_FULL);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
      const int kv0 = key0 + j * 128;
      // a row sees keys (pos - window, pos]; in the middle of a long window no row of the tile has to mask
      const bool need_mask = kv0 + 127 > pos0 || kv0 <= pos0 + n_q - 1 - p.window;
      const int first = pos - p.window + 1 - kv0, last = pos - kv0;      // columns of this tile the row sees
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll 1
      for (int hh = 0; hh < 2; ++hh) {
        uint32_t sreg[2][32];
        tmem_ld_32x32b_x32(s_addr + hh * 64, sreg[0]);
        tmem_ld_32x32b_x32(s_addr + hh * 64 + 32, sreg[1]);
        tmem_ld_wait();
        if (need_mask) {
#pragma unroll
          for (int c = 0; c < 2; ++c)
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (hh * 64 + c * 32 + i <= last && hh * 64 + c * 32 + i >= first) mx4[i & 3] = fmaxf(mx4[i & 3], __uint_as_float(sreg[c][i]));
        } else {
#pragma unroll
          for (int c = 0; c < 2; ++c)
#pragma unroll
            for (int i = 0; i < 32; ++i) mx4[i & 3] = fmaxf(mx4[i & 3], __uint_as_float(sreg[c][i]));
        }
      }
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      const float m_new = fmaxf(m_used, mx * p.scale_log2);
      const bool need = m_new > m_used + 8.0f;
      if (j >= 2) {
        ok = mbar_wait(smem_u32(&pv_done[wg]), ((j - 2) >> 1) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_TMEM_EMPTY);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        tc_fence_after();
      }
      if (__any_sync(0xffffffffu, need)) {         // the TMEM accesses below are warp-wide: uniform branch
        float alpha = 1.0f;
        if (need) {
          alpha = (m_used == -INFINITY) ? 0.0f : fast_exp2(m_used - m_new);
          m_used = m_new;
          l *= alpha;
        }
        if (j >= 2) {
#pragma unroll 1
          for (int c = 0; c < VS * 2; ++c) {
            uint32_t r[32];
            tmem_ld_32x32b_x32(o_mine + c * 32, r);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * alpha);
            tmem_st_32x32b_x32(o_mine + c * 32, r);
          }
          tmem_st_wait();
        }
      }
      const float neg_m = (m_used == -INFINITY) ? 0.f : -m_used;
      float l4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 1
      for (int hh = 0; hh < 2; ++hh) {
        uint32_t sreg[2][32];
        tmem_ld_32x32b_x32(s_addr + hh * 64, sreg[0]);
        tmem_ld_32x32b_x32(s_addr + hh * 64 + 32, sreg[1]);
        tmem_ld_wait();
        uint32_t packed[32];
#pragma unroll
        for (int c = 0; c < 2; ++c)
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            float p0 = fast_exp2(fmaf(__uint_as_float(sreg[c][i]), p.scale_log2, neg_m));
            float p1 = fast_exp2(fmaf(__uint_as_float(sreg[c][i + 1]), p.scale_log2, neg_m));
            if (need_mask) {
              const int k = hh * 64 + c * 32 + i;
              if (k > last || k < first) p0 = 0.f;
              if (k + 1 > last || k + 1 < first) p1 = 0.f;
            }
            l4[(i >> 1) & 3] += p0 + p1;
            packed[c * 16 + (i >> 1)] = pack2<T>(p0, p1);
          }
        // keys [64 hh, 64 hh + 64) packed in pairs over columns [32 hh, 32 hh + 32): columns this thread has
        // already read
        tmem_st_32x32b_x32(s_addr + hh * 32, packed);
      }
      tmem_st_wait();
      l += (l4[0] + l4[1]) + (l4[2] + l4[3]);
      tc_fence_before();
      mbar_arrive(smem_u32(&p_ready[wg]));
    }
    const int last0 = ((n_tiles - 1) & 1) == 0 ? n_tiles - 1 : n_tiles - 2;
    const int last1 = ((n_tiles - 1) & 1) == 1 ? n_tiles - 1 : n_tiles - 2;   // -1: no odd tile
    if (ok) {
      ok = mbar_wait(smem_u32(&pv_done[0]), (last0 >> 1) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_TMEM_EMPTY);
      if (ok && last1 >= 0)
        ok = mbar_wait(smem_u32(&pv_done[1]), (last1 >> 1) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_TMEM_EMPTY);
    }
    ok = __all_sync(0xffffffffu, ok);
    float2* fin = reinterpret_cast<float2*>(sQ);                 // [2][128]; the Q tile is no longer needed
    fin[wg * 128 + t] = make_float2(m_used, l);
    asm volatile("bar.sync 1, 256;" ::: "memory");               // the 8 softmax warps; reached on every path
    if (ok) {
      tc_fence_after();
      const float2 other = fin[(wg ^ 1) * 128 + t];
      const float sk = p.sink ? p.sink[h] * 1.4426950408889634f : -INFINITY;
      const float m_all = fmaxf(fmaxf(m_used, other.x), sk);
      const float f_me = (m_used == -INFINITY) ? 0.f : fast_exp2(m_used - m_all);
      const float f_ot = (other.x == -INFINITY) ? 0.f : fast_exp2(other.x - m_all);
      float l_all = l * f_me + other.y * f_ot;
      if (p.sink) l_all += fast_exp2(sk - m_all);
      const float inv_l = l_all > 0.f ? 1.0f / l_all : 0.f;
      const bool has_odd = last1 >= 0;
      const float w_even = (wg == 0 ? f_me : f_ot) * inv_l;
      const float w_odd = has_odd ? (wg == 0 ? f_ot : f_me) * inv_l : 0.f;
      const long long row = q_row0 + t;
      // warpgroup w writes value columns [w * VS * 32, (w + 1) * VS * 32)
#pragma unroll 1
      for (int c = 0; c < VS; ++c) {
        const int d0 = wg * VS * 32 + c * 32;
        uint32_t re[32], ro[32];
        tmem_ld_32x32b_x32(lane_addr + C::O_COL + d0, re);
        if (has_odd) tmem_ld_32x32b_x32(lane_addr + C::O_COL + 128 + d0, ro);
        tmem_ld_wait();
        if (t < n_q) {
          T* o = reinterpret_cast<T*>(p.out) + row * p.ldo + (long long)h * p.vdim + d0;
          const T* g = reinterpret_cast<const T*>(p.gate) + row * p.ldg + (p.gate_kind == ATTN_GATE_HEAD ? h : (long long)h * p.vdim + d0);
          const float head_gate = p.gate_kind == ATTN_GATE_HEAD ? 1.0f / (1.0f + __expf(-to_f32<T>(*g))) : 1.0f;
          const bool each = p.gate_kind == ATTN_GATE_ELEMENT;
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            if (d0 + q * 8 < p.vdim) {
              uint4 v, gv = make_uint4(0, 0, 0, 0);
              if (each) gv = *reinterpret_cast<const uint4*>(g + q * 8);
              T* e = reinterpret_cast<T*>(&v);
              const T* ge = reinterpret_cast<const T*>(&gv);
#pragma unroll
              for (int i = 0; i < 8; ++i) {
                float val = __uint_as_float(re[q * 8 + i]) * w_even;
                if (has_odd) val += __uint_as_float(ro[q * 8 + i]) * w_odd;
                if (each) val = val / (1.0f + __expf(-to_f32<T>(ge[i])));
                e[i] = from_f32<T>(val * head_gate);
              }
              *reinterpret_cast<uint4*>(o + q * 8) = v;
            }
          }
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp_idx == 9) {
    tc_fence_after();
    tmem_dealloc(tmem_base, C::TMEM_COLS);
  }
}

struct WindowPrefillArgs {
  int dtype;
  const void *q, *k_pool, *v_pool;
  long long ldq;
  int tokens, pool_rows, dim_p, n_items;      // pool_rows: blocks x kv_heads x block_size
};

template <typename T, int KS, int VS>
int launch_window_prefill(const WindowPrefillArgs& a, const WindowPrefillParams& p, cudaStream_t st) {
  using C = WindowPrefillCfg<KS, VS>;
  CUtensorMap tq, tk, tv;
  int rc;
  {
    // [head][row][column] with 64-column, 128-row boxes; columns past the extent arrive as zeros
    uint64_t dims[3] = {(uint64_t)a.dim_p, (uint64_t)a.tokens, (uint64_t)p.heads};
    uint64_t strides[3] = {2, (uint64_t)a.ldq * 2, (uint64_t)a.dim_p * 2};
    uint32_t box[3] = {64, 128, 1};
    rc = rbh::encode_tensor_map(&tq, a.dtype, 3, const_cast<void*>(a.q), dims, strides, box, 1);
  }
  auto pool = [&](CUtensorMap* m, const void* base, int cols) {
    uint64_t dims[2] = {(uint64_t)cols, (uint64_t)a.pool_rows};
    uint64_t strides[2] = {2, (uint64_t)cols * 2};
    uint32_t box[2] = {64, (uint32_t)p.box_rows};
    return rbh::encode_tensor_map(m, a.dtype, 2, const_cast<void*>(base), dims, strides, box, 1);
  };
  if (!rc) rc = pool(&tk, a.k_pool, a.dim_p);
  if (!rc) rc = pool(&tv, a.v_pool, p.vdim);
  if (rc) return 1000 + rc;
  auto kern = window_prefill_kernel<T, KS, VS>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM_BYTES);
  if (e != cudaSuccess) return 2000 + (int)e;
  kern<<<dim3(p.heads, a.n_items), 320, C::SMEM_BYTES, st>>>(tq, tk, tv, p);
  e = cudaGetLastError();
  return e == cudaSuccess ? 0 : 3000 + (int)e;
}

}  // namespace rb

extern "C" {

// What the tensor-core kernel covers: 16-bit, dim and vdim up to 128 (padded to eights), pages that tile 128 keys.
int rb_window_prefill_ok(int dtype, int dim_p, int vdim_p, int block_size) {
  return dtype == rbh::DT_BF16 && dim_p <= 128 && vdim_p <= 128 && dim_p % 8 == 0 && vdim_p % 8 == 0 &&
         (block_size % 128 == 0 || (block_size >= 8 && 128 % block_size == 0));
}

// q: row t, head h at q[t * ldq + h * dim_p].  Pools [blocks, kv_heads, block_size, dim_p | vdim_p].
// items: int32 [n_items, 4], see WindowPrefillParams.  All strides are multiples of eight elements.
int rb_window_prefill(int dtype, const void* q, long long ldq, const void* k_pool, const void* v_pool, int num_blocks,
                      const int* tables, const int* items, int n_items, const float* sink, const void* gate, long long ldg,
                      int gate_kind, void* out, long long ldo, int tokens, int heads, int kv_heads, int dim_p, int vdim_p,
                      int window, int block_size, int max_blocks, float scale, void* stream) {
  using namespace rb;
  if (n_items <= 0) return 0;
  if (!rb_window_prefill_ok(dtype, dim_p, vdim_p, block_size) || n_items > 65535 || heads % kv_heads || window < 1 || !(scale > 0.f))
    return 22;
  auto al = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
  if (!al(q) || !al(k_pool) || !al(v_pool) || !al(out) || !al(items) || ldq % 8 || ldo % 8 ||
      (gate && gate_kind == ATTN_GATE_ELEMENT && (!al(gate) || ldg % 8)))
    return 21;
  WindowPrefillParams p{};
  p.heads = heads; p.rep = heads / kv_heads; p.kv_heads = kv_heads; p.vdim = vdim_p; p.k_steps = (dim_p + 15) / 16;
  p.window = window; p.block_size = block_size; p.box_rows = block_size < 128 ? block_size : 128; p.max_blocks = max_blocks;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.items = (const int4*)items; p.tables = tables; p.sink = sink; p.gate = gate; p.gate_kind = gate ? gate_kind : ATTN_GATE_NONE;
  p.out = out; p.ldg = ldg; p.ldo = ldo; p.status = rbh::device_status_word();
  WindowPrefillArgs a{dtype, q, k_pool, v_pool, ldq, tokens, num_blocks * kv_heads * block_size, dim_p, n_items};
  using T = __nv_bfloat16;
  cudaStream_t st = (cudaStream_t)stream;
  if (dim_p <= 64) return vdim_p <= 64 ? launch_window_prefill<T, 1, 1>(a, p, st) : launch_window_prefill<T, 1, 2>(a, p, st);
  return vdim_p <= 64 ? launch_window_prefill<T, 2, 1>(a, p, st) : launch_window_prefill<T, 2, 2>(a, p, st);
}
}
