// Prompt attention whose heads talk, sm_100a (tcgen05 + TMEM + TMA), over a sliding window and the pages of the cache.
//
// A head's mixed score is one product: s'_h = q'_h . (keys of all key/value heads side by side), with q'_h the rotated
// queries mixed group by group (talk_post_kernel).  So a CTA has one head of up to 128 query rows as in window_prefill.cu and
// needs no other head's scores; what grows is the inner dimension, to kv_heads x dim, and with it the operands:
//
//   * keys come in sub-tiles of 128 keys x 64 numbers, CS at a time, through a ring, one key/value head after the other
//     (products of 64 keys take as long as products of 128);
//   * the first sub-tiles of queries lie in tensor memory as the left operand of the products, which leaves shared memory's
//     room and bandwidth to the keys, the rest in shared memory;
//   * there is one buffer of scores and one of weights (TILE_APART): the scores of the next tile are computed while the softmax
//     works on this one's, and the product with the last tile's values covers the time the scores take into registers.  Where a
//     single CTA's queries leave shared memory no room for that, weights lie over their scores (TILE_ONE) and more queries
//     in tensor memory.
//
//   warp 4      TMA producer: queries in shared memory once, then keys and values tile by tile
//   warp 5      tcgen05 issuer: S = Q' K^T, O += P V
//   warps 0-3   queries into tensor memory, then softmax; a thread owns one query row (attn_tile.cuh)
//
// Two CTAs whose heads share a key/value head may work as a pair (PAIR): keys and values are the same for both, each CTA brings
// half of them (64 keys; 64 numbers of the values) and the products take 256 rows, which halves what comes out of L2 and what a
// tile takes of shared memory.  The first CTA issues for both; full and ready barriers are its own, empty and done ones are each CTA's.
#include "attn_tile.cuh"
#include "pair_common.cuh"

namespace rb {

constexpr int kTpKeys = 128, kTpSlots = 8;     // keys of a tile, most stages of the ring

struct TalkPrefillParams {
  int heads, rep, kv_heads, dim;
  int subs, n_sub, n_tmem;    // sub-tiles of a key, of all keys side by side, of those queries that lie in tensor memory
  int slots, v_slots;         // stages of the ring, of CS sub-tiles each; of values
  int window, block_size, box_rows, max_blocks;
  int row0;                   // query row of the batch that is row 0 of the mixed queries
  float scale_log2;
  const int4* items;          // {first query row, query rows, row of the block table, position of the first query}
  const int* tables;
  const __nv_bfloat16* qmix;  // [rows, heads, kv_heads, dim]
  AttnOut o;
  int* status;
};

template <int VS, int CS, int MODE, bool PAIR>     // 64-column sub-tiles of values, of keys in a stage of the ring
struct TalkPrefillCfg {
  using Cols = AttnTileCols<kTpKeys, MODE>;
  static constexpr int MY_KEYS = PAIR ? kTpKeys / 2 : kTpKeys, MY_VS = PAIR ? VS / 2 : VS;      // what a CTA brings
  static constexpr int SUB = MY_KEYS * 128, STAGE = CS * SUB, Q_SUB = 128 * 128, V_SUB = kTpKeys * 128, V_BYTES = MY_VS * V_SUB;
  static constexpr int IN_TMEM = (512 - Cols::END) / 32;     // sub-tiles of queries
  static constexpr int smem(int q_subs, int slots, int v_slots) { return q_subs * Q_SUB + slots * STAGE + v_slots * V_BYTES + 1024 + 512; }
};

template <int VS, int CS, int MODE, bool PAIR>
__global__ void __launch_bounds__(192, 1)
    talk_prefill_kernel(const __grid_constant__ CUtensorMap tq, const __grid_constant__ CUtensorMap tk,
                        const __grid_constant__ CUtensorMap tv, const TalkPrefillParams p) {
  static_assert(!PAIR || VS == 2);
  using C = TalkPrefillCfg<VS, CS, MODE, PAIR>;
  constexpr bool APART = MODE == TILE_APART;
  constexpr int CTAS = PAIR ? 2 : 1, ARRIVALS = PAIR ? 2 * 4 : 128;      // see attn_arrive
  using T = __nv_bfloat16;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~static_cast<uintptr_t>(1023));
  const int q_subs = p.n_sub - p.n_tmem;
  uint8_t* sQ = smem;
  uint8_t* sV = sQ + q_subs * C::Q_SUB;      // [v_slots]
  uint8_t* sK = sV + p.v_slots * C::V_BYTES; // [slots]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sK + p.slots * C::STAGE);
  uint64_t* q_full = bars;         // shared memory
  uint64_t* q_ready = bars + 1;    // tensor memory
  uint64_t* s_full = bars + 2;
  uint64_t* s_free = bars + 3;
  uint64_t* p_ready = bars + 4;
  uint64_t* pv_done = bars + 5;    // [2]
  uint64_t* v_full = bars + 7;     // [2]
  uint64_t* v_empty = bars + 9;    // [2]
  uint64_t* k_full = bars + 11;    // [slots]
  uint64_t* k_empty = k_full + kTpSlots;
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(k_empty + kTpSlots);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_ptr + 1);

  const int warp_idx = uniform_warp_idx();
  const int lane = threadIdx.x & 31;
  const int h = blockIdx.x;
  const int rank = PAIR ? (int)cluster_ctarank() : 0;
  // a barrier of the first CTA, for arrivals and copies of both
  auto lead = [&](uint64_t* bar) { return PAIR ? map_to_cta(smem_u32(bar), 0) : smem_u32(bar); };
  const int4 it = p.items[blockIdx.y];
  const int q_row0 = it.x, n_q = it.y, pos0 = it.w;
  // keys from the box that holds the first row's oldest key up to the last row's own; at least one tile
  const int key0 = max(0, pos0 - p.window + 1) / p.box_rows * p.box_rows;
  const int n_tiles = (pos0 + n_q - key0 + kTpKeys - 1) / kTpKeys;

  if (threadIdx.x == 0) {
    mbar_init(smem_u32(q_full), 1);
    mbar_init(smem_u32(q_ready), ARRIVALS);
    mbar_init(smem_u32(s_full), 1);
    mbar_init(smem_u32(s_free), ARRIVALS);
    mbar_init(smem_u32(p_ready), ARRIVALS);
    for (int s = 0; s < 2; ++s) {
      mbar_init(smem_u32(&v_full[s]), 1);
      mbar_init(smem_u32(&v_empty[s]), 1);
      mbar_init(smem_u32(&pv_done[s]), 1);
    }
    for (int s = 0; s < p.slots; ++s) {
      mbar_init(smem_u32(&k_full[s]), 1);
      mbar_init(smem_u32(&k_empty[s]), 1);
    }
    *abort_flag = 0;
    fence_barrier_init();
  } else if (threadIdx.x == 128) {
    prefetch_tensormap(&tq);
    prefetch_tensormap(&tk);
    prefetch_tensormap(&tv);
  }
  __syncwarp();
  if constexpr (PAIR) cluster_sync_all();          // barriers of both exist before anything is signalled across
  if (warp_idx == 5) {
    if constexpr (PAIR) {
      tmem_alloc_2cta(smem_u32(tmem_ptr), 512);
      tmem_relinquish_2cta();
    } else {
      tmem_alloc(smem_u32(tmem_ptr), 512);
      tmem_relinquish();
    }
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_ptr;

  if (warp_idx == 4) {
    auto load = [&](uint32_t dst, const CUtensorMap* m, uint32_t bar, int x, int y) {
      if constexpr (PAIR) tma_load_2d_pair(dst, m, bar, x, y);
      else tma_load_2d(dst, m, bar, x, y);
    };
    if (lane == 0 && q_subs) {
      if (rank == 0) mbar_arrive_expect_tx(smem_u32(q_full), CTAS * q_subs * C::Q_SUB);
      const uint32_t bar = lead(q_full);
      for (int s = 0; s < q_subs; ++s) {
        const int x = p.n_tmem + s, c = x / p.subs;
        const uint32_t dst = smem_u32(sQ + s * C::Q_SUB);
        if constexpr (PAIR) tma_load_3d_pair(dst, &tq, bar, (x - c * p.subs) * 64, q_row0 - p.row0, h * p.kv_heads + c);
        else tma_load_3d(dst, &tq, bar, (x - c * p.subs) * 64, q_row0 - p.row0, h * p.kv_heads + c);
      }
    }
    __syncwarp();
    const int* table = p.tables + (long long)it.z * p.max_blocks;
    const int g = h / p.rep, boxes = kTpKeys / p.box_rows;      // at most 16
    // lane x looks up where box x of a tile starts (key/value head 0), ahead of its loads.  Boxes past the last key are
    // masked later; they are read from its page.
    const int last_box = (pos0 + n_q - 1) / p.box_rows * p.box_rows;
    auto lookup = [&](int j) -> int {
      const int t = min(key0 + j * kTpKeys + min(lane, boxes - 1) * p.box_rows, last_box);
      return table[min(t / p.block_size, p.max_blocks - 1)] * p.kv_heads * p.block_size + t % p.block_size;
    };
    bool ok = true;
    int slot = 0, phase = 1;
    auto keys = [&](int rows) {
      for (int s = 0, c = 0, col = 0; s < p.n_sub && ok; s += CS) {
        ok = mbar_wait(smem_u32(&k_empty[slot]), phase, abort_flag, p.status, RB_ERR_TIMEOUT_EMPTY);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        const uint32_t bar = lead(&k_full[slot]), dst = smem_u32(sK + slot * C::STAGE);
        if (lane == 0 && rank == 0) mbar_arrive_expect_tx(smem_u32(&k_full[slot]), CTAS * C::STAGE);
#pragma unroll
        for (int y = 0; y < CS; ++y) {
          for (int x = 0; x < boxes / CTAS; ++x) {
            const int row = __shfl_sync(0xffffffffu, rows, x + rank * (boxes / CTAS)) + c * p.block_size;
            if (lane == 0) load(dst + y * C::SUB + x * p.box_rows * 128, &tk, bar, col, row);
          }
          if ((col += 64) >= p.subs * 64) {
            col = 0;
            ++c;
          }
        }
        if (++slot == p.slots) {
          slot = 0;
          phase ^= 1;
        }
      }
    };
    int v_slot = 0, v_phase = 1;
    auto values = [&](int rows) {
      if (!ok) return;
      ok = mbar_wait(smem_u32(&v_empty[v_slot]), v_phase, abort_flag, p.status, RB_ERR_TIMEOUT_EMPTY);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) return;
      const uint32_t bar = lead(&v_full[v_slot]), dst = smem_u32(sV + v_slot * C::V_BYTES);
      if (lane == 0 && rank == 0) mbar_arrive_expect_tx(smem_u32(&v_full[v_slot]), CTAS * C::V_BYTES);
      for (int x = 0; x < boxes; ++x) {
        const int row = __shfl_sync(0xffffffffu, rows, x) + g * p.block_size;
        if (lane == 0)
          for (int s = 0; s < C::MY_VS; ++s) load(dst + s * C::V_SUB + x * p.box_rows * 128, &tv, bar, (rank + s) * 64, row);
      }
      if (++v_slot == p.v_slots) {
        v_slot = 0;
        v_phase ^= 1;
      }
    };
    // in the order of the products
    int rows = lookup(0), last = 0;
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int next = j + 1 < n_tiles ? lookup(j + 1) : 0;
      keys(rows);
      if (!APART) values(rows);
      else if (j > 0) values(last);
      last = rows;
      rows = next;
    }
    if (APART) values(last);
    if (!ok)
      for (int i = 0; i < 64; ++i) __nanosleep(10000);
  } else if (warp_idx == 5 && rank == 0) {
    constexpr uint32_t idesc_s = make_idesc(UmmaFormat<T>::value, 0, 0, CTAS * 128, kTpKeys);
    constexpr uint32_t idesc_o = make_idesc(UmmaFormat<T>::value, 0, 1, CTAS * 128, VS * 64);
    bool ok = true;
    auto wait = [&](uint64_t* bar, int parity, int code) {
      if constexpr (PAIR) {
        if (ok) ok = mbar_wait_cluster(smem_u32(bar), parity, abort_flag, p.status, code);
      } else {
        if (ok) ok = mbar_wait(smem_u32(bar), parity, abort_flag, p.status, code);
      }
      return ok;
    };
    auto commit = [&](uint64_t* bar) {       // to every CTA
      if constexpr (PAIR) {
        umma_commit_pair_w(smem_u32(bar));
        umma_commit_pair_w(map_to_cta(smem_u32(bar), 1));
      } else {
        umma_commit_w(smem_u32(bar));
      }
    };
    if (q_subs) wait(q_full, 0, RB_ERR_TIMEOUT_FULL);
    if (p.n_tmem) wait(q_ready, 0, RB_ERR_TIMEOUT_FLAG);
    tc_fence_after();
    int slot = 0, phase = 0, v_slot = 0, v_phase = 0;
    auto scores = [&]() {
      // whole sub-tiles of 64 numbers: past the end of a head both operands are zeros
      for (int s = 0; s < p.n_sub; s += CS) {
        if (!wait(&k_full[slot], phase, RB_ERR_TIMEOUT_FULL)) return;
        tc_fence_after();
        const uint64_t k = make_smem_desc_sw128(smem_u32(sK + slot * C::STAGE), 16, 1024);
        if (s < p.n_tmem) {
          const uint32_t q = tmem_base + C::Cols::END + s * 32;
#pragma unroll
          for (int y = 0; y < CS; ++y) {
            if constexpr (PAIR) umma_f16_ts_pair_w4<8, 2>(tmem_base, q + y * 32, k + y * (C::SUB >> 4), idesc_s, s + y != 0);
            else umma_f16_ts_w4<8, 2>(tmem_base, q + y * 32, k + y * (C::SUB >> 4), idesc_s, s + y != 0);
          }
        } else {
          const uint64_t q = make_smem_desc_sw128(smem_u32(sQ + (s - p.n_tmem) * C::Q_SUB), 16, 1024);
#pragma unroll
          for (int y = 0; y < CS; ++y) {
            if constexpr (PAIR) umma_f16_pair_w4<2, 2>(tmem_base, q + y * (C::Q_SUB >> 4), k + y * (C::SUB >> 4), idesc_s, s + y != 0);
            else umma_f16_w4<2, 2>(tmem_base, q + y * (C::Q_SUB >> 4), k + y * (C::SUB >> 4), idesc_s, s + y != 0);
          }
        }
        commit(&k_empty[slot]);
        if (++slot == p.slots) {
          slot = 0;
          phase ^= 1;
        }
      }
      commit(s_full);
    };
    auto values = [&](int j) {
      if (!wait(&v_full[v_slot], v_phase, RB_ERR_TIMEOUT_FULL) || !wait(p_ready, j & 1, RB_ERR_TIMEOUT_FLAG)) return;
      tc_fence_after();
      const uint64_t v = make_smem_desc_sw128(smem_u32(sV + v_slot * C::V_BYTES), C::V_SUB, 1024);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const uint32_t w = tmem_base + C::Cols::P + i * 32;
        if constexpr (PAIR) umma_f16_ts_pair_w4<8, 128>(tmem_base + C::Cols::O, w, v + i * 512, idesc_o, j + i != 0);
        else umma_f16_ts_w4<8, 128>(tmem_base + C::Cols::O, w, v + i * 512, idesc_o, j + i != 0);
      }
      commit(&v_empty[v_slot]);
      commit(&pv_done[j & 1]);
      if (++v_slot == p.v_slots) {
        v_slot = 0;
        v_phase ^= 1;
      }
    };
    scores();
    for (int j = 0; j < n_tiles && ok; ++j) {
      if constexpr (APART) {
        if (j > 0) values(j - 1);
        if (j + 1 == n_tiles) values(j);
        else if (wait(s_free, j & 1, RB_ERR_TIMEOUT_TMEM_EMPTY)) scores();
      } else {
        values(j);
        if (ok && j + 1 < n_tiles) scores();     // over the weights, whose product was issued before and runs before
      }
    }
  } else if (warp_idx < 4) {
    const int t = warp_idx * 32 + lane;            // query row of the tile == TMEM lane
    const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>(warp_idx * 32) << 16);
    for (int s = 0; s < p.n_tmem; ++s) {
      const int c = s / p.subs, col = (s - c * p.subs) * 64;
      const T* src = p.qmix + (((long long)(q_row0 - p.row0 + t) * p.heads + h) * p.kv_heads + c) * p.dim + col;
      uint32_t x[32];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const uint4 v = t < n_q && col + i * 8 < p.dim ? *reinterpret_cast<const uint4*>(src + i * 8) : make_uint4(0, 0, 0, 0);
        x[4 * i] = v.x; x[4 * i + 1] = v.y; x[4 * i + 2] = v.z; x[4 * i + 3] = v.w;
      }
      tmem_st_32x32b_x32(lane_addr + C::Cols::END + s * 32, x);
    }
    if (p.n_tmem) {
      tmem_st_wait();
      tc_fence_before();
      attn_arrive<PAIR>(lead(q_ready));
    }
    const AttnTile a{lane_addr, n_tiles, pos0, n_q, q_row0, p.window, 0, p.scale_log2, smem_u32(s_full), lead(p_ready), smem_u32(pv_done), lead(s_free), abort_flag, p.status};
    AttnRow r;
    const bool ok = attn_tile_softmax<T, VS, kTpKeys, MODE, PAIR>(a, t, [&](int j) { return key0 + j * kTpKeys; }, [](float s) { return s; }, r);
    attn_tile_out<T, VS, kTpKeys, MODE>(a, p.o, h, t, r, ok);
  }

  tc_fence_before();
  __syncwarp();
  if constexpr (PAIR) cluster_sync_all();          // nothing is signalled to a CTA, or read from its memory, after it left
  else __syncthreads();
  if (warp_idx == 5) {
    tc_fence_after();
    if constexpr (PAIR) tmem_dealloc_2cta(tmem_base, 512);
    else tmem_dealloc(tmem_base, 512);
  }
}

template <int VS, int CS, int MODE, bool PAIR>
int launch_talk_prefill(TalkPrefillParams& p, const void* k_pool, const void* v_pool, long long pool_rows, int n_items, int q_rows,
                        cudaStream_t st) {
  using C = TalkPrefillCfg<VS, CS, MODE, PAIR>;
  CUtensorMap tq, tk, tv;
  int rc;
  {
    // [head, key/value head][row][column] with 64-column, 128-row boxes; columns past the extent arrive as zeros
    const uint64_t wide = (uint64_t)p.heads * p.kv_heads;
    uint64_t dims[3] = {(uint64_t)p.dim, (uint64_t)q_rows, wide};
    uint64_t strides[3] = {2, wide * p.dim * 2, (uint64_t)p.dim * 2};
    uint32_t box[3] = {64, 128, 1};
    rc = rbh::encode_tensor_map(&tq, rbh::DT_BF16, 3, const_cast<__nv_bfloat16*>(p.qmix), dims, strides, box, 1);
  }
  auto pool = [&](CUtensorMap* m, const void* base, int cols) {
    uint64_t dims[2] = {(uint64_t)cols, (uint64_t)pool_rows};
    uint64_t strides[2] = {2, (uint64_t)cols * 2};
    uint32_t box[2] = {64, (uint32_t)p.box_rows};
    return rbh::encode_tensor_map(m, rbh::DT_BF16, 2, const_cast<void*>(base), dims, strides, box, 1);
  };
  if (!rc) rc = pool(&tk, k_pool, p.dim);
  if (!rc) rc = pool(&tv, v_pool, p.o.vdim);
  if (rc) return 1000 + rc;
  p.n_tmem = p.n_sub < C::IN_TMEM ? p.n_sub : C::IN_TMEM;
  // as long a ring as fits, with two stages of values if that leaves three of keys
  constexpr int most = 226 * 1024;
  const int q_subs = p.n_sub - p.n_tmem;
  p.v_slots = C::smem(q_subs, 3, 2) <= most ? 2 : 1;
  p.slots = kTpSlots;
  while (p.slots > 1 && C::smem(q_subs, p.slots, p.v_slots) > most) --p.slots;
  const int smem = C::smem(q_subs, p.slots, p.v_slots);
  auto kern = talk_prefill_kernel<VS, CS, MODE, PAIR>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return 2000 + (int)e;
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = dim3(p.heads, n_items);
  cfg.blockDim = dim3(192);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute at[1];
  at[0].id = cudaLaunchAttributeClusterDimension;
  at[0].val.clusterDim.x = PAIR ? 2 : 1; at[0].val.clusterDim.y = 1; at[0].val.clusterDim.z = 1;
  cfg.attrs = at;
  cfg.numAttrs = 1;
  e = cudaLaunchKernelEx(&cfg, kern, tq, tk, tv, (const TalkPrefillParams&)p);
  return e == cudaSuccess ? 0 : 3000 + (int)e;
}

}  // namespace rb

extern "C" {

// What the kernel covers: 16-bit, heads of up to 128 (padded to eights), up to 16 sub-tiles of 64 numbers in the keys of all
// key/value heads, pages that tile 64 keys.
int rb_talk_prefill_ok(int dtype, int heads, int kv_heads, int dim_p, int vdim_p, int block_size) {
  return dtype == rbh::DT_BF16 && dim_p <= 128 && vdim_p <= 128 && dim_p % 8 == 0 && vdim_p % 8 == 0 && kv_heads * ((dim_p + 63) / 64) <= 16 &&
         heads / kv_heads <= 8 && heads * (dim_p + kv_heads * 8) * 4 <= 200 * 1024 &&
         (block_size % 64 == 0 || (block_size >= 8 && 64 % block_size == 0));
}

// qmix: mixed queries of rows row0 .. row0 + q_rows of the batch, [q_rows, heads, kv_heads, dim_p].  Pools [blocks, kv_heads,
// block_size, dim_p | vdim_p].  items: int32 [n_items, 4], see TalkPrefillParams.  All strides are multiples of eight elements.
int rb_talk_prefill(int dtype, const void* qmix, int row0, int q_rows, const void* k_pool, const void* v_pool, int num_blocks,
                    const int* tables, const int* items, int n_items, const float* sink, const void* gate, long long ldg, int gate_kind,
                    void* out, long long ldo, int heads, int kv_heads, int dim_p, int vdim_p, int window, int block_size, int max_blocks,
                    float scale, void* stream) {
  using namespace rb;
  if (n_items <= 0) return 0;
  if (!rb_talk_prefill_ok(dtype, heads, kv_heads, dim_p, vdim_p, block_size) || n_items > 65535 || heads % kv_heads || window < 1 ||
      !(scale > 0.f))
    return 22;
  auto al = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
  if (!al(qmix) || !al(k_pool) || !al(v_pool) || !al(out) || !al(items) || ldo % 8 ||
      (gate && gate_kind == ATTN_GATE_ELEMENT && (!al(gate) || ldg % 8)))
    return 21;
  TalkPrefillParams p{};
  p.heads = heads; p.rep = heads / kv_heads; p.kv_heads = kv_heads; p.dim = dim_p;
  p.subs = (dim_p + 63) / 64; p.n_sub = kv_heads * p.subs;
  p.window = window; p.block_size = block_size; p.max_blocks = max_blocks;
  p.box_rows = block_size % 128 == 0 ? 128 : block_size % 64 == 0 ? 64 : block_size;
  p.row0 = row0; p.scale_log2 = scale * 1.4426950408889634f;
  p.items = (const int4*)items; p.tables = tables; p.qmix = (const __nv_bfloat16*)qmix;
  p.o = AttnOut{sink, gate, gate ? gate_kind : ATTN_GATE_NONE, out, ldg, ldo, vdim_p, 1.0f};
  p.status = rbh::device_status_word();
  const long long pool_rows = (long long)num_blocks * kv_heads * block_size;
  auto go = [&](auto launch) { return launch(p, k_pool, v_pool, pool_rows, n_items, q_rows, (cudaStream_t)stream); };
  // weights apart from the scores while the queries leave room for three stages, as they always do in a pair.  Stages of two
  // sub-tiles where queries in tensor memory and in shared memory are whole stages
  const bool apart = p.n_sub <= 12, even = p.n_sub % 2 == 0;
  if (vdim_p > 64 && p.rep % 2 == 0 && even && p.n_sub > 2) {
    p.box_rows = p.box_rows < 64 ? p.box_rows : 64;
    return go(launch_talk_prefill<2, 2, TILE_APART, true>);
  }
  if (!apart) {
    if (even) return vdim_p <= 64 ? go(launch_talk_prefill<1, 2, TILE_ONE, false>) : go(launch_talk_prefill<2, 2, TILE_ONE, false>);
    return vdim_p <= 64 ? go(launch_talk_prefill<1, 1, TILE_ONE, false>) : go(launch_talk_prefill<2, 1, TILE_ONE, false>);
  }
  if (even) return vdim_p <= 64 ? go(launch_talk_prefill<1, 2, TILE_APART, false>) : go(launch_talk_prefill<2, 2, TILE_APART, false>);
  return vdim_p <= 64 ? go(launch_talk_prefill<1, 1, TILE_APART, false>) : go(launch_talk_prefill<2, 1, TILE_APART, false>);
}
}
