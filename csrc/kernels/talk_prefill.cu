// Prompt attention whose heads talk, sm_100a (tcgen05 + TMEM + TMA), over a sliding window and the pages of the cache.
//
// A head's mixed score is one product: s'_h = q'_h . (keys of all key/value heads side by side), with q'_h the rotated
// queries mixed group by group (talk_post_kernel).  So a CTA has one head of up to 128 query rows as in window_prefill.cu and
// needs no other head's scores; what grows is the inner dimension, to kv_heads x dim, and with it the operands:
//
//   * keys come in sub-tiles of 64 keys x 64 numbers through a ring, one key/value head after the other;
//   * up to four sub-tiles of queries lie in shared memory (two CTAs per SM then); with more, the first eight lie in tensor
//     memory as the left operand of the products, which leaves shared memory's bandwidth to the keys, and the rest in
//     shared memory.
//
//   warp 4      TMA producer: queries in shared memory once, then keys and values tile by tile
//   warp 5      tcgen05 issuer: S = Q' K^T into one of two TMEM buffers (S of the next tile while the softmax works on
//               this one), O += P V
//   warps 0-3   queries into tensor memory, then softmax; a thread owns one query row (attn_tile.cuh)
#include "attn_tile.cuh"

namespace rb {

constexpr int kTpSlots = 16, kTpInTmem = 8, kTpQ0 = 256;     // most slots of the ring, sub-tiles of queries in TMEM, their first column

struct TalkPrefillParams {
  int heads, rep, kv_heads, dim;
  int subs, n_sub, n_tmem;    // sub-tiles of a key, of all keys side by side, of those queries that lie in tensor memory
  int slots, tmem_cols;
  int window, block_size, box_rows, max_blocks;
  int row0;                   // query row of the batch that is row 0 of the mixed queries
  float scale_log2;
  const int4* items;          // {first query row, query rows, row of the block table, position of the first query}
  const int* tables;
  const __nv_bfloat16* qmix;  // [rows, heads, kv_heads, dim]
  AttnOut o;
  int* status;
};

template <int VS>             // 64-column sub-tiles of values
struct TalkPrefillCfg {
  static constexpr int SUB = kTileKeys * 128, Q_SUB = 128 * 128, V_BYTES = VS * SUB;
  static constexpr int smem(int q_subs, int slots) { return q_subs * Q_SUB + slots * SUB + 2 * V_BYTES + 1024 + 512; }
};

template <int VS>
__global__ void __launch_bounds__(192, 2)
    talk_prefill_kernel(const __grid_constant__ CUtensorMap tq, const __grid_constant__ CUtensorMap tk,
                        const __grid_constant__ CUtensorMap tv, const TalkPrefillParams p) {
  using C = TalkPrefillCfg<VS>;
  using T = __nv_bfloat16;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~static_cast<uintptr_t>(1023));
  const int q_subs = p.n_sub - p.n_tmem;
  uint8_t* sQ = smem;
  uint8_t* sV = sQ + q_subs * C::Q_SUB;      // [2]
  uint8_t* sK = sV + 2 * C::V_BYTES;         // [slots]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sK + p.slots * C::SUB);
  uint64_t* q_full = bars;         // shared memory
  uint64_t* q_ready = bars + 1;    // tensor memory
  uint64_t* v_full = bars + 2;     // [2]
  uint64_t* v_empty = bars + 4;    // [2]
  uint64_t* s_full = bars + 6;     // [2]
  uint64_t* p_ready = bars + 8;    // [2]: the softmax may be a tile ahead of the values
  uint64_t* pv_done = bars + 10;   // [2]: nobody waits for every one of them, and a parity tells only two phases apart
  uint64_t* k_full = bars + 12;    // [slots]
  uint64_t* k_empty = k_full + kTpSlots;
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(k_empty + kTpSlots);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_ptr + 1);

  const int warp_idx = uniform_warp_idx();
  const int lane = threadIdx.x & 31;
  const int h = blockIdx.x;
  const int4 it = p.items[blockIdx.y];
  const int q_row0 = it.x, n_q = it.y, pos0 = it.w;
  // keys from the box that holds the first row's oldest key up to the last row's own; at least one tile
  const int key0 = max(0, pos0 - p.window + 1) / p.box_rows * p.box_rows;
  const int n_tiles = (pos0 + n_q - key0 + kTileKeys - 1) / kTileKeys;

  if (threadIdx.x == 0) {
    mbar_init(smem_u32(q_full), 1);
    mbar_init(smem_u32(q_ready), 128);
    for (int s = 0; s < 2; ++s) {
      mbar_init(smem_u32(&v_full[s]), 1);
      mbar_init(smem_u32(&v_empty[s]), 1);
      mbar_init(smem_u32(&s_full[s]), 1);
      mbar_init(smem_u32(&p_ready[s]), 128);
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
  if (warp_idx == 5) {
    tmem_alloc(smem_u32(tmem_ptr), p.tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_ptr;

  if (warp_idx == 4) {
    if (lane == 0 && q_subs) {
      mbar_arrive_expect_tx(smem_u32(q_full), q_subs * C::Q_SUB);
      for (int s = 0; s < q_subs; ++s) {
        const int x = p.n_tmem + s, c = x / p.subs;
        tma_load_3d(smem_u32(sQ + s * C::Q_SUB), &tq, smem_u32(q_full), (x - c * p.subs) * 64, q_row0 - p.row0, h * p.kv_heads + c);
      }
    }
    __syncwarp();
    const int* table = p.tables + (long long)it.z * p.max_blocks;
    const int g = h / p.rep, boxes = kTileKeys / p.box_rows;      // at most 8
    // lane x looks up where box x of a tile starts (key/value head 0), ahead of its loads.  Boxes past the last key are
    // masked later; they are read from its page.
    const int last_box = (pos0 + n_q - 1) / p.box_rows * p.box_rows;
    auto lookup = [&](int j) -> int {
      const int t = min(key0 + j * kTileKeys + min(lane, boxes - 1) * p.box_rows, last_box);
      return table[min(t / p.block_size, p.max_blocks - 1)] * p.kv_heads * p.block_size + t % p.block_size;
    };
    bool ok = true;
    int slot = 0, phase = 1, rows = lookup(0);
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int next = j + 1 < n_tiles ? lookup(j + 1) : 0;
      for (int s = 0; s < p.n_sub && ok; ++s) {
        ok = mbar_wait(smem_u32(&k_empty[slot]), phase, abort_flag, p.status, RB_ERR_TIMEOUT_EMPTY);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        const uint32_t bar = smem_u32(&k_full[slot]), dst = smem_u32(sK + slot * C::SUB);
        const int c = s / p.subs, col = (s - c * p.subs) * 64;
        if (lane == 0) mbar_arrive_expect_tx(bar, C::SUB);
        for (int x = 0; x < boxes; ++x) {
          const int row = __shfl_sync(0xffffffffu, rows, x) + c * p.block_size;
          if (lane == 0) tma_load_2d(dst + x * p.box_rows * 128, &tk, bar, col, row);
        }
        if (++slot == p.slots) {
          slot = 0;
          phase ^= 1;
        }
      }
      if (!ok) break;
      const int st = j & 1;
      ok = mbar_wait(smem_u32(&v_empty[st]), ((j >> 1) & 1) ^ 1, abort_flag, p.status, RB_ERR_TIMEOUT_EMPTY);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      const uint32_t bar = smem_u32(&v_full[st]), dst = smem_u32(sV + st * C::V_BYTES);
      if (lane == 0) mbar_arrive_expect_tx(bar, C::V_BYTES);
      for (int x = 0; x < boxes; ++x) {
        const int row = __shfl_sync(0xffffffffu, rows, x) + g * p.block_size;
        if (lane == 0)
          for (int s = 0; s < VS; ++s) tma_load_2d(dst + s * C::SUB + x * p.box_rows * 128, &tv, bar, s * 64, row);
      }
      rows = next;
    }
    if (!ok)
      for (int i = 0; i < 64; ++i) __nanosleep(10000);
  } else if (warp_idx == 5) {
    constexpr uint32_t idesc_s = make_idesc(UmmaFormat<T>::value, 0, 0, 128, kTileKeys);
    constexpr uint32_t idesc_o = make_idesc(UmmaFormat<T>::value, 0, 1, 128, VS * 64);
    bool ok = true;
    if (q_subs) ok = mbar_wait(smem_u32(q_full), 0, abort_flag, p.status, RB_ERR_TIMEOUT_FULL);
    if (ok && p.n_tmem) ok = mbar_wait(smem_u32(q_ready), 0, abort_flag, p.status, RB_ERR_TIMEOUT_FLAG);
    tc_fence_after();
    int slot = 0, phase = 0;
    auto issue_s = [&](int j) {
      const uint32_t d = tmem_base + (j & 1) * kTileKeys;
      // whole sub-tiles of 64 numbers: past the end of a head both operands are zeros
      for (int s = 0; s < p.n_sub; ++s) {
        if (!mbar_wait(smem_u32(&k_full[slot]), phase, abort_flag, p.status, RB_ERR_TIMEOUT_FULL)) return false;
        tc_fence_after();
        const uint64_t k = make_smem_desc_sw128(smem_u32(sK + slot * C::SUB), 16, 1024);
        if (s < p.n_tmem) {
          const uint32_t q = tmem_base + kTpQ0 + s * 32;
#pragma unroll
          for (int i = 0; i < 4; ++i) umma_f16_ts_w(d, q + i * 8, k + 2 * i, idesc_s, s != 0 || i != 0);
        } else {
          umma_f16_w4<2, 2>(d, make_smem_desc_sw128(smem_u32(sQ + (s - p.n_tmem) * C::Q_SUB), 16, 1024), k, idesc_s, s != 0);
        }
        umma_commit_w(smem_u32(&k_empty[slot]));
        if (++slot == p.slots) {
          slot = 0;
          phase ^= 1;
        }
      }
      umma_commit_w(smem_u32(&s_full[j & 1]));
      return true;
    };
    ok = ok && issue_s(0);
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int st = j & 1;
      if (j + 1 < n_tiles && !issue_s(j + 1)) break;      // goes over P(j-1), whose product was issued before and runs before
      ok = mbar_wait(smem_u32(&v_full[st]), (j >> 1) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_FULL);
      if (!ok) break;
      ok = mbar_wait(smem_u32(&p_ready[st]), (j >> 1) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_FLAG);
      if (!ok) break;
      tc_fence_after();
      const uint32_t v = smem_u32(sV + st * C::V_BYTES), pt = tmem_base + st * kTileKeys;
#pragma unroll
      for (int i = 0; i < kTileKeys / 16; ++i)
        umma_f16_ts_w(tmem_base + kTileOut, pt + i * 8, make_smem_desc_sw128(v + i * 2048, C::SUB, 1024), idesc_o,
                      (j != 0 || i != 0) ? 1u : 0u);
      umma_commit_w(smem_u32(&v_empty[st]));
      umma_commit_w(smem_u32(&pv_done[st]));
    }
  } else {
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
      tmem_st_32x32b_x32(lane_addr + kTpQ0 + s * 32, x);
    }
    if (p.n_tmem) {
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(smem_u32(q_ready));
    }
    const AttnTile a{lane_addr, n_tiles, pos0, n_q, q_row0, p.window, 0, p.scale_log2, s_full, p_ready, pv_done, abort_flag, p.status};
    AttnRow r;
    const bool ok = attn_tile_softmax<T, VS>(a, t, [&](int j) { return key0 + j * kTileKeys; }, [](float s) { return s; }, r);
    attn_tile_out<T, VS>(a, p.o, h, t, r, ok);
  }

  tc_fence_before();
  __syncthreads();
  if (warp_idx == 5) {
    tc_fence_after();
    tmem_dealloc(tmem_base, p.tmem_cols);
  }
}

template <int VS>
int launch_talk_prefill(TalkPrefillParams& p, const void* k_pool, const void* v_pool, long long pool_rows, int n_items, int q_rows,
                        cudaStream_t st) {
  using C = TalkPrefillCfg<VS>;
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
  p.n_tmem = p.n_sub <= 4 ? 0 : p.n_sub < kTpInTmem ? p.n_sub : kTpInTmem;
  p.tmem_cols = p.n_tmem ? 512 : 256;
  // two CTAs per SM where the queries leave tensor memory to both, else as long a ring as fits
  const int q_subs = p.n_sub - p.n_tmem, most = p.n_tmem ? 226 * 1024 : 113 * 1024;
  p.slots = kTpSlots;
  while (p.slots > 2 && C::smem(q_subs, p.slots) > most) --p.slots;
  const int smem = C::smem(q_subs, p.slots);
  auto kern = talk_prefill_kernel<VS>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return 2000 + (int)e;
  kern<<<dim3(p.heads, n_items), 192, smem, st>>>(tq, tk, tv, p);
  e = cudaGetLastError();
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
  p.window = window; p.block_size = block_size; p.box_rows = block_size < kTileKeys ? block_size : kTileKeys; p.max_blocks = max_blocks;
  p.row0 = row0; p.scale_log2 = scale * 1.4426950408889634f;
  p.items = (const int4*)items; p.tables = tables; p.qmix = (const __nv_bfloat16*)qmix;
  p.o = AttnOut{sink, gate, gate ? gate_kind : ATTN_GATE_NONE, out, ldg, ldo, vdim_p, 1.0f};
  p.status = rbh::device_status_word();
  const long long pool_rows = (long long)num_blocks * kv_heads * block_size;
  return vdim_p <= 64 ? launch_talk_prefill<1>(p, k_pool, v_pool, pool_rows, n_items, q_rows, (cudaStream_t)stream)
                      : launch_talk_prefill<2>(p, k_pool, v_pool, pool_rows, n_items, q_rows, (cudaStream_t)stream);
}
}
