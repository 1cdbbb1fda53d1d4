// Prompt attention with a sliding window for sm_100a (tcgen05 + TMEM + TMA): keys and values are read straight from
// the pages of the cache, where this step's tokens have been put before; query heads share key/value heads.
//
// The batch is ragged: a work item is a tile of up to 128 query rows of one prompt portion; it sees the keys of its
// own sequence from its first row's window on up to its last row.  One CTA per (item, query head), two CTAs per SM so
// that one fills its pipeline, or writes its rows out, while the other computes:
//
//   warp 4      TMA producer: Q once, K and V tiles of 64 keys (one page or several) through two-stage rings
//   warp 5      tcgen05 issuer: S = Q K^T into one of two TMEM buffers (S of the next tile while the softmax works on
//               this one), O += P V
//   warps 0-3   softmax; a thread owns one query row
//
// What happens to the rows between the products is in attn_tile.cuh.
#include <type_traits>

#include "attn_tile.cuh"

namespace rb {

struct WindowPrefillParams {
  int heads, rep;             // query heads, query heads per key/value head
  int kv_heads;
  int window, block_size, box_rows, max_blocks;
  int keep;                   // the first tokens stay visible outside the window
  float scale_log2, cap_in, cap_out;   // CAP: soft cap of unscaled scores, cap_out soft_cap(s, cap_in)
  const int4* items;          // {first query row, query rows, row of the block table, position of the first query}
  const int* tables;
  AttnOut o;
  int* status;
};

constexpr int kWpKeys = 64;

template <int KS, int VS>     // 64-column sub-tiles of keys and of values
struct WindowPrefillCfg {
  static constexpr int Q_SUB = 128 * 128, KV_SUB = kWpKeys * 128;
  static constexpr int Q_BYTES = KS * Q_SUB, K_BYTES = KS * KV_SUB, V_BYTES = VS * KV_SUB;
  static constexpr int SMEM_BYTES = Q_BYTES + 2 * (K_BYTES + V_BYTES) + 1024 + 256;
  static constexpr int S_COL = 0, O_COL = AttnTileCols<kWpKeys, TILE_TWO>::O, TMEM_COLS = 256;
};

template <typename T, int KS, int VS, bool CAP>
__global__ void __launch_bounds__(192, 2)
    window_prefill_kernel(const __grid_constant__ CUtensorMap tq, const __grid_constant__ CUtensorMap tk,
                          const __grid_constant__ CUtensorMap tv, const WindowPrefillParams p) {
  using C = WindowPrefillCfg<KS, VS>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~static_cast<uintptr_t>(1023));
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + C::Q_BYTES;             // [2]
  uint8_t* sV = sK + 2 * C::K_BYTES;         // [2]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sV + 2 * C::V_BYTES);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;     // [2]
  uint64_t* k_empty = bars + 3;    // [2]
  uint64_t* v_full = bars + 5;     // [2]
  uint64_t* v_empty = bars + 7;    // [2]
  uint64_t* s_full = bars + 9;     // [2]
  uint64_t* p_ready = bars + 11;   // [2]: the softmax may be a tile ahead of the values
  uint64_t* pv_done = bars + 13;   // [2]: nobody waits for every one of them, and a parity tells only two phases apart
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(bars + 15);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_ptr + 1);

  const int warp_idx = uniform_warp_idx();
  const int lane = threadIdx.x & 31;
  const int h = blockIdx.x;
  const int4 it = p.items[blockIdx.y];
  const int q_row0 = it.x, n_q = it.y, pos0 = it.w;
  // keys from the box that holds the first row's oldest key up to the last row's own; at least one tile
  const int win0 = max(0, pos0 - p.window + 1) / p.box_rows * p.box_rows;
  // tiles of the kept tokens first; where the window reaches into them there is one run of tiles from token 0 on
  const int n_kept = (min(p.keep, pos0 + 1) + kWpKeys - 1) / kWpKeys;
  const int n_keep = p.keep > 0 && win0 >= n_kept * kWpKeys ? n_kept : 0;
  const int key0 = p.keep > 0 && n_keep == 0 ? 0 : win0;
  const int n_tiles = n_keep + (pos0 + n_q - key0 + kWpKeys - 1) / kWpKeys;
  auto key_of = [&](int j) { return j < n_keep ? j * kWpKeys : key0 + (j - n_keep) * kWpKeys; };

  if (threadIdx.x == 0) {
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
  } else if (threadIdx.x == 128) {
    prefetch_tensormap(&tq);
    prefetch_tensormap(&tk);
    prefetch_tensormap(&tv);
  }
  if (warp_idx == 5) {
    tmem_alloc(smem_u32(tmem_ptr), C::TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_ptr;

  if (warp_idx == 4) {
    if (lane == 0) {
      mbar_arrive_expect_tx(smem_u32(q_full), C::Q_BYTES);
#pragma unroll
      for (int s = 0; s < KS; ++s)
        tma_load_3d(smem_u32(sQ + s * C::Q_SUB), &tq, smem_u32(q_full), s * 64, q_row0, h);
    }
    const int* table = p.tables + (long long)it.z * p.max_blocks;
    const int g = h / p.rep, boxes = kWpKeys / p.box_rows;      // at most 8
    // lane x looks up where box x of a tile starts, ahead of its loads.  Boxes past the last key are
    // masked later; they are read from its page.
    const int last_box = (pos0 + n_q - 1) / p.box_rows * p.box_rows;
    auto lookup = [&](int j) -> int {
      const int t = min(key_of(j) + min(lane, boxes - 1) * p.box_rows, last_box);
      return (table[min(t / p.block_size, p.max_blocks - 1)] * p.kv_heads + g) * p.block_size + t % p.block_size;
    };
    // one tile of keys (or values) into its stage once the products on the one before are through
    auto bring = [&](const CUtensorMap* m, uint64_t* full, uint64_t* empty, uint8_t* ring, int stage_bytes, int subs, int j, int rows) {
      const int st = j & 1;
      bool go = mbar_wait(smem_u32(&empty[st]), ((j >> 1) & 1) ^ 1, abort_flag, p.status, RB_ERR_TIMEOUT_EMPTY);
      go = __all_sync(0xffffffffu, go);
      if (!go) return false;
      const uint32_t bar = smem_u32(&full[st]), dst = smem_u32(ring + st * stage_bytes);
      if (lane == 0) mbar_arrive_expect_tx(bar, stage_bytes);
      for (int x = 0; x < boxes; ++x) {
        const int row = __shfl_sync(0xffffffffu, rows, x);
        if (lane == 0)
          for (int s = 0; s < subs; ++s) tma_load_2d(dst + s * C::KV_SUB + x * p.box_rows * 128, m, bar, s * 64, row);
      }
      return true;
    };
    // keys go a tile ahead of values, whose stage is free only after a later product
    int row = lookup(0), next_row = n_tiles > 1 ? lookup(1) : row;
    bool ok = bring(&tk, k_full, k_empty, sK, C::K_BYTES, KS, 0, row);
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int after = j + 2 < n_tiles ? lookup(j + 2) : 0;
      if (j + 1 < n_tiles) ok = bring(&tk, k_full, k_empty, sK, C::K_BYTES, KS, j + 1, next_row);
      if (ok) ok = bring(&tv, v_full, v_empty, sV, C::V_BYTES, VS, j, row);
      row = next_row;
      next_row = after;
    }
    if (!ok)
      for (int i = 0; i < 64; ++i) __nanosleep(10000);
  } else if (warp_idx == 5) {
    constexpr uint32_t idesc_s = make_idesc(UmmaFormat<T>::value, 0, 0, 128, kWpKeys);
    constexpr uint32_t idesc_o = make_idesc(UmmaFormat<T>::value, 0, 1, 128, VS * 64);
    bool ok = mbar_wait(smem_u32(q_full), 0, abort_flag, p.status, RB_ERR_TIMEOUT_FULL);
    auto issue_s = [&](int j) {
      const int st = j & 1;
      const uint64_t q = make_smem_desc_sw128(smem_u32(sQ), 16, 1024);
      const uint64_t k = make_smem_desc_sw128(smem_u32(sK + st * C::K_BYTES), 16, 1024);
      const uint32_t d = tmem_base + C::S_COL + st * kWpKeys;
      // whole sub-tiles of 64 numbers: past the end of a head both operands are zeros
#pragma unroll
      for (int s = 0; s < KS; ++s)
        umma_f16_w4<2, 2>(d, q + s * (C::Q_SUB >> 4), k + s * (C::KV_SUB >> 4), idesc_s, s != 0);
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
      ok = mbar_wait(smem_u32(&v_full[st]), (j >> 1) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_FULL);
      if (!ok) break;
      ok = mbar_wait(smem_u32(&p_ready[st]), (j >> 1) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_FLAG);
      if (!ok) break;
      tc_fence_after();
      const uint32_t v = smem_u32(sV + st * C::V_BYTES);
      const uint32_t pt = tmem_base + C::S_COL + st * kWpKeys;
#pragma unroll
      for (int i = 0; i < kWpKeys / 16; ++i)
        umma_f16_ts_w(tmem_base + C::O_COL, pt + i * 8, make_smem_desc_sw128(v + i * 2048, C::KV_SUB, 1024), idesc_o,
                      (j != 0 || i != 0) ? 1u : 0u);
      umma_commit_w(smem_u32(&v_empty[st]));
      umma_commit_w(smem_u32(&pv_done[st]));
    }
  } else {
    const int t = warp_idx * 32 + lane;            // query row of the tile == TMEM lane
    const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>(warp_idx * 32) << 16);
    const AttnTile a{lane_addr, n_tiles, pos0, n_q, q_row0, p.window, p.keep, p.scale_log2, smem_u32(s_full), smem_u32(p_ready), smem_u32(pv_done), 0, abort_flag, p.status};
    AttnRow r;
    const bool ok = attn_tile_softmax<T, VS, kWpKeys, TILE_TWO>(a, t, key_of, [&](float s) { return CAP ? soft_cap(s, p.cap_in, p.cap_out) : s; }, r);
    attn_tile_out<T, VS, kWpKeys, TILE_TWO>(a, p.o, h, t, r, ok);
  }

  tc_fence_before();
  __syncthreads();
  if (warp_idx == 5) {
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

template <typename T, int KS, int VS, bool CAP>
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
  if (!rc) rc = pool(&tv, a.v_pool, p.o.vdim);
  if (rc) return 1000 + rc;
  auto kern = window_prefill_kernel<T, KS, VS, CAP>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM_BYTES);
  if (e != cudaSuccess) return 2000 + (int)e;
  kern<<<dim3(p.heads, a.n_items), 192, C::SMEM_BYTES, st>>>(tq, tk, tv, p);
  e = cudaGetLastError();
  return e == cudaSuccess ? 0 : 3000 + (int)e;
}

}  // namespace rb

extern "C" {

// What the tensor-core kernel covers: 16-bit, dim and vdim up to 128 (padded to eights), pages that tile 64 keys.
int rb_window_prefill_ok(int dtype, int dim_p, int vdim_p, int block_size) {
  return dtype == rbh::DT_BF16 && dim_p <= 128 && vdim_p <= 128 && dim_p % 8 == 0 && vdim_p % 8 == 0 &&
         (block_size % 64 == 0 || (block_size >= 8 && 64 % block_size == 0));
}

// q: row t, head h at q[t * ldq + h * dim_p].  Pools [blocks, kv_heads, block_size, dim_p | vdim_p].
// items: int32 [n_items, 4], see WindowPrefillParams.  All strides are multiples of eight elements.
int rb_window_prefill(int dtype, const void* q, long long ldq, const void* k_pool, const void* v_pool, int num_blocks,
                      const int* tables, const int* items, int n_items, const float* sink, const void* gate, long long ldg,
                      int gate_kind, void* out, long long ldo, int tokens, int heads, int kv_heads, int dim_p, int vdim_p,
                      int window, int keep, int block_size, int max_blocks, float scale, float cap, float out_scale,
                      void* stream) {
  using namespace rb;
  if (n_items <= 0) return 0;
  if (!rb_window_prefill_ok(dtype, dim_p, vdim_p, block_size) || n_items > 65535 || heads % kv_heads || window < 1 || keep < 0 || !(scale > 0.f))
    return 22;
  auto al = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
  if (!al(q) || !al(k_pool) || !al(v_pool) || !al(out) || !al(items) || ldq % 8 || ldo % 8 ||
      (gate && gate_kind == ATTN_GATE_ELEMENT && (!al(gate) || ldg % 8)))
    return 21;
  WindowPrefillParams p{};
  p.heads = heads; p.rep = heads / kv_heads; p.kv_heads = kv_heads;
  p.window = window; p.block_size = block_size; p.box_rows = block_size < kWpKeys ? block_size : kWpKeys; p.max_blocks = max_blocks;
  p.scale_log2 = scale * 1.4426950408889634f; p.keep = keep;
  if (cap > 0.f) {
    p.cap_in = 2.8853900817779268f * scale / cap;      // 2 log2(e) / cap on scaled scores
    p.cap_out = cap / scale;
  }
  p.items = (const int4*)items; p.tables = tables; 
  p.o = AttnOut{sink, gate, gate ? gate_kind : ATTN_GATE_NONE, out, ldg, ldo, vdim_p, out_scale}; p.status = rbh::device_status_word();
  WindowPrefillArgs a{dtype, q, k_pool, v_pool, ldq, tokens, num_blocks * kv_heads * block_size, dim_p, n_items};
  using T = __nv_bfloat16;
  cudaStream_t st = (cudaStream_t)stream;
  auto by_size = [&](auto capped) {
    constexpr bool CAP = decltype(capped)::value;
    if (dim_p <= 64) return vdim_p <= 64 ? launch_window_prefill<T, 1, 1, CAP>(a, p, st) : launch_window_prefill<T, 1, 2, CAP>(a, p, st);
    return vdim_p <= 64 ? launch_window_prefill<T, 2, 1, CAP>(a, p, st) : launch_window_prefill<T, 2, 2, CAP>(a, p, st);
  };
  return cap > 0.f ? by_size(std::true_type{}) : by_size(std::false_type{});
}
}
