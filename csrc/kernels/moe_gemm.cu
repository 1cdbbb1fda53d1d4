// Grouped products of a mixture of experts on the tensor cores, sm_100a (tcgen05 + TMEM + TMA).
//
// moe_gemm_kernel: few tokens per expert.  The weights lie on the M side and the tokens of one expert on the N side,
// 16 to 128 of them, so a decoded batch with one token per expert is bound by the weights' bytes and nothing else.
// A CTA keeps two accumulators of 128 weight rows that share every token tile:
//
//   GLU:  gate rows and up rows; the epilogue writes weight * clamped_unit(gate, up) to the expert's slots.  A small
//         batch's rows are gathered by TMA straight from the normed activations (tile::gather4, four row numbers a copy),
//         a large one's have been sorted by slot
//   down: two neighbouring blocks of 128 rows
//
//   warps 0-7   epilogue (a quarter of the lanes each, the columns in two halves)
//   warp 8      TMA producer, one gather per lane
//   warp 9      tcgen05 issuer
//
// moe_pair_kernel: many tokens per expert.  The activations have been sorted by expert, each expert's rows starting at
// a multiple of 256, so the product is the CTA-pair GEMM (gemm_pair.cuh) with the weights of a row tile chosen by its
// expert.
#include "gemm_pair_launch.cuh"

namespace rb {

struct MoeGemmParams {
  const int4* items;             // {expert, first slot, slots}
  const int* n_items;
  const int* slot_token;         // GLU
  const float* slot_weight;      // GLU
  void* out;                     // row = slot
  long long ldo;
  int n_in, n_out;               // n_out: rows of one block (the gates, the ups, or all of them)
  GluParams glu;
  int* status;
};

template <int NT>
struct MoeGemmCfg {
  static constexpr int A_BYTES = 2 * 128 * 128, B_BYTES = NT * 128;
  static constexpr int STAGE = A_BYTES + B_BYTES;
  static constexpr int STAGES = (200 * 1024) / STAGE;
  static constexpr int SMEM_BYTES = STAGES * STAGE + 1024 + 256;
  static constexpr int TMEM_COLS = 2 * NT < 32 ? 32 : 2 * NT;
};

// four rows of 64 columns each
__device__ __forceinline__ void tma_gather4(uint32_t dst, const CUtensorMap* m, uint32_t bar, int x, int y0, int y1, int y2, int y3) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cta.global.tile::gather4.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5, %6, %7}], [%2];" ::"r"(dst),
      "l"(reinterpret_cast<uint64_t>(m)), "r"(bar), "r"(x), "r"(y0), "r"(y1), "r"(y2), "r"(y3)
      : "memory");
}

template <typename T, int NT, bool GLU, bool GATHER>
__global__ void __launch_bounds__(320, 1)
    moe_gemm_kernel(const __grid_constant__ CUtensorMap tw, const __grid_constant__ CUtensorMap tx, const MoeGemmParams p) {
  using C = MoeGemmCfg<NT>;
  if ((int)blockIdx.y >= *p.n_items) return;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~static_cast<uintptr_t>(1023));
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + C::STAGES * C::STAGE);
  uint64_t* empty = full + C::STAGES;
  uint64_t* done = empty + C::STAGES;
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(done + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_ptr + 1);
  const int warp_idx = uniform_warp_idx();
  const int lane = threadIdx.x & 31;
  const int4 it = p.items[blockIdx.y];
  const int m0 = blockIdx.x * (GLU ? 128 : 256);
  // first row of the two blocks in the weights of all experts (GLU: in units of 32, which gates and ups take in
  // turns); what runs past an expert's end is not written
  const int row0 = GLU ? (it.x * p.n_out + m0) / 32 : it.x * p.n_out + m0;
  const int num_kb = (p.n_in + 63) / 64;
  if (threadIdx.x == 0) {
    prefetch_tensormap(&tw);
    prefetch_tensormap(&tx);
    for (int s = 0; s < C::STAGES; ++s) {
      mbar_init(smem_u32(&full[s]), 1);
      mbar_init(smem_u32(&empty[s]), 1);
    }
    mbar_init(smem_u32(done), 1);
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
    constexpr int GATHERS = (NT / 4 + 31) / 32;      // per lane and stage
    int y[GATHERS][4];
    if constexpr (GATHER) {
#pragma unroll
      for (int i = 0; i < GATHERS; ++i)
#pragma unroll
        for (int k = 0; k < 4; ++k) y[i][k] = p.slot_token[it.y + min((i * 32 + lane) * 4 + k, it.z - 1)];
    }
    bool ok = true;
    for (int kb = 0; kb < num_kb; ++kb) {
      const int st = kb % C::STAGES;
      ok = mbar_wait(smem_u32(&empty[st]), ((kb / C::STAGES) & 1) ^ 1, abort_flag, p.status, RB_ERR_TIMEOUT_EMPTY);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      const uint32_t bar = smem_u32(&full[st]);
      const uint32_t a = smem_u32(smem + st * C::STAGE), b = a + C::A_BYTES;
      if (lane == 0) {
        mbar_arrive_expect_tx(bar, C::STAGE);
        if constexpr (GLU) {
          tma_load_4d(a, &tw, bar, kb * 64, 0, 0, row0);
          tma_load_4d(a + 128 * 128, &tw, bar, kb * 64, 0, 1, row0);
        } else {
          tma_load_2d(a, &tw, bar, kb * 64, row0);
          tma_load_2d(a + 128 * 128, &tw, bar, kb * 64, row0 + 128);
        }
        if constexpr (!GATHER) tma_load_2d(b, &tx, bar, kb * 64, it.y);
      }
      __syncwarp();
      if constexpr (GATHER) {
#pragma unroll
        for (int i = 0; i < GATHERS; ++i)
          if ((i * 32 + lane) * 4 < NT) tma_gather4(b + (i * 32 + lane) * 512, &tx, bar, kb * 64, y[i][0], y[i][1], y[i][2], y[i][3]);
      }
    }
    if (!ok)
      for (int i = 0; i < 64; ++i) __nanosleep(10000);
  } else if (warp_idx == 9) {
    constexpr uint32_t idesc = make_idesc(UmmaFormat<T>::value, 0, 0, 128, NT);
    bool ok = true;
    for (int kb = 0; kb < num_kb; ++kb) {
      const int st = kb % C::STAGES;
      ok = mbar_wait(smem_u32(&full[st]), (kb / C::STAGES) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_FULL);
      if (!ok) break;
      tc_fence_after();
      const uint64_t a = make_smem_desc_sw128(smem_u32(smem + st * C::STAGE), 16, 1024);
      const uint64_t b = make_smem_desc_sw128(smem_u32(smem + st * C::STAGE + C::A_BYTES), 16, 1024);
      umma_f16_w4<2, 2>(tmem_base, a, b, idesc, kb != 0);
      umma_f16_w4<2, 2>(tmem_base + NT, a + (128 * 128 >> 4), b, idesc, kb != 0);
      umma_commit_w(smem_u32(&empty[st]));
    }
    if (ok) umma_commit_w(smem_u32(done));
  } else {
    constexpr int COLS = NT >= 32 ? NT / 2 : NT;     // columns per warp
    const int quarter = warp_idx & 3, half = warp_idx >> 2;
    const int m = m0 + quarter * 32 + lane;
    const uint32_t addr = tmem_base + (static_cast<uint32_t>(quarter * 32) << 16);
    T* o = reinterpret_cast<T*>(p.out) + it.y * p.ldo + m;
    bool ok = mbar_wait(smem_u32(done), 0, abort_flag, p.status, RB_ERR_TIMEOUT_TMEM_FULL);
    ok = __all_sync(0xffffffffu, ok);
    if (ok && half * COLS < NT) {
      tc_fence_after();
#pragma unroll 1
      for (int c = half * COLS; c < (half + 1) * COLS && c < it.z; c += 16) {
        uint32_t r0[16], r1[16];
        tmem_ld_32x32b_x16(addr + c, r0);
        tmem_ld_32x32b_x16(addr + NT + c, r1);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 16; ++i)
          if (c + i < it.z) {
            const float u = __uint_as_float(r0[i]), v = __uint_as_float(r1[i]);
            T* row = o + (long long)(c + i) * p.ldo;
            if constexpr (GLU) {
              if (m < p.n_out) *row = from_f32<T>(clamped_unit_fast(u, v, p.glu) * p.slot_weight[it.y + c + i]);
            } else {
              if (m < p.n_out) *row = from_f32<T>(u);
              if (m + 128 < p.n_out) row[128] = from_f32<T>(v);
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

template <typename T, int NT, bool GLU, bool GATHER>
int launch_moe_gemm(int dtype, const void* x, long long ldx, int x_rows, const void* w, int experts, int max_items,
                    const MoeGemmParams& p, cudaStream_t st) {
  using C = MoeGemmCfg<NT>;
  CUtensorMap tw, tx;
  auto map = [&](CUtensorMap* m, const void* base, long long rows, long long ld, int box_rows) {
    uint64_t dims[2] = {(uint64_t)p.n_in, (uint64_t)rows};
    uint64_t strides[2] = {2, (uint64_t)ld * 2};
    uint32_t box[2] = {64, (uint32_t)box_rows};
    return rbh::encode_tensor_map(m, dtype, 2, const_cast<void*>(base), dims, strides, box, 1);
  };
  int rc;
  if (GLU) {
    // [block of 32 gates + 32 ups][gate or up][32 rows][n_in]: a box takes the gates (or ups) of four blocks
    uint64_t dims[4] = {(uint64_t)p.n_in, 32, 2, (uint64_t)experts * p.n_out / 32};
    uint64_t strides[4] = {2, (uint64_t)p.n_in * 2, (uint64_t)p.n_in * 64, (uint64_t)p.n_in * 128};
    uint32_t box[4] = {64, 32, 1, 4};
    rc = rbh::encode_tensor_map(&tw, dtype, 4, const_cast<void*>(w), dims, strides, box, 1);
  } else {
    rc = map(&tw, w, (long long)experts * p.n_out, p.n_in, 128);
  }
  if (!rc) rc = map(&tx, x, x_rows, ldx, GATHER ? 1 : NT);        // a gathering map's box is one row high
  if (rc) return 1000 + rc;
  auto kern = moe_gemm_kernel<T, NT, GLU, GATHER>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM_BYTES);
  if (e != cudaSuccess) return 2000 + (int)e;
  const int mt = GLU ? 128 : 256;
  kern<<<dim3((p.n_out + mt - 1) / mt, max_items), 320, C::SMEM_BYTES, st>>>(tw, tx, p);
  e = cudaGetLastError();
  return e == cudaSuccess ? 0 : 3000 + (int)e;
}

template <bool GLU, bool GATHER>
int moe_gemm_by_tile(int tile, int dtype, const void* x, long long ldx, int x_rows, const void* w, int experts, int max_items,
                     const MoeGemmParams& p, cudaStream_t st) {
  using T = __nv_bfloat16;
  switch (tile) {
    case 16: return launch_moe_gemm<T, 16, GLU, GATHER>(dtype, x, ldx, x_rows, w, experts, max_items, p, st);
    case 32: return launch_moe_gemm<T, 32, GLU, GATHER>(dtype, x, ldx, x_rows, w, experts, max_items, p, st);
    case 64: return launch_moe_gemm<T, 64, GLU, GATHER>(dtype, x, ldx, x_rows, w, experts, max_items, p, st);
    case 128: return launch_moe_gemm<T, 128, GLU, GATHER>(dtype, x, ldx, x_rows, w, experts, max_items, p, st);
  }
  return 22;
}

// ---------------------------------------------------------------------------------------------------------
// many tokens per expert: row tile i of the sorted activations belongs to item i
// ---------------------------------------------------------------------------------------------------------
struct MoeHooks : NoHooks {
  static constexpr bool kGrouped = true;
  const int4* items;
  const int* n_items;
  const float* slot_weight;
  int rows_per_expert;           // rows of B
  GluParams glu;
  __device__ __forceinline__ int num_m() const { return *n_items; }
  __device__ __forceinline__ int b_row(int m_idx) const { return items[m_idx].x * rows_per_expert; }
  __device__ __forceinline__ float row_scale(long long row) const { return slot_weight[row]; }
};

template <typename T, int EPI>
__global__ void __cluster_dims__(2, 1, 1) __launch_bounds__(G2_THREADS, 1)
    moe_pair_kernel(const __grid_constant__ CUtensorMap tma_a, const __grid_constant__ CUtensorMap tma_b,
                    const __grid_constant__ CUtensorMap tma_c, const GemmParams p, const MoeHooks hooks) {
  extern __shared__ uint8_t smem_raw[];
  gemm_pair_body<T, 1, EPI, false, false, MoeHooks>(&tma_a, &tma_b, &tma_c, p, hooks, smem_raw, blockIdx.x / 2, gridDim.x / 2);
}

template <typename T, int EPI>
int launch_moe_pair(GemmArgs a, const MoeHooks& hooks, int experts, cudaStream_t st) {
  using C = PairCfg<1>;
  CUtensorMap ta, tb, tc;
  GemmArgs maps = a;
  maps.p.N = experts * hooks.rows_per_expert;
  int rc = make_pair_operand_maps<T, false, false>(maps, &ta, &tb);
  maps.p.N = EPI == EPI_GLU ? a.p.N / 2 : a.p.N;
  if (!rc) rc = make_pair_output_map(maps.p, a.dtype, &tc);
  if (rc) return 1000 + rc;
  auto kern = moe_pair_kernel<T, EPI>;
  static int resident = 0;
  if (resident == 0) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM_BYTES);
    if (e != cudaSuccess) return 2000 + (int)e;
    resident = max_resident_clusters(kern, C::SMEM_BYTES);
  }
  const long long tiles = (long long)(a.p.M / C::BM) * ((a.p.N + G2_BN - 1) / G2_BN);
  const int clusters = tiles < resident ? (int)tiles : resident;
  kern<<<2 * clusters, G2_THREADS, C::SMEM_BYTES, st>>>(ta, tb, tc, a.p, hooks);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : 3000 + (int)e;
}

}  // namespace rb

extern "C" {

// The products over sorted rows: x [max_items * 256, n_in] by slot, w as in rb_moe_gemm, out the same rows.  Rows of a
// tile that belong to no slot are computed from whatever x holds there.
int rb_moe_pair(int dtype, int glu, const void* x, long long ldx, const void* w, int experts, void* out, long long ldo,
                const int* items, const int* n_items, int max_items, const float* slot_weight, int n_in, int n_out, float limit,
                float slope, float shift, void* stream) {
  using namespace rb;
  if (max_items <= 0) return 0;
  auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  if (dtype != rbh::DT_BF16 || (glu && n_out % 32)) return 22;
  if (!al(x) || !al(w) || !al(out) || !al(items) || ldx % 8 || n_in % 8 || ldo % 8) return 21;
  GemmArgs a{};
  a.dtype = dtype; a.A = x; a.lda = ldx; a.B = w; a.ldb = n_in; a.stream = (cudaStream_t)stream;
  GemmParams& p = a.p;
  p.M = max_items * 256; p.N = glu ? 2 * n_out : n_out; p.K = n_in; p.out = out; p.ldc = ldo; p.alpha = 1.0f; p.vec_ok = 1;
  p.tma_store = 1; p.split_k = 1; p.group_m = 4; p.status = rbh::device_status_word();
  p.sched = rbh::dynamic_tiles() ? rbh::next_sched_slot() : nullptr;
  MoeHooks h{};
  h.items = (const int4*)items; h.n_items = n_items; h.slot_weight = slot_weight; h.rows_per_expert = p.N;
  h.glu = GluParams{limit, slope, shift};
  return glu ? launch_moe_pair<__nv_bfloat16, EPI_GLU>(a, h, experts, a.stream)
             : launch_moe_pair<__nv_bfloat16, EPI_LEAN>(a, h, experts, a.stream);
}

// glu: x = activations, w [experts][2 n_out][n_in] (32 gates, 32 ups, ...; n_out a multiple of 32); x is [x_rows, n_in]
// by slot, or by token when slot_token tells which row a slot has; else: x [slots, n_in] by slot, w
// [experts][n_out][n_in].  tile: the most slots an item has (16 .. 128, a power of two).  Widths and strides are
// multiples of eight.
int rb_moe_gemm(int dtype, int glu, const void* x, long long ldx, int x_rows, const void* w, int experts, void* out,
                long long ldo, const int* items, const int* n_items, int max_items, int tile, const int* slot_token,
                const float* slot_weight, int n_in, int n_out, float limit, float slope, float shift, void* stream) {
  using namespace rb;
  if (max_items <= 0) return 0;
  auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  if (dtype != rbh::DT_BF16 || max_items > 65535 || (glu && n_out % 32)) return 22;
  if (!al(x) || !al(w) || !al(items) || ldx % 8 || n_in % 8) return 21;
  MoeGemmParams p{(const int4*)items, n_items, slot_token, slot_weight, out, ldo, n_in, n_out, GluParams{limit, slope, shift},
                  rbh::device_status_word()};
  cudaStream_t st = (cudaStream_t)stream;
  if (!glu) return moe_gemm_by_tile<false, false>(tile, dtype, x, ldx, x_rows, w, experts, max_items, p, st);
  return slot_token ? moe_gemm_by_tile<true, true>(tile, dtype, x, ldx, x_rows, w, experts, max_items, p, st)
                    : moe_gemm_by_tile<true, false>(tile, dtype, x, ldx, x_rows, w, experts, max_items, p, st);
}
}
