// Tensor-core kernels for single query rows over key/value latents, sm_100a (tcgen05 + TMEM + TMA).
//
// latent_decode_kernel: all heads of a row attend to the same cache rows [latent | shared key part], so one
// CTA takes a slice of one row's context for a group of NH heads and reads every cache row once.  Both
// products are written with the cache on the M side, where tiles are full whatever the number of heads is:
//
//   S^T [64 keys x NH]  = rows (keys x numbers, K-major)  . Q^T        one 16-wide step after the other
//   O^T [rank   x NH]  += rows^T (numbers x keys, M-major) . P^T       128 numbers at a time
//
// The same shared-memory tile serves both: 64 keys x 64 numbers, 128-byte swizzle, loaded by TMA straight
// from the cache pages (a tile of keys is one page or several).  Tiles are ringed in pairs (128 numbers), so
// loads of the next keys run under the softmax of the current ones.
//
// head_gemm_kernel: one small product per head with the weights on the M side (they dominate the bytes):
// carries queries into latent space, and weighted latents out of it with the output gate in its epilogue.
#include "sm100_common.cuh"

namespace rb {

struct LatentDecodeParams {
  int heads, rank_p, rot_p, block_size, max_blocks, splits;
  int rank_pairs, pairs;        // pairs of 64-number tiles: of the latent, in all
  int ring;                     // pairs the ring holds
  int box_rows;                 // keys per TMA box
  float scale_log2;
  const int* tables;
  const int* ctx;
  float* part_o;                // [rows, heads, splits, rank_p]
  float* part_ml;               // [rows, heads, splits, 2]
  int* status;
};

constexpr int kLdKeys = 64;
constexpr int kLdSlot = kLdKeys * 128;        // bytes of 64 keys x 64 numbers
constexpr int kLdPair = 2 * kLdSlot;
constexpr int kLdMaxRing = 16;

// barrier over the four softmax warps that also ORs a condition
__device__ __forceinline__ bool ld_any_of_128(int barrier, bool c) {
  uint32_t any;
  asm volatile(
      "{\n\t.reg .pred a, b;\n\tsetp.ne.u32 a, %1, 0;\n\tbar.red.or.pred b, %2, 128, a;\n\tselp.u32 %0, 1, 0, b;\n\t}\n"
      : "=r"(any)
      : "r"((uint32_t)c), "r"(barrier)
      : "memory");
  return any != 0;
}

__host__ __device__ constexpr int ld_fixed_bytes(int nh, int pairs) {
  // queries (two 64-number tiles per pair), two P buffers, scores, barriers
  return pairs * 2 * nh * 128 + 2 * nh * 128 + ((kLdKeys * (nh + 1) * 4 + 1023) & ~1023) + 2048;
}

template <typename T, int NH>
__global__ void __launch_bounds__(224, 1)
    latent_decode_kernel(const __grid_constant__ CUtensorMap tqa, const __grid_constant__ CUtensorMap tqr,
                         const __grid_constant__ CUtensorMap tc, const __grid_constant__ CUtensorMap tr,
                         const LatentDecodeParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~static_cast<uintptr_t>(1023));
  constexpr int q_tile = NH * 128;                             // bytes of NH heads x 64 numbers
  uint8_t* sRing = smem;
  uint8_t* sQ = sRing + p.ring * kLdPair;
  uint8_t* sP = sQ + p.pairs * 2 * q_tile;                  // [2][NH x 64 keys]
  float* sS = reinterpret_cast<float*>(sP + 2 * q_tile);    // [64][NH + 1]
  uint64_t* bars = reinterpret_cast<uint64_t*>(reinterpret_cast<uint8_t*>(sS) + ((kLdKeys * (NH + 1) * 4 + 1023) & ~1023));
  uint64_t* full = bars;                    // [ring]
  uint64_t* empty = bars + kLdMaxRing;      // [ring]
  uint64_t* q_full = bars + 2 * kLdMaxRing;
  uint64_t* s_full = q_full + 1;            // [2] one per score buffer
  uint64_t* s_empty = q_full + 3;           // [2]
  uint64_t* p_ready = q_full + 5;
  uint64_t* pv_done = q_full + 6;
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(q_full + 7);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_ptr + 1);
  float* s_alpha = reinterpret_cast<float*>(tmem_ptr + 4);  // [NH]

  const int warp_idx = uniform_warp_idx();
  const int lane = threadIdx.x & 31;
  const int h0 = blockIdx.x * NH;
  const int b = blockIdx.y, sp = blockIdx.z;
  const int ctx = p.ctx[b];
  // slices are whole tiles of keys
  const int tiles_all = (ctx + kLdKeys - 1) / kLdKeys;
  const int per = (tiles_all + p.splits - 1) / p.splits;
  const int tile0 = sp * per;
  const int n_tiles = max(0, min(per, tiles_all - tile0));
  const int rank_slots = (p.rank_p + 63) >> 6, rot_slots = (p.rot_p + 63) >> 6;

  if (n_tiles == 0) {                       // whole CTA: nothing of this row falls into the slice
    for (int n = threadIdx.x; n < NH; n += 224)
      if (h0 + n < p.heads) {
        float* ml = p.part_ml + (((long long)b * p.heads + h0 + n) * p.splits + sp) * 2;
        ml[0] = -INFINITY;
        ml[1] = 0.f;
      }
    return;
  }

  // two score buffers at [0, 2 NH), then NH columns per 128 numbers of the latent
  constexpr int TMEM_COLS = NH <= 16 ? 128 : NH <= 32 ? 256 : 512;
  if (threadIdx.x == 0) {
    prefetch_tensormap(&tqa);
    prefetch_tensormap(&tqr);
    prefetch_tensormap(&tc);
    prefetch_tensormap(&tr);
    for (int s = 0; s < p.ring; ++s) {
      mbar_init(smem_u32(&full[s]), 1);
      mbar_init(smem_u32(&empty[s]), 1);
    }
    mbar_init(smem_u32(q_full), 1);
    mbar_init(smem_u32(&s_full[0]), 1);
    mbar_init(smem_u32(&s_full[1]), 1);
    mbar_init(smem_u32(&s_empty[0]), 128);
    mbar_init(smem_u32(&s_empty[1]), 128);
    mbar_init(smem_u32(p_ready), 128);
    mbar_init(smem_u32(pv_done), 1);
    *abort_flag = 0;
    fence_barrier_init();
  }
  if (warp_idx == 5) {
    tmem_alloc(smem_u32(tmem_ptr), TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_ptr;

  if (warp_idx == 4) {
    // ------------------------------ TMA producer ------------------------------
    if (lane == 0) {
      mbar_arrive_expect_tx(smem_u32(q_full), (rank_slots + rot_slots) * q_tile);
      for (int s = 0; s < rank_slots; ++s)
        tma_load_3d(smem_u32(sQ + s * q_tile), &tqa, smem_u32(q_full), s * 64, h0, b);
      for (int s = 0; s < rot_slots; ++s)
        tma_load_3d(smem_u32(sQ + (p.rank_pairs * 2 + s) * q_tile), &tqr, smem_u32(q_full), s * 64, h0, b);
    }
    const int* table = p.tables + (long long)b * p.max_blocks;
    const int boxes = kLdKeys / p.box_rows;       // at most 8
    // lane x looks up where box x of a tile starts, one tile ahead of its loads.  Keys past the context are
    // masked later; they are read from its last page.
    auto lookup = [&](int j) -> int {
      const int t = min((tile0 + j) * kLdKeys + min(lane, boxes - 1) * p.box_rows, (ctx - 1) / p.box_rows * p.box_rows);
      return table[t / p.block_size] * p.block_size + t % p.block_size;
    };
    int slot = 0, next_row = lookup(0);
    uint32_t phase = 0;
    bool ok = true;
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int my_row = next_row;
      if (j + 1 < n_tiles) next_row = lookup(j + 1);
      for (int pr = 0; pr < p.pairs; ++pr) {
        ok = mbar_wait(smem_u32(&empty[slot]), phase ^ 1, abort_flag, p.status, RB_ERR_TIMEOUT_EMPTY);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        const bool rot = pr >= p.rank_pairs;
        const int first = rot ? (pr - p.rank_pairs) * 2 : pr * 2;
        const int n = min(2, (rot ? rot_slots : rank_slots) - first);
        const uint32_t bar = smem_u32(&full[slot]);
        if (lane == 0) mbar_arrive_expect_tx(bar, n * kLdSlot);
        for (int x = 0; x < boxes; ++x) {
          const int row = __shfl_sync(0xffffffffu, my_row, x);
          if (lane == 0) {
            const uint32_t dst = smem_u32(sRing + slot * kLdPair) + x * p.box_rows * 128;
            tma_load_2d(dst, rot ? &tr : &tc, bar, first * 64, row);
            if (n > 1) tma_load_2d(dst + kLdSlot, rot ? &tr : &tc, bar, first * 64 + 64, row);
          }
        }
        if (++slot == p.ring) {
          slot = 0;
          phase ^= 1;
        }
      }
    }
    if (!ok)
      for (int i = 0; i < 64; ++i) __nanosleep(10000);
  } else if (warp_idx == 5) {
    // ------------------------------ issuer of the score products --------------
    constexpr uint32_t idesc_s = make_idesc(UmmaFormat<T>::value, 0, 0, 64, NH);
    bool ok = mbar_wait(smem_u32(q_full), 0, abort_flag, p.status, RB_ERR_TIMEOUT_FULL);
    int slot = 0;
    uint32_t phase = 0;
    for (int j = 0; j < n_tiles && ok; ++j) {
      ok = mbar_wait(smem_u32(&s_empty[j & 1]), ((j >> 1) & 1) ^ 1, abort_flag, p.status, RB_ERR_TIMEOUT_TMEM_EMPTY);
      if (!ok) break;
      const uint32_t d = tmem_base + (j & 1) * NH;
      for (int pr = 0; pr < p.pairs; ++pr) {
        ok = mbar_wait(smem_u32(&full[slot]), phase, abort_flag, p.status, RB_ERR_TIMEOUT_FULL);
        if (!ok) break;
        tc_fence_after();
        const bool rot = pr >= p.rank_pairs;
        const int first = rot ? (pr - p.rank_pairs) * 2 : pr * 2;
        const bool both = (rot ? rot_slots : rank_slots) - first > 1;
        // whole tiles of 64 numbers: past the end of a part both operands are zeros
        const uint64_t a = make_smem_desc_sw128(smem_u32(sRing + slot * kLdPair), 16, 1024);
        const uint64_t q = make_smem_desc_sw128(smem_u32(sQ + pr * 2 * q_tile), 16, 1024);
        umma_f16_w4<2, 2>(d, a, q, idesc_s, pr != 0);
        if (both) umma_f16_w4<2, 2>(d, a + (kLdSlot >> 4), q + (q_tile >> 4), idesc_s, 1u);
        if (rot) umma_commit_w(smem_u32(&empty[slot]));        // the values end before the shared key part
        if (++slot == p.ring) {
          slot = 0;
          phase ^= 1;
        }
      }
      if (ok) umma_commit_w(smem_u32(&s_full[j & 1]));
    }
  } else if (warp_idx == 6) {
    // ------------------------------ issuer of the value products --------------
    // A warp of its own: products this short are bound by the issuing warp, and these need not queue behind
    // the scores of the next keys.
    constexpr uint32_t idesc_o = make_idesc(UmmaFormat<T>::value, 1, 0, 128, NH);
    int slot = 0;
    uint32_t phase = 0;
    bool ok = true;
    for (int j = 0; j < n_tiles && ok; ++j) {
      ok = mbar_wait(smem_u32(p_ready), j & 1, abort_flag, p.status, RB_ERR_TIMEOUT_FLAG);
      if (!ok) break;
      const uint64_t pb = make_smem_desc_sw128(smem_u32(sP + (j & 1) * q_tile), 16, 1024);
      for (int pr = 0; pr < p.pairs; ++pr) {
        if (pr < p.rank_pairs) {
          ok = mbar_wait(smem_u32(&full[slot]), phase, abort_flag, p.status, RB_ERR_TIMEOUT_FULL);
          if (!ok) break;
          tc_fence_after();
          // 16 keys a step; rows of numbers beyond the latent are not read back
          umma_f16_w4<128, 2>(tmem_base + 2 * NH + pr * NH,
                              make_smem_desc_sw128(smem_u32(sRing + slot * kLdPair), kLdSlot, 1024), pb, idesc_o, j != 0);
          umma_commit_w(smem_u32(&empty[slot]));
        }
        if (++slot == p.ring) {
          slot = 0;
          phase ^= 1;
        }
      }
      if (ok) umma_commit_w(smem_u32(pv_done));
    }
  } else {
    // ------------------------------ softmax: 4 warps --------------------------
    constexpr int PARTS = 128 / NH;            // threads that share a head
    constexpr int KPT = kLdKeys / PARTS;       // keys per thread: 8, 16, 32
    const int tid = threadIdx.x;
    const int n = tid / PARTS, part = tid % PARTS;
    const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>(warp_idx * 32) << 16);
    float m_used = -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = 0; j < n_tiles; ++j) {
      if (ok) ok = mbar_wait(smem_u32(&s_full[j & 1]), (j >> 1) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_TMEM_FULL);
      ok = __all_sync(0xffffffffu, ok);
      if (ok) {
        tc_fence_after();
        // the 64 rows of an M = 64 accumulator lie in the first 16 lanes of each warp's quarter
        const int key = warp_idx * 16 + (lane & 15);
        const bool seen = (tile0 + j) * kLdKeys + key < ctx;
#pragma unroll
        for (int c = 0; c < NH; c += 16) {
          uint32_t r[16];
          tmem_ld_32x32b_x16(lane_addr + (j & 1) * NH + c, r);
          tmem_ld_wait();
          if (lane < 16) {
#pragma unroll
            for (int i = 0; i < 16; ++i)
              sS[key * (NH + 1) + c + i] = seen ? __uint_as_float(r[i]) * p.scale_log2 : -INFINITY;
          }
        }
        tc_fence_before();
        mbar_arrive(smem_u32(&s_empty[j & 1]));
      }
      ok = !ld_any_of_128(1, !ok);      // a wait that ran out in one warp ends all four here
      if (!ok) break;
      float v[KPT], mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        v[i] = sS[(part * KPT + i) * (NH + 1) + n];
        mx = fmaxf(mx, v[i]);
      }
#pragma unroll
      for (int o = 1; o < PARTS; o <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float m_new = fmaxf(m_used, mx);
      const bool need = m_new > m_used + 8.0f;
      float alpha = 1.0f;
      if (need) {
        alpha = (m_used == -INFINITY) ? 0.f : fast_exp2(m_used - m_new);
        m_used = m_new;
        l *= alpha;
      }
      if (part == 0) s_alpha[n] = alpha;
      // also publishes s_alpha; the scores above are in registers by now
      const bool any = ld_any_of_128(2, need);
      if (j > 0) {
        // the previous tile's value product has to be done before O is rescaled, and before this tile's P is
        // announced (p_ready counts one tile at a time)
        ok = mbar_wait(smem_u32(pv_done), (j - 1) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_TMEM_EMPTY);
        ok = __all_sync(0xffffffffu, ok);
        if (any && ok) {
          tc_fence_after();
          for (int pr = 0; pr < p.rank_pairs; ++pr)
#pragma unroll
            for (int c = 0; c < NH; c += 16) {
              uint32_t r[16];
              const uint32_t at = lane_addr + 2 * NH + pr * NH + c;
              tmem_ld_32x32b_x16(at, r);
              tmem_ld_wait();
#pragma unroll
              for (int i = 0; i < 16; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * s_alpha[c + i]);
              tmem_st_32x32b_x16(at, r);
            }
          tmem_st_wait();
          tc_fence_before();
        }
      }
      uint8_t* prow = sP + (j & 1) * q_tile + n * 128;
#pragma unroll
      for (int q = 0; q < KPT / 8; ++q) {
        uint32_t w[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float a = fast_exp2(v[q * 8 + 2 * i] - m_used), c = fast_exp2(v[q * 8 + 2 * i + 1] - m_used);
          l += a + c;
          w[i] = pack2<T>(a, c);
        }
        const int chunk = part * (KPT / 8) + q;
        *reinterpret_cast<uint4*>(prow + ((chunk ^ (n & 7)) << 4)) = make_uint4(w[0], w[1], w[2], w[3]);
      }
      fence_proxy_async_smem();
      mbar_arrive(smem_u32(p_ready));
    }
#pragma unroll
    for (int o = 1; o < PARTS; o <<= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
    if (part == 0 && h0 + n < p.heads) {
      float* ml = p.part_ml + (((long long)b * p.heads + h0 + n) * p.splits + sp) * 2;
      ml[0] = m_used;
      ml[1] = l;
    }
    if (ok) ok = mbar_wait(smem_u32(pv_done), (n_tiles - 1) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_TMEM_EMPTY);
    ok = __all_sync(0xffffffffu, ok);
    if (ok) {
      tc_fence_after();
      for (int pr = 0; pr < p.rank_pairs; ++pr) {
        const int d = pr * 128 + warp_idx * 32 + lane;
#pragma unroll
        for (int c = 0; c < NH; c += 16) {
          uint32_t r[16];
          tmem_ld_32x32b_x16(lane_addr + 2 * NH + pr * NH + c, r);
          tmem_ld_wait();
          if (d < p.rank_p) {
#pragma unroll
            for (int i = 0; i < 16; ++i)
              if (h0 + c + i < p.heads)
                p.part_o[(((long long)b * p.heads + h0 + c + i) * p.splits + sp) * p.rank_p + d] = __uint_as_float(r[i]);
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp_idx == 5) {
    tc_fence_after();
    tmem_dealloc(tmem_base, TMEM_COLS);
  }
}

// Heads per CTA and ring length; 0 heads: outside what the kernel covers.
static void latent_decode_plan(int heads, int rank_p, int rot_p, int* nh, int* ring) {
  const int pairs = (rank_p + 127) / 128 + (rot_p + 127) / 128;
  *nh = 0;
  *ring = 0;
  if (rank_p > 512 || rot_p > 128) return;
  for (int n = 64; n >= 16; n >>= 1) {
    if (n > 16 && heads <= n / 2) continue;
    int r = (227 * 1024 - 1024 - ld_fixed_bytes(n, pairs)) / kLdPair;
    if (r > kLdMaxRing) r = kLdMaxRing;
    if (r > 4 * pairs) r = 4 * pairs;
    if (r < pairs + 1 && n > 16) continue;
    if (r < pairs) return;
    *nh = n;
    *ring = r;
    return;
  }
}

template <typename T, int NH>
int launch_latent_decode(int dtype, const void* qa, const void* qr, long long ldq, int hq, const void* pool,
                         int pool_rows, int rows, LatentDecodeParams& p, cudaStream_t st) {
  CUtensorMap tqa, tqr, tc, tr;
  const int row = p.rank_p + p.rot_p;
  auto qmap = [&](CUtensorMap* m, const void* base, int cols, long long head_stride, long long row_stride) {
    uint64_t dims[3] = {(uint64_t)cols, (uint64_t)p.heads, (uint64_t)rows};
    uint64_t strides[3] = {2, (uint64_t)head_stride * 2, (uint64_t)row_stride * 2};
    uint32_t box[3] = {64, NH, 1};
    return rbh::encode_tensor_map(m, dtype, 3, const_cast<void*>(base), dims, strides, box, 1);
  };
  auto cmap = [&](CUtensorMap* m, const T* base, int cols) {
    uint64_t dims[2] = {(uint64_t)cols, (uint64_t)pool_rows};
    uint64_t strides[2] = {2, (uint64_t)row * 2};
    uint32_t box[2] = {64, (uint32_t)p.box_rows};
    return rbh::encode_tensor_map(m, dtype, 2, const_cast<T*>(base), dims, strides, box, 1);
  };
  int rc = qmap(&tqa, qa, p.rank_p, p.rank_p, (long long)p.heads * p.rank_p);
  if (!rc) rc = qmap(&tqr, qr, p.rot_p, hq, ldq);
  if (!rc) rc = cmap(&tc, (const T*)pool, p.rank_p);
  if (!rc) rc = cmap(&tr, (const T*)pool + p.rank_p, p.rot_p);
  if (rc) return 1000 + rc;
  const int smem = p.ring * kLdPair + ld_fixed_bytes(NH, p.pairs) + 1024;
  auto kern = latent_decode_kernel<T, NH>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return 2000 + (int)e;
  kern<<<dim3((p.heads + NH - 1) / NH, rows, p.splits), 224, smem, st>>>(tqa, tqr, tc, tr, p);
  e = cudaGetLastError();
  return e == cudaSuccess ? 0 : 3000 + (int)e;
}

// ---------------------------------------------------------------------------------------------------------
// out[t, h, :] = W[h] a[t, h, :]  (optionally times sigmoid(gate[t, h, :])), one 128-output x NT-row tile per
// CTA.  W_T: W[h] stored [in][out] (out contiguous), else [out][in].
// ---------------------------------------------------------------------------------------------------------
struct HeadGemmParams {
  int rows, n_in, n_out;
  void* out;
  long long ldo, hso;            // row and head stride of out
  const void* gate;              // or null
  long long ldg, hsg;
  int* status;
};

template <int NT>
struct HeadGemmCfg {
  static constexpr int STAGES = 4;
  static constexpr int A_BYTES = 128 * 128, B_BYTES = NT * 128;
  static constexpr int SMEM_BYTES = STAGES * (A_BYTES + B_BYTES) + 1024 + 256;
  static constexpr int TMEM_COLS = NT < 32 ? 32 : NT;
};

template <typename T, int NT, bool W_T>
__global__ void __launch_bounds__(192)
    head_gemm_kernel(const __grid_constant__ CUtensorMap tw, const __grid_constant__ CUtensorMap ta,
                     const HeadGemmParams p) {
  using C = HeadGemmCfg<NT>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~static_cast<uintptr_t>(1023));
  uint8_t* sA = smem;
  uint8_t* sB = smem + C::STAGES * C::A_BYTES;
  uint64_t* full = reinterpret_cast<uint64_t*>(sB + C::STAGES * C::B_BYTES);
  uint64_t* empty = full + C::STAGES;
  uint64_t* done = empty + C::STAGES;
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(done + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_ptr + 1);
  const int warp_idx = uniform_warp_idx();
  const int lane = threadIdx.x & 31;
  const int m0 = blockIdx.x * 128, h = blockIdx.y, r0 = blockIdx.z * NT;
  const int num_kb = (p.n_in + 63) / 64;
  if (threadIdx.x == 0) {
    prefetch_tensormap(&tw);
    prefetch_tensormap(&ta);
    for (int s = 0; s < C::STAGES; ++s) {
      mbar_init(smem_u32(&full[s]), 1);
      mbar_init(smem_u32(&empty[s]), 1);
    }
    mbar_init(smem_u32(done), 1);
    *abort_flag = 0;
    fence_barrier_init();
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
      bool ok = true;
      for (int kb = 0; kb < num_kb; ++kb) {
        const int st = kb % C::STAGES;
        ok = mbar_wait(smem_u32(&empty[st]), ((kb / C::STAGES) & 1) ^ 1, abort_flag, p.status, RB_ERR_TIMEOUT_EMPTY);
        if (!ok) break;
        const uint32_t bar = smem_u32(&full[st]);
        mbar_arrive_expect_tx(bar, C::A_BYTES + C::B_BYTES);
        const uint32_t a = smem_u32(sA + st * C::A_BYTES);
        if constexpr (W_T) {
          tma_load_3d(a, &tw, bar, m0, kb * 64, h);              // 64 inputs x 64 outputs
          tma_load_3d(a + 64 * 128, &tw, bar, m0 + 64, kb * 64, h);
        } else {
          tma_load_3d(a, &tw, bar, kb * 64, m0, h);              // 128 outputs x 64 inputs
        }
        tma_load_3d(smem_u32(sB + st * C::B_BYTES), &ta, bar, kb * 64, r0, h);
      }
      if (!ok)
        for (int i = 0; i < 64; ++i) __nanosleep(10000);
    }
  } else if (warp_idx == 5) {
    constexpr uint32_t idesc = make_idesc(UmmaFormat<T>::value, W_T ? 1 : 0, 0, 128, NT);
    bool ok = true;
    for (int kb = 0; kb < num_kb; ++kb) {
      const int st = kb % C::STAGES;
      ok = mbar_wait(smem_u32(&full[st]), (kb / C::STAGES) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_FULL);
      if (!ok) break;
      tc_fence_after();
      const uint32_t a = smem_u32(sA + st * C::A_BYTES), bb = smem_u32(sB + st * C::B_BYTES);
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const uint64_t ad = W_T ? make_smem_desc_sw128(a + k * 2048, 64 * 128, 1024)
                                : make_smem_desc_sw128(a + k * 32, 16, 1024);
        umma_f16_w(tmem_base, ad, make_smem_desc_sw128(bb + k * 32, 16, 1024), idesc, (kb | k) != 0);
      }
      umma_commit_w(smem_u32(&empty[st]));
    }
    if (ok) umma_commit_w(smem_u32(done));
  } else {
    const int m = m0 + warp_idx * 32 + lane;
    const uint32_t addr = tmem_base + (static_cast<uint32_t>(warp_idx * 32) << 16);
    T* o = reinterpret_cast<T*>(p.out) + h * p.hso + m;
    // the gates are on their way while the product runs
    T gate[NT];
    if (p.gate && m < p.n_out) {
      const T* g = reinterpret_cast<const T*>(p.gate) + h * p.hsg + m;
#pragma unroll
      for (int i = 0; i < NT; ++i) gate[i] = r0 + i < p.rows ? g[(long long)(r0 + i) * p.ldg] : from_f32<T>(0.f);
    }
    bool ok = mbar_wait(smem_u32(done), 0, abort_flag, p.status, RB_ERR_TIMEOUT_TMEM_FULL);
    ok = __all_sync(0xffffffffu, ok);
    if (ok) {
      tc_fence_after();
#pragma unroll
      for (int c = 0; c < NT; c += 16) {
        uint32_t r[16];
        tmem_ld_32x32b_x16(addr + c, r);
        tmem_ld_wait();
        if (m < p.n_out) {
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            const long long t = r0 + c + i;
            if (t < p.rows) {
              float v = __uint_as_float(r[i]);
              if (p.gate) v = v / (1.0f + __expf(-to_f32<T>(gate[c + i])));
              o[t * p.ldo] = from_f32<T>(v);
            }
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp_idx == 5) {
    tc_fence_after();
    tmem_dealloc(tmem_base, C::TMEM_COLS);
  }
}

template <typename T, int NT, bool W_T>
int launch_head_gemm(int dtype, const void* a, long long lda, long long hsa, const void* w, int heads,
                     const HeadGemmParams& p, cudaStream_t st) {
  using C = HeadGemmCfg<NT>;
  CUtensorMap tw, ta;
  int rc;
  {
    const uint64_t inner = W_T ? p.n_out : p.n_in, outer = W_T ? p.n_in : p.n_out;
    uint64_t dims[3] = {inner, outer, (uint64_t)heads};
    uint64_t strides[3] = {2, inner * 2, inner * outer * 2};
    uint32_t box[3] = {64, W_T ? 64u : 128u, 1};
    rc = rbh::encode_tensor_map(&tw, dtype, 3, const_cast<void*>(w), dims, strides, box, 1);
  }
  if (!rc) {
    uint64_t dims[3] = {(uint64_t)p.n_in, (uint64_t)p.rows, (uint64_t)heads};
    uint64_t strides[3] = {2, (uint64_t)lda * 2, (uint64_t)hsa * 2};
    uint32_t box[3] = {64, NT, 1};
    rc = rbh::encode_tensor_map(&ta, dtype, 3, const_cast<void*>(a), dims, strides, box, 1);
  }
  if (rc) return 1000 + rc;
  auto kern = head_gemm_kernel<T, NT, W_T>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM_BYTES);
  if (e != cudaSuccess) return 2000 + (int)e;
  kern<<<dim3((p.n_out + 127) / 128, heads, (p.rows + NT - 1) / NT), 192, C::SMEM_BYTES, st>>>(tw, ta, p);
  e = cudaGetLastError();
  return e == cudaSuccess ? 0 : 3000 + (int)e;
}

}  // namespace rb

extern "C" {

// Whether the tensor-core decode kernel covers these sizes.
int rb_latent_decode_ok(int dtype, int heads, int rank_p, int rot_p, int block_size) {
  if (dtype != rbh::DT_BF16 || rank_p % 8 || rot_p % 8 || rot_p <= 0) return 0;
  if (!(block_size % 64 == 0 || (block_size >= 8 && 64 % block_size == 0))) return 0;
  int nh, ring;
  rb::latent_decode_plan(heads, rank_p, rot_p, &nh, &ring);
  return nh > 0;
}

// Slices of the context per row for `rows` rows of up to max_ctx keys: fills the SMs in whole waves.
int rb_latent_decode_splits(int heads, int rank_p, int rot_p, int rows, int max_ctx) {
  int nh, ring;
  rb::latent_decode_plan(heads, rank_p, rot_p, &nh, &ring);
  if (nh == 0) return 1;
  const long long ctas = (long long)((heads + nh - 1) / nh) * rows;
  const int tiles = (max_ctx + rb::kLdKeys - 1) / rb::kLdKeys, sms = rbh::sm_count();
  int best = 1;
  double best_cost = 1e30;
  for (int s = 1; s <= 64 && s <= tiles; ++s) {
    const long long waves = (ctas * s + sms - 1) / sms;
    const double cost = (double)waves * ((tiles + s - 1) / s + 3.0);   // about three tiles' worth of set-up and tail
    if (cost < best_cost - 1e-9) {
      best_cost = cost;
      best = s;
    }
  }
  return best;
}

// qa [rows, heads, rank_p] contiguous; qr: rotated parts, row stride ldq, head stride hq; pool
// [pool_rows, rank_p + rot_p].  Writes the partial results rb_latent_merge combines.
int rb_latent_decode(int dtype, const void* qa, const void* qr, long long ldq, int hq, const void* pool, int pool_rows,
                     const int* tables, const int* ctx, float* part_o, float* part_ml, int rows, int heads, int rank_p,
                     int rot_p, int block_size, int max_blocks, int splits, float scale, void* stream) {
  using namespace rb;
  if (rows <= 0) return 0;
  if (!rb_latent_decode_ok(dtype, heads, rank_p, rot_p, block_size) || rows > 65535 || splits < 1 || !(scale > 0.f)) return 22;
  auto al = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
  if (!al(qa) || !al(qr) || !al(pool) || ldq % 8 || hq % 8) return 21;
  LatentDecodeParams p{};
  int nh, ring;
  latent_decode_plan(heads, rank_p, rot_p, &nh, &ring);
  p.heads = heads; p.rank_p = rank_p; p.rot_p = rot_p; p.block_size = block_size; p.max_blocks = max_blocks;
  p.splits = splits; p.rank_pairs = (rank_p + 127) / 128; p.pairs = p.rank_pairs + (rot_p + 127) / 128; p.ring = ring;
  p.box_rows = block_size < 64 ? block_size : 64;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.tables = tables; p.ctx = ctx; p.part_o = part_o; p.part_ml = part_ml; p.status = rbh::device_status_word();
  cudaStream_t st = (cudaStream_t)stream;
  if (nh == 16) return launch_latent_decode<__nv_bfloat16, 16>(dtype, qa, qr, ldq, hq, pool, pool_rows, rows, p, st);
  if (nh == 32) return launch_latent_decode<__nv_bfloat16, 32>(dtype, qa, qr, ldq, hq, pool, pool_rows, rows, p, st);
  return launch_latent_decode<__nv_bfloat16, 64>(dtype, qa, qr, ldq, hq, pool, pool_rows, rows, p, st);
}

// w: [heads][n_in][n_out] when w_t, else [heads][n_out][n_in], contiguous; a, out, gate: row and head strides.
int rb_head_gemm(int dtype, const void* a, long long lda, long long hsa, const void* w, int w_t, void* out,
                 long long ldo, long long hso, const void* gate, long long ldg, long long hsg, int rows, int heads,
                 int n_in, int n_out, void* stream) {
  using namespace rb;
  if (rows <= 0) return 0;
  auto al = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
  if (dtype != rbh::DT_BF16 || !al(a) || !al(w) || lda % 8 || hsa % 8 || n_in % 8 || n_out % 8) return 21;
  HeadGemmParams p{rows, n_in, n_out, out, ldo, hso, gate, ldg, hsg, rbh::device_status_word()};
  cudaStream_t st = (cudaStream_t)stream;
  using T = __nv_bfloat16;
  // rows per CTA: as few as still give every SM a tile, the weights of a head then come from L2
  int nt = 64;
  while (nt > 16 && (rows <= nt / 2 || (long long)((n_out + 127) / 128) * heads * ((rows + nt - 1) / nt) < rbh::sm_count())) nt /= 2;
  if (nt == 16) return w_t ? launch_head_gemm<T, 16, true>(dtype, a, lda, hsa, w, heads, p, st) : launch_head_gemm<T, 16, false>(dtype, a, lda, hsa, w, heads, p, st);
  if (nt == 32) return w_t ? launch_head_gemm<T, 32, true>(dtype, a, lda, hsa, w, heads, p, st) : launch_head_gemm<T, 32, false>(dtype, a, lda, hsa, w, heads, p, st);
  return w_t ? launch_head_gemm<T, 64, true>(dtype, a, lda, hsa, w, heads, p, st) : launch_head_gemm<T, 64, false>(dtype, a, lda, hsa, w, heads, p, st);
}
}
