// Matrix product of few rows (decoded tokens) with a large weight, sm_100a (tcgen05 + TMEM + TMA + clusters):
// out [M, N] = act(alpha x [M, K] w [N, K]^T + bias) + residual, M up to 128, 16-bit operands, both K-major.
//
// Such a product is bound by the weight's bytes, and with whole columns of K per CTA by how few CTAs a small N gives.  So
// the weight lies on the M side, 128 rows a CTA, the tokens on the N side, and a cluster of up to eight CTAs shares K: each
// takes a slice, all of its loads in flight at once, and leaves its sums in shared memory, from where every CTA of the
// cluster adds up its own share of the rows in a fixed order.
//
//   warp 4      TMA producer          warp 5      tcgen05 issuer          warps 0-3   accumulators -> shared memory
//   all warps   sum over the cluster, epilogue
#include "gemm_pair_launch.cuh"

namespace rb {

struct GemmRowsParams {
  void* out;
  const void *bias, *residual;
  long long ldo, ldr;
  int M, N, K, kb_per, act, out_f32;
  float alpha;
  int* status;
};

template <int NT>
struct GemmRowsCfg {
  static constexpr int A_BYTES = 128 * 128, B_BYTES = NT * 128, STAGE = A_BYTES + B_BYTES;
  static constexpr int STAGES = 4, SUM_BYTES = NT * 128 * 4;     // the sums go where the stages were
  static constexpr int SMEM_BYTES = (STAGES * STAGE > SUM_BYTES ? STAGES * STAGE : SUM_BYTES) + 1024;
  static constexpr int TMEM_COLS = NT < 32 ? 32 : NT;
};

__device__ __forceinline__ float ld_cluster_f32(uint32_t addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr));
  return v;
}

template <typename T>
__device__ __forceinline__ void gemm_rows_store(const GemmRowsParams& p, int t, int n, float v, float bias) {
  v = apply_act(v * p.alpha + bias, p.act);
  if (p.out_f32) {
    if (p.residual) v += reinterpret_cast<const float*>(p.residual)[t * p.ldr + n];
    reinterpret_cast<float*>(p.out)[t * p.ldo + n] = v;
  } else {
    if (p.residual) v += to_f32<T>(reinterpret_cast<const T*>(p.residual)[t * p.ldr + n]);
    reinterpret_cast<T*>(p.out)[t * p.ldo + n] = from_f32<T>(v);
  }
}

template <typename T, int NT, int CLUSTER>
__global__ void __launch_bounds__(192)
    gemm_rows_kernel(const __grid_constant__ CUtensorMap tw, const __grid_constant__ CUtensorMap tx, const GemmRowsParams p) {
  using C = GemmRowsCfg<NT>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  __shared__ uint64_t full[C::STAGES], empty[C::STAGES], done;
  __shared__ uint32_t tmem_ptr;
  __shared__ int s_abort;
  volatile int* abort_flag = &s_abort;
  const int warp_idx = uniform_warp_idx(), lane = threadIdx.x & 31;
  const int rank = blockIdx.x % CLUSTER, n0 = blockIdx.x / CLUSTER * 128;
  const int kb0 = rank * p.kb_per, kb1 = min((p.K + 63) / 64, kb0 + p.kb_per);
  if (threadIdx.x == 0) {
    prefetch_tensormap(&tw);
    prefetch_tensormap(&tx);
    for (int s = 0; s < C::STAGES; ++s) {
      mbar_init(smem_u32(&full[s]), 1);
      mbar_init(smem_u32(&empty[s]), 1);
    }
    mbar_init(smem_u32(&done), 1);
    s_abort = 0;
    fence_barrier_init();
  }
  if (warp_idx == 5) {
    tmem_alloc(smem_u32(&tmem_ptr), C::TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = tmem_ptr;
  if (warp_idx == 4) {
    bool ok = true;
    for (int kb = kb0; kb < kb1; ++kb) {
      const int i = kb - kb0, st = i % C::STAGES;
      ok = mbar_wait(smem_u32(&empty[st]), ((i / C::STAGES) & 1) ^ 1, abort_flag, p.status, RB_ERR_TIMEOUT_EMPTY);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      if (lane == 0) {
        const uint32_t bar = smem_u32(&full[st]), a = smem_u32(smem + st * C::STAGE);
        mbar_arrive_expect_tx(bar, C::STAGE);
        tma_load_2d(a, &tw, bar, kb * 64, n0);
        tma_load_2d(a + C::A_BYTES, &tx, bar, kb * 64, 0);
      }
      __syncwarp();
    }
    if (!ok)
      for (int i = 0; i < 64; ++i) __nanosleep(10000);
  } else if (warp_idx == 5) {
    constexpr uint32_t idesc = make_idesc(UmmaFormat<T>::value, 0, 0, 128, NT);
    bool ok = true;
    for (int kb = kb0; kb < kb1; ++kb) {
      const int i = kb - kb0, st = i % C::STAGES;
      ok = mbar_wait(smem_u32(&full[st]), (i / C::STAGES) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_FULL);
      if (!ok) break;
      tc_fence_after();
      const uint32_t a = smem_u32(smem + st * C::STAGE);
      umma_f16_w4<2, 2>(tmem_base, make_smem_desc_sw128(a, 16, 1024), make_smem_desc_sw128(a + C::A_BYTES, 16, 1024), idesc, i != 0);
      umma_commit_w(smem_u32(&empty[st]));
    }
    if (ok) umma_commit_w(smem_u32(&done));
  }
  // every load has been consumed once the last product is done: the stages are free
  bool ok = mbar_wait(smem_u32(&done), 0, abort_flag, p.status, RB_ERR_TIMEOUT_TMEM_FULL);
  ok = __all_sync(0xffffffffu, ok);
  float* sum = reinterpret_cast<float*>(smem);              // [token][weight row]
  if (warp_idx < 4 && ok) {
    tc_fence_after();
    const uint32_t addr = tmem_base + (static_cast<uint32_t>(warp_idx * 32) << 16);
    const int m = warp_idx * 32 + lane, n = n0 + m;
    const float bias = CLUSTER == 1 && p.bias && n < p.N ? to_f32<T>(reinterpret_cast<const T*>(p.bias)[n]) : 0.f;
#pragma unroll 1
    for (int c = 0; c < NT && c < p.M; c += 16) {
      uint32_t r[16];
      tmem_ld_32x32b_x16(addr + c, r);
      tmem_ld_wait();
      if constexpr (CLUSTER > 1) {
#pragma unroll
        for (int i = 0; i < 16; ++i) sum[(c + i) * 128 + m] = __uint_as_float(r[i]);
      } else if (n < p.N) {
#pragma unroll
        for (int i = 0; i < 16; ++i)
          if (c + i < p.M) gemm_rows_store<T>(p, c + i, n, __uint_as_float(r[i]), bias);
      }
    }
  }
  tc_fence_before();
  if constexpr (CLUSTER > 1) cluster_sync_all();
  else __syncthreads();
  if (warp_idx == 5) {
    tc_fence_after();
    tmem_dealloc(tmem_base, C::TMEM_COLS);
  }
  if constexpr (CLUSTER > 1) {
    constexpr int ROWS = 128 / CLUSTER, STEP = 192 / ROWS;  // a thread keeps its weight row and takes every STEP-th token
    const int i = rank * ROWS + threadIdx.x % ROWS, n = n0 + i;
    if (ok && n < p.N) {
      const float bias = p.bias ? to_f32<T>(reinterpret_cast<const T*>(p.bias)[n]) : 0.f;
      uint32_t from[CLUSTER];
#pragma unroll
      for (int q = 0; q < CLUSTER; ++q) from[q] = map_to_cta(smem_u32(sum + i), q);
#pragma unroll 4
      for (int t = threadIdx.x / ROWS; t < p.M; t += STEP) {
        float part[CLUSTER], v = 0.f;
#pragma unroll
        for (int q = 0; q < CLUSTER; ++q) part[q] = ld_cluster_f32(from[q] + t * 512);
#pragma unroll
        for (int q = 0; q < CLUSTER; ++q) v += part[q];
        gemm_rows_store<T>(p, t, n, v, bias);
      }
    }
    cluster_sync_all();                                     // nobody's sums go while others read them
  }
}

template <typename T, int NT>
int launch_gemm_rows(int dtype, const void* x, long long ldx, const void* w, long long ldw, GemmRowsParams p, cudaStream_t st) {
  using C = GemmRowsCfg<NT>;
  CUtensorMap tw, tx;
  auto map = [&](CUtensorMap* m, const void* base, int rows, long long ld, int box_rows) {
    uint64_t dims[2] = {(uint64_t)p.K, (uint64_t)rows};
    uint64_t strides[2] = {2, (uint64_t)ld * 2};
    uint32_t box[2] = {64, (uint32_t)box_rows};
    return rbh::encode_tensor_map(m, dtype, 2, const_cast<void*>(base), dims, strides, box, 1);
  };
  int rc = map(&tw, w, p.N, ldw, 128);
  if (!rc) rc = map(&tx, x, p.M, ldx, NT);
  if (rc) return 1000 + rc;
  const int tiles = (p.N + 127) / 128, num_kb = (p.K + 63) / 64;
  // up to two CTAs per SM, slices of two blocks of K at least
  int cluster = 1;
  while (cluster < 8 && tiles * cluster <= rbh::sm_count() && num_kb >= 4 * cluster) cluster *= 2;
  p.kb_per = (num_kb + cluster - 1) / cluster;
  while (cluster > 1 && (cluster - 1) * p.kb_per >= num_kb) {      // every CTA gets something
    cluster /= 2;
    p.kb_per = (num_kb + cluster - 1) / cluster;
  }
  auto go = [&](auto kern) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM_BYTES);
    if (e != cudaSuccess) return 2000 + (int)e;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(tiles * cluster);
    cfg.blockDim = dim3(192);
    cfg.dynamicSmemBytes = C::SMEM_BYTES;
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = cluster;
    attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    e = cudaLaunchKernelEx(&cfg, kern, tw, tx, p);
    return e == cudaSuccess ? 0 : 3000 + (int)e;
  };
  switch (cluster) {
    case 1: return go(gemm_rows_kernel<T, NT, 1>);
    case 2: return go(gemm_rows_kernel<T, NT, 2>);
    case 4: return go(gemm_rows_kernel<T, NT, 4>);
    default: return go(gemm_rows_kernel<T, NT, 8>);
  }
}

template <typename T>
int gemm_rows_by_tile(int dtype, const void* x, long long ldx, const void* w, long long ldw, const GemmRowsParams& p, cudaStream_t st) {
  if (p.M <= 16) return launch_gemm_rows<T, 16>(dtype, x, ldx, w, ldw, p, st);
  if (p.M <= 32) return launch_gemm_rows<T, 32>(dtype, x, ldx, w, ldw, p, st);
  if (p.M <= 64) return launch_gemm_rows<T, 64>(dtype, x, ldx, w, ldw, p, st);
  return launch_gemm_rows<T, 128>(dtype, x, ldx, w, ldw, p, st);
}

}  // namespace rb

extern "C" {

// x [M, K], w [N, K] (rows 16-byte aligned); bias of the operands' type or null, residual of the output's or null.  Returns
// 13 when the operands are outside what this kernel covers.
int rb_gemm_rows(int dtype, const void* x, long long ldx, const void* w, long long ldw, int M, int N, int K, void* out, long long ldo,
                 int out_f32, const void* bias, const void* residual, long long ldr, int act, float alpha, void* stream) {
  using namespace rb;
  if (M <= 0 || N <= 0) return 0;
  auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  if (dtype != rbh::DT_BF16 || M > 128 || K <= 0 || !al(x) || !al(w) || ldx % 8 || ldw % 8) return 13;
  GemmRowsParams p{out, bias, residual, ldo, ldr, M, N, K, 0, act, out_f32, alpha, rbh::device_status_word()};
  return gemm_rows_by_tile<__nv_bfloat16>(dtype, x, ldx, w, ldw, p, (cudaStream_t)stream);
}
}
