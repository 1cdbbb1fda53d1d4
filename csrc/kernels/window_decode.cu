// Sliding-window attention of single query rows over pages of keys and values, sm_100a, 16-bit: the query heads that
// share a key/value head attend together, so every page crosses HBM once.
//
// The kernel is bound by those bytes; what it must not be is bound by instructions.  A row has at most 16 query heads
// per key/value head, a quarter of the smallest tile of tcgen05, whose accumulators also lie in tensor memory, a
// round trip away from the softmax.  So the products are warp-level ones of 16 heads x 8 keys (or numbers), whose
// fragments stay in registers from scores to values, and the tensor pipe idles most of the time.
//
// A CTA takes a slice of one row's tiles of 64 keys: TMA brings keys and values of a tile (one page or several,
// 128-byte swizzle) into a ring, the four warps take turns at asking for them, and warp w attends to keys 16 w .. 16 w
// + 15 of every tile with a maximum, sum and accumulator of its own.  They meet at the end; slices meet in attn_merge.
#include "attn_merge.cuh"
#include "warp_mma.cuh"

namespace rb {

struct WindowDecodeParams {
  const void* q;                 // row b, head h at q[b * ldq + h * dim]
  long long ldq;
  const int *tables, *ctx;       // [rows, max_blocks], [rows]: keys up to and with the row's own
  const float* sink;             // [heads] or null
  const void* gate;
  long long ldg, ldo;
  void* out;
  float *part_o, *part_ml;       // used when splits > 1
  int heads, kv_heads, dim, vdim, window, block_size, box_rows, max_blocks, splits, gate_kind, blocks_per_kv;
  int keep;                      // the first tokens stay visible outside the window
  float scale_log2, scale, cap, out_scale;   // cap 0: none
  int* status;
};

constexpr int kWdKeys = 64;

template <int KS, int VS>        // 64-column sub-tiles of keys and of values
struct WindowDecodeCfg {
  static constexpr int SUB = kWdKeys * 128;
  static constexpr int K_BYTES = KS * SUB, STAGE = (KS + VS) * SUB;
  static constexpr int STAGES = KS + VS == 4 ? 2 : KS + VS == 3 ? 3 : 4;
  static constexpr int SMEM_BYTES = STAGES * STAGE + 1024;
};

template <int KS, int VS>
__global__ void __launch_bounds__(128, 3)
    window_decode_kernel(const __grid_constant__ CUtensorMap tk, const __grid_constant__ CUtensorMap tv, const WindowDecodeParams p) {
  using C = WindowDecodeCfg<KS, VS>;
  using T = __nv_bfloat16;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~static_cast<uintptr_t>(1023));
  __shared__ uint64_t bars[8];
  __shared__ int s_abort;
  __shared__ float s_ml[4][16][2];
  uint64_t *full = bars, *empty = bars + 4;
  volatile int* abort_flag = &s_abort;
  const int warp = uniform_warp_idx(), lane = threadIdx.x & 31;
  const int g = blockIdx.x / p.blocks_per_kv, rep = p.heads / p.kv_heads;
  const int h0 = g * rep + (blockIdx.x - g * p.blocks_per_kv) * 16;           // first head of the CTA
  const int nh = min(16, (g + 1) * rep - h0);
  const int b = blockIdx.y, sp = blockIdx.z;
  const int ctx = p.ctx[b], lo = max(0, ctx - p.window);
  // slices are whole tiles; a tile at either end of the window is masked
  // (the kept tokens' tiles come first; where the window reaches into them there is one run of tiles)
  const int keep_tiles = (min(p.keep, lo) + kWdKeys - 1) / kWdKeys, win_tile = lo / kWdKeys;
  const int n_keep = win_tile > keep_tiles ? keep_tiles : 0, first = n_keep || keep_tiles == 0 ? win_tile : 0;
  const int all = n_keep + (ctx + kWdKeys - 1) / kWdKeys - first;
  const int per = (all + p.splits - 1) / p.splits;
  const int tile0 = sp * per, n_tiles = min(per, all - sp * per);
  auto key_of = [&](int i) { return (tile0 + i < n_keep ? tile0 + i : first + tile0 + i - n_keep) * kWdKeys; };
  if (n_tiles <= 0) {                          // nothing of this row falls into the slice (splits > 1)
    if (threadIdx.x < nh) {
      float* ml = p.part_ml + (((long long)b * p.heads + h0 + threadIdx.x) * p.splits + sp) * 2;
      ml[0] = -INFINITY;
      ml[1] = 0.f;
    }
    return;
  }
  if (threadIdx.x == 0) {
    for (int s = 0; s < C::STAGES; ++s) {
      mbar_init(smem_u32(&full[s]), 1);
      mbar_init(smem_u32(&empty[s]), 4);
    }
    s_abort = 0;
    fence_barrier_init();
  } else if (threadIdx.x == 32) {
    prefetch_tensormap(&tk);
    prefetch_tensormap(&tv);
  }
  const int* table = p.tables + (long long)b * p.max_blocks;
  const int boxes = kWdKeys / p.box_rows;      // at most 8
  // row of the pools where box `lane` of tile i starts.  Boxes past the context are read from its last one.
  auto lookup = [&](int i) -> int {
    if (i >= n_tiles) return 0;
    const int t = min(key_of(i) + min(lane, boxes - 1) * p.box_rows, (ctx - 1) / p.box_rows * p.box_rows);
    return (table[min(t / p.block_size, p.max_blocks - 1)] * p.kv_heads + g) * p.block_size + t % p.block_size;
  };
  // whole warp: tile i into its stage
  auto bring = [&](int i, int rows) {
    const int st = i % C::STAGES;
    const uint32_t bar = smem_u32(&full[st]), dst = smem_u32(smem + st * C::STAGE);
    if (lane == 0) mbar_arrive_expect_tx(bar, C::STAGE);
    for (int x = 0; x < boxes; ++x) {
      const int row = __shfl_sync(0xffffffffu, rows, x);
      if (lane == 0) {
#pragma unroll
        for (int s = 0; s < KS; ++s) tma_load_2d(dst + s * C::SUB + x * p.box_rows * 128, &tk, bar, s * 64, row);
#pragma unroll
        for (int s = 0; s < VS; ++s) tma_load_2d(dst + C::K_BYTES + s * C::SUB + x * p.box_rows * 128, &tv, bar, s * 64, row);
      }
    }
  };
  const int rows0 = lookup(warp);
  __syncthreads();
  // warp w brings tiles w, w + 4, ...; the first STAGES of them need no room made for them
  if (warp < C::STAGES && warp < n_tiles) bring(warp, rows0);
  int duty = warp < C::STAGES ? warp + 4 : warp;
  int duty_rows = warp < C::STAGES ? lookup(duty) : rows0;

  // fragments: this lane has rows (heads) r, r + 8 and columns 2 c, 2 c + 1 of every 16 x 8 accumulator
  const int r = lane >> 2, c = lane & 3;
  uint32_t qa[KS * 4][4];
#pragma unroll
  for (int k = 0; k < KS * 4; ++k)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int h = r + (e & 1) * 8, d = k * 16 + (e >> 1) * 8 + 2 * c;
      qa[k][e] = h < nh && d < p.dim
                     ? *reinterpret_cast<const uint32_t*>(reinterpret_cast<const T*>(p.q) + b * p.ldq + (long long)(h0 + h) * p.dim + d)
                     : 0u;
    }
  float acc[VS * 8][4];
#pragma unroll
  for (int j = 0; j < VS * 8; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  // which row of a tile this lane points ldmatrix at (keys: two key groups x two halves of 16 numbers; values: two
  // halves of 16 keys x two groups of 8 numbers)
  const int k_row = warp * 16 + (lane >> 4) * 8 + (lane & 7), k_half = (lane >> 3) & 1;
  const int v_row = warp * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), v_half = lane >> 4;
  bool ok = true;
  for (int i = 0; i < n_tiles; ++i) {
    const int st = i % C::STAGES;
    // the stage that tile i - 1 had is for tile i - 1 + STAGES
    if (i > 0 && duty == i - 1 + C::STAGES) {
      if (duty < n_tiles) {
        ok = mbar_wait(smem_u32(&empty[(i - 1) % C::STAGES]), ((i - 1) / C::STAGES) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_EMPTY);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        bring(duty, duty_rows);
        duty_rows = lookup(duty + 4);
      }
      duty += 4;
    }
    ok = mbar_wait(smem_u32(&full[st]), (i / C::STAGES) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_FULL);
    ok = __all_sync(0xffffffffu, ok);
    if (!ok) break;
    const uint32_t ks = smem_u32(smem + st * C::STAGE), vs = ks + C::K_BYTES;
    float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};      // two groups of 8 keys
#pragma unroll
    for (int k = 0; k < KS * 4; ++k) {
      const int chunk = (k & 3) * 2 + k_half;
      uint32_t kb[4];
      ldmatrix_x4(ks + (k >> 2) * C::SUB + k_row * 128 + ((chunk ^ (k_row & 7)) << 4), kb);
      mma_bf16(s[0], qa[k], kb[0], kb[1]);
      mma_bf16(s[1], qa[k], kb[2], kb[3]);
    }
    if (p.cap > 0.f) {
      const float in = 2.8853900817779268f * p.scale / p.cap, out = p.cap / p.scale;   // scaled again below
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[n][e] = soft_cap(s[n][e], in, out);
    }
    const int key = key_of(i) + warp * 16 + 2 * c;
    if (key - 2 * c < lo || key - 2 * c + 15 >= ctx) {                 // uniform over the warp
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int at = key + n * 8 + (e & 1);
          if ((at < lo && at >= p.keep) || at >= ctx) s[n][e] = -INFINITY;
        }
    }
    float mx[2];
    bool need = false;
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      mx[x] = fmaxf(fmaxf(s[0][2 * x], s[0][2 * x + 1]), fmaxf(s[1][2 * x], s[1][2 * x + 1]));
      mx[x] = fmaxf(mx[x], __shfl_xor_sync(0xffffffffu, mx[x], 1));
      mx[x] = fmaxf(mx[x], __shfl_xor_sync(0xffffffffu, mx[x], 2)) * p.scale_log2;
      need |= mx[x] > m[x] + 8.0f;
    }
    if (__any_sync(0xffffffffu, need)) {                               // rare after the first tiles
      float alpha[2];
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        alpha[x] = 1.f;
        if (mx[x] > m[x]) {
          alpha[x] = m[x] == -INFINITY ? 0.f : fast_exp2(m[x] - mx[x]);
          m[x] = mx[x];
          l[x] *= alpha[x];
        }
      }
#pragma unroll
      for (int j = 0; j < VS * 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[j][e] *= alpha[e >> 1];
    }
    const float neg0 = m[0] == -INFINITY ? 0.f : -m[0], neg1 = m[1] == -INFINITY ? 0.f : -m[1];
    uint32_t pa[4];
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      const float a0 = fast_exp2(fmaf(s[n][0], p.scale_log2, neg0)), a1 = fast_exp2(fmaf(s[n][1], p.scale_log2, neg0));
      const float b0 = fast_exp2(fmaf(s[n][2], p.scale_log2, neg1)), b1 = fast_exp2(fmaf(s[n][3], p.scale_log2, neg1));
      l[0] += a0 + a1;
      l[1] += b0 + b1;
      pa[2 * n] = pack2<T>(a0, a1);
      pa[2 * n + 1] = pack2<T>(b0, b1);
    }
#pragma unroll
    for (int j = 0; j < VS * 4; ++j) {
      const int chunk = (j & 3) * 2 + v_half;
      uint32_t vb[4];
      ldmatrix_x4_trans(vs + (j >> 2) * C::SUB + v_row * 128 + ((chunk ^ (v_row & 7)) << 4), vb);
      mma_bf16(acc[2 * j], pa, vb[0], vb[1]);
      mma_bf16(acc[2 * j + 1], pa, vb[2], vb[3]);
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(smem_u32(&empty[st]));
  }
  if (!ok)                                   // copies in flight land before the shared memory gets another use
    for (int i = 0; i < 64; ++i) __nanosleep(10000);
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    l[x] += __shfl_xor_sync(0xffffffffu, l[x], 1);
    l[x] += __shfl_xor_sync(0xffffffffu, l[x], 2);
    if (c == 0) {
      s_ml[warp][r + 8 * x][0] = m[x];
      s_ml[warp][r + 8 * x][1] = l[x];
    }
  }
  __syncthreads();                           // every warp is through with the ring before sums go over it
  constexpr int W = VS * 64 + 8;
  float* so = reinterpret_cast<float*>(smem);            // [4 warps][16 heads][W]
#pragma unroll
  for (int j = 0; j < VS * 8; ++j)
#pragma unroll
    for (int x = 0; x < 2; ++x)
      if (r + 8 * x < nh)
        *reinterpret_cast<float2*>(so + (warp * 16 + r + 8 * x) * W + j * 8 + 2 * c) = make_float2(acc[j][2 * x], acc[j][2 * x + 1]);
  __syncthreads();
  for (int x = threadIdx.x; x < nh * p.vdim; x += 128) {
    const int hl = x / p.vdim, d = x - hl * p.vdim, h = h0 + hl;
    const float sk = p.splits == 1 && p.sink ? p.sink[h] * 1.4426950408889634f : -INFINITY;
    float gm = sk;
#pragma unroll
    for (int w = 0; w < 4; ++w) gm = fmaxf(gm, s_ml[w][hl][0]);
    float gl = 0.f, o = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float mv = s_ml[w][hl][0];
      const float fw = mv == -INFINITY ? 0.f : fast_exp2(mv - gm);
      gl += s_ml[w][hl][1] * fw;
      o += so[(w * 16 + hl) * W + d] * fw;
    }
    if (p.splits > 1) {
      const long long pi = ((long long)b * p.heads + h) * p.splits + sp;
      p.part_o[pi * p.vdim + d] = o;
      if (d == 0) {
        p.part_ml[pi * 2] = gm;
        p.part_ml[pi * 2 + 1] = gl;
      }
    } else {
      if (sk != -INFINITY) gl += fast_exp2(sk - gm);
      float v = gl > 0.f ? o / gl * p.out_scale : 0.f;
      if (p.gate_kind == ATTN_GATE_ELEMENT) v *= sigmoid_f<T>(to_f32<T>(reinterpret_cast<const T*>(p.gate)[b * p.ldg + (long long)h * p.vdim + d]));
      else if (p.gate_kind == ATTN_GATE_HEAD) v *= sigmoid_f<T>(to_f32<T>(reinterpret_cast<const T*>(p.gate)[b * p.ldg + h]));
      reinterpret_cast<T*>(p.out)[b * p.ldo + (long long)h * p.vdim + d] = from_f32<T>(v);
    }
  }
}

template <int KS, int VS>
int launch_window_decode(const void* k_pool, const void* v_pool, long long pool_rows, int rows, const WindowDecodeParams& p,
                         cudaStream_t st) {
  using C = WindowDecodeCfg<KS, VS>;
  CUtensorMap tk, tv;
  auto map = [&](CUtensorMap* m, const void* base, int cols) {
    uint64_t dims[2] = {(uint64_t)cols, (uint64_t)pool_rows};
    uint64_t strides[2] = {2, (uint64_t)cols * 2};
    uint32_t box[2] = {64, (uint32_t)p.box_rows};
    return rbh::encode_tensor_map(m, rbh::DT_BF16, 2, const_cast<void*>(base), dims, strides, box, 1);
  };
  int rc = map(&tk, k_pool, p.dim);
  if (!rc) rc = map(&tv, v_pool, p.vdim);
  if (rc) return 1000 + rc;
  auto kern = window_decode_kernel<KS, VS>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM_BYTES);
  if (e != cudaSuccess) return 2000 + (int)e;
  kern<<<dim3(p.kv_heads * p.blocks_per_kv, rows, p.splits), 128, C::SMEM_BYTES, st>>>(tk, tv, p);
  e = cudaGetLastError();
  return e == cudaSuccess ? 0 : 3000 + (int)e;
}

}  // namespace rb

extern "C" {

// Whether the kernel covers these sizes (others run on rb_window_rows).
int rb_window_decode_ok(int dtype, int dim_p, int vdim_p, int block_size) {
  return dtype == rbh::DT_BF16 && dim_p <= 128 && vdim_p <= 128 && dim_p % 8 == 0 && vdim_p % 8 == 0 &&
         (block_size % 64 == 0 || (block_size >= 8 && 64 % block_size == 0));
}

// Slices of a row's visible keys (at most max_keys of them): whole waves of three CTAs per SM.
int rb_window_decode_splits(int heads, int kv_heads, int rows, int max_keys) {
  const long long ctas = (long long)kv_heads * ((heads / kv_heads + 15) / 16) * rows, slots = 3LL * rbh::sm_count();
  const int tiles = (max_keys + rb::kWdKeys - 1) / rb::kWdKeys + 1;      // kept tokens count among max_keys
  int best = 1;
  double best_cost = 1e30;
  for (int s = 1; s <= 64 && s <= tiles; ++s) {
    const long long waves = (ctas * s + slots - 1) / slots;
    const double cost = (double)waves * ((tiles + s - 1) / s + 8.0) + (s > 1 ? 3.0 : 0.0);   // set-up and tail, merge
    if (cost < best_cost - 1e-9) {
      best_cost = cost;
      best = s;
    }
  }
  return best;
}

// Arguments as rb_window_rows.
int rb_window_decode(int dtype, const void* q, long long ldq, const void* k_pool, const void* v_pool, int num_blocks,
                     const int* tables, const int* ctx, const float* sink, const void* gate, long long ldg, int gate_kind,
                     void* out, long long ldo, float* part_o, float* part_ml, int rows, int heads, int kv_heads, int dim_p,
                     int vdim_p, int window, int keep, int block_size, int max_blocks, int splits, float scale, float cap,
                     float out_scale, void* stream) {
  using namespace rb;
  if (rows <= 0) return 0;
  if (!rb_window_decode_ok(dtype, dim_p, vdim_p, block_size) || rows > 65535 || splits < 1 || splits > 64 || heads % kv_heads ||
      window < 1 || keep < 0 || !(scale > 0.f))
    return 22;
  auto al = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
  if (!al(q) || !al(k_pool) || !al(v_pool) || ldq % 8) return 21;
  WindowDecodeParams p{};
  p.q = q; p.ldq = ldq; p.tables = tables; p.ctx = ctx; p.sink = sink; p.gate = gate; p.ldg = ldg; p.ldo = ldo; p.out = out;
  p.part_o = part_o; p.part_ml = part_ml; p.heads = heads; p.kv_heads = kv_heads; p.dim = dim_p; p.vdim = vdim_p;
  p.window = window; p.block_size = block_size; p.box_rows = block_size < kWdKeys ? block_size : kWdKeys;
  p.max_blocks = max_blocks; p.splits = splits; p.gate_kind = gate ? gate_kind : ATTN_GATE_NONE;
  p.blocks_per_kv = (heads / kv_heads + 15) / 16; p.scale_log2 = scale * 1.4426950408889634f;
  p.keep = keep; p.scale = scale; p.cap = cap; p.out_scale = out_scale;
  p.status = rbh::device_status_word();
  const long long pool_rows = (long long)num_blocks * kv_heads * block_size;
  cudaStream_t st = (cudaStream_t)stream;
  int rc;
  if (dim_p <= 64) rc = vdim_p <= 64 ? launch_window_decode<1, 1>(k_pool, v_pool, pool_rows, rows, p, st) : launch_window_decode<1, 2>(k_pool, v_pool, pool_rows, rows, p, st);
  else rc = vdim_p <= 64 ? launch_window_decode<2, 1>(k_pool, v_pool, pool_rows, rows, p, st) : launch_window_decode<2, 2>(k_pool, v_pool, pool_rows, rows, p, st);
  if (rc || splits == 1) return rc;
  using T = __nv_bfloat16;
  launch_attn_merge<T>(part_o, part_ml, sink, (const T*)gate, ldg, p.gate_kind, (T*)out, ldo, rows, heads, vdim_p, splits, st, out_scale);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : 3000 + (int)e;
}
}
