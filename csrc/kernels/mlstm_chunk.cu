// Matrix memory with exponential gates over prompt portions, sm_100a (tcgen05 + TMEM + TMA), 16-bit activations: chunks of
// 128 tokens in three passes instead of a loop over tokens.
//
// With F the running sum of log forget gates inside a chunk and g_j = i_j - F_j, the recurrence's running maximum is
// m_t = F_t + c_t, c_t = max(m_0, max over j <= t of g_j), and in its units
//
//   S_t = exp(m_0 - c_t) S_0 + sum over j <= t of exp(g_j - c_t) k_j v_j^T        (n_t the same with k alone)
//
//   states   per chunk and head: the sum over the chunk's own tokens at its end, relative to its own largest g
//   scan     per portion, head and piece of the state: runs over the chunks, leaves what every chunk starts from, and the
//            state after the portion
//   outputs  per chunk and head: S_0 part and the chunk's own part, which is attention with weights exp(g_j - c_t) instead
//            of a softmax; division, output norm and gate
//
// Queries, keys and values are 16-bit numbers as they come from the projection; everything else is fp32, and where it
// meets a tensor product it goes in as a pair of 16-bit numbers (weights, gates times values, state), so the products
// keep 16 bits of it.  Tiles are 128 wide whatever the sizes of a head are; TMA fills what is missing with zeros.
#include "recurrent.cuh"
#include "warp_mma.cuh"

namespace rb {

constexpr int kMlstmChunk = 128;
// A tile: 128 rows x 128 numbers as two sub-tiles of 64 numbers (128 bytes, swizzled), TMA boxes of 64 rows each.
constexpr int kMlstmBox = 64 * 128, kMlstmSub = 2 * kMlstmBox, kMlstmTile = 2 * kMlstmSub;

__device__ __forceinline__ uint32_t mlstm_at(int r, int c) {          // byte offset of 16-byte chunk c of row r
  return (c >> 3) * kMlstmSub + r * 128 + (((c & 7) ^ (r & 7)) << 4);
}

// Tensor maps over the activations: [head][row][number], boxes of 64 rows x 64 numbers.
struct MlstmMaps {
  CUtensorMap q, k, v, gate;
};

struct MlstmChunkParams {
  const float* gates;            // row: heads input gates, heads forget gates, before the cap
  long long ldz;
  const int4* items;             // chunks: {first row, tokens, portion}, a portion's chunks neighbours
  const int4* seqs;              // portions
  const int* first;              // [portions + 1] first chunk
  float *S, *n, *m;              // state by place
  // by chunk and head: sum of the chunk's own tokens [dim_p, vdim_p] and [dim_p], {sum of forget gates, largest g}; per
  // token {g, largest g so far, F}
  float *loc, *loc_n;
  float2* loc_m;
  float4* trace;
  // what the chunk starts from: two tiles (high and low parts) as they lie in shared memory; [dim_p]; m
  uint8_t* s0;
  float *n0, *m0;
  int heads, dim_p, vdim_p, vdim;
  float q_scale, cap;
  RecOut<__nv_bfloat16> o;
  int* status;
};

// one thread: a whole tile of rows row .. row + 127
__device__ __forceinline__ void mlstm_load(uint32_t dst, const CUtensorMap* map, uint64_t* bar, int row, int h) {
  mbar_arrive_expect_tx(smem_u32(bar), kMlstmTile);
#pragma unroll
  for (int x = 0; x < 4; ++x) tma_load_3d(dst + x * kMlstmBox, map, smem_u32(bar), (x >> 1) * 64, row + (x & 1) * 64, h);
}

// ---------------------------------------------------------------------------------------------------------
// states: sum over j of exp(g_j - max g) k_j v_j^T, relative to max g + (sum of forget gates)
// ---------------------------------------------------------------------------------------------------------
constexpr int kMlstmStateSmem = 3 * kMlstmTile + 1024;

__global__ void __launch_bounds__(256, 2) mlstm_chunk_states_kernel(const __grid_constant__ MlstmMaps maps, const MlstmChunkParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  __shared__ float s_w[kMlstmChunk], s_top[8], s_n[256];
  __shared__ uint64_t full, done;
  __shared__ uint32_t tmem_ptr;
  __shared__ int s_abort;
  const int4 it = p.items[blockIdx.x];
  const int h = blockIdx.y, tid = threadIdx.x, warp = uniform_warp_idx(), lane = tid & 31;
  const long long ch = (long long)blockIdx.x * p.heads + h;
  uint8_t *s_k = smem, *s_v = smem + kMlstmTile;              // values become the high plane, the low one follows
  if (tid == 0) {
    mbar_init(smem_u32(&full), 2);
    mbar_init(smem_u32(&done), 1);
    s_abort = 0;
    fence_barrier_init();
    mlstm_load(smem_u32(s_k), &maps.k, &full, it.x, h);
    mlstm_load(smem_u32(s_v), &maps.v, &full, it.x, h);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(&tmem_ptr), 128);
    tmem_relinquish();
  }
  // running sums and maxima of the gates: thread j < 128 is token j
  float f = 0.f, g = -INFINITY, i = -INFINITY;
  if (tid < kMlstmChunk) {
    if (tid < it.y) {
      const float* z = p.gates + (long long)(it.x + tid) * p.ldz;
      const float2 x = mlstm_gates(z[h], z[p.heads + h], p.cap);
      i = x.x;
      f = x.y;
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, f, o);
      if (lane >= o) f += x;
    }
    if (lane == 31) s_top[warp] = f;
  }
  __syncthreads();
  float top = -INFINITY;
  if (tid < kMlstmChunk) {
    for (int w = 0; w < warp; ++w) f += s_top[w];
    g = i - f;
    top = g;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, top, o);
      if (lane >= o) top = fmaxf(top, x);
    }
    if (lane == 31) s_top[4 + warp] = top;
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const float most = fmaxf(fmaxf(s_top[4], s_top[5]), fmaxf(s_top[6], s_top[7]));
  if (tid < kMlstmChunk) {
    for (int w = 0; w < warp; ++w) top = fmaxf(top, s_top[4 + w]);
    s_w[tid] = expf(g - most);
    p.trace[ch * kMlstmChunk + tid] = make_float4(g, top, f, 0.f);
    if (tid == kMlstmChunk - 1) p.loc_m[ch] = make_float2(f, most);
  }
  bool ok = mbar_wait(smem_u32(&full), 0, &s_abort, p.status, RB_ERR_TIMEOUT_FULL);
  ok = __syncthreads_and(ok);
  if (ok) {
#pragma unroll 4
    for (int x = tid; x < kMlstmChunk * 16; x += 256) {        // a thread's own chunks: in place
      const int r = x >> 4;
      const uint32_t at = mlstm_at(r, x & 15);
      const uint4 v = *reinterpret_cast<const uint4*>(s_v + at);
      const float w = s_w[r];
      uint4 hi, lo;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 q = unpack2<__nv_bfloat16>(reinterpret_cast<const uint32_t*>(&v)[e]);
        const SplitPair s = split2(q.x * w, q.y * w);
        reinterpret_cast<uint32_t*>(&hi)[e] = s.hi;
        reinterpret_cast<uint32_t*>(&lo)[e] = s.lo;
      }
      *reinterpret_cast<uint4*>(s_v + at) = hi;
      *reinterpret_cast<uint4*>(s_v + kMlstmTile + at) = lo;
    }
  }
  fence_proxy_async_smem();
  __syncthreads();
  const uint32_t tmem = tmem_ptr;
  if (warp == 0 && ok) {
    constexpr uint32_t idesc = make_idesc(UmmaFormat<__nv_bfloat16>::value, 1, 1, 128, 128);
    const uint32_t k = smem_u32(s_k), v = smem_u32(s_v);
#pragma unroll
    for (int x = 0; x < 4; ++x) {                              // 64 tokens of the high, then of the low plane
      const uint32_t half = (x & 1) * 64 * 128;
      umma_f16_w4<128, 128>(tmem, make_smem_desc_sw128(k + half, kMlstmSub, 1024),
                            make_smem_desc_sw128(v + (x >> 1) * kMlstmTile + half, kMlstmSub, 1024), idesc, x != 0);
    }
    umma_commit_w(smem_u32(&done));
  }
  // keys alone, meanwhile: a thread per key number and half of the tokens
  if (ok) {
    const int d = tid & 127;
    float s = 0.f;
#pragma unroll 8
    for (int r = tid >> 7 << 6; r < (tid >> 7 << 6) + 64; ++r)
      s = fmaf(s_w[r], __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(s_k + mlstm_at(r, d >> 3) + (d & 7) * 2)), s);
    s_n[tid] = s;
    ok = mbar_wait(smem_u32(&done), 0, &s_abort, p.status, RB_ERR_TIMEOUT_TMEM_FULL);
  }
  ok = __syncthreads_and(ok);
  if (ok) {
    if (tid < p.dim_p) p.loc_n[ch * p.dim_p + tid] = s_n[tid] + s_n[128 + tid];
    tc_fence_after();
    const int d = (warp & 3) * 32 + lane, c0 = (warp >> 2) * 64;
    const uint32_t addr = tmem + (static_cast<uint32_t>((warp & 3) * 32) << 16) + c0;
    float* out = p.loc + (ch * p.dim_p + d) * p.vdim_p;
#pragma unroll
    for (int c = 0; c < 64; c += 32) {
      uint32_t r[32];
      tmem_ld_32x32b_x32(addr + c, r);
      tmem_ld_wait();
      if (d < p.dim_p) {
#pragma unroll
        for (int x = 0; x < 32; x += 4)
          if (c0 + c + x < p.vdim_p) *reinterpret_cast<uint4*>(out + c0 + c + x) = make_uint4(r[x], r[x + 1], r[x + 2], r[x + 3]);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 128);
  }
}

// ---------------------------------------------------------------------------------------------------------
// scan: grid (16 pieces of the state's tile, then one for n and m; heads; portions)
// ---------------------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) mlstm_chunk_scan_kernel(const MlstmChunkParams p) {
  const int h = blockIdx.y, tid = threadIdx.x;
  const int4 seq = p.seqs[blockIdx.z];
  const int c0 = p.first[blockIdx.z], c1 = p.first[blockIdx.z + 1];
  const long long sh = (long long)seq.z * p.heads + h;
  const bool fresh = seq.w == 0;
  const int size = p.dim_p * p.vdim_p;
  float m = fresh ? 0.f : p.m[sh];
  // factors of a chunk: {state, chunk's own sum}
  auto step = [&](float2 fg) {
    const float c = fmaxf(m, fg.y);
    const float2 w = make_float2(expf(m - c), expf(fg.y - c));
    m = fg.x + c;
    return w;
  };
  if (blockIdx.x < 16) {
    const int x4 = (blockIdx.x * 256 + tid) * 4, d = x4 >> 7, col = x4 & 127, i = d * p.vdim_p + col;
    const bool live = d < p.dim_p && col < p.vdim_p;
    uint8_t* out = p.s0 + mlstm_at(d, col >> 3) + (col & 7) * 2;
    float4 s = !fresh && live ? *reinterpret_cast<const float4*>(p.S + sh * size + i) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int c = c0; c < c1; ++c) {
      const long long ch = (long long)c * p.heads + h;
      const float4 x = live ? *reinterpret_cast<const float4*>(p.loc + ch * size + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      const float2 w = step(p.loc_m[ch]);
      const SplitPair a = split2(s.x, s.y), b = split2(s.z, s.w);
      uint8_t* at = out + ch * 2 * kMlstmTile;
      *reinterpret_cast<uint2*>(at) = make_uint2(a.hi, b.hi);
      *reinterpret_cast<uint2*>(at + kMlstmTile) = make_uint2(a.lo, b.lo);
      s = make_float4(fmaf(w.x, s.x, w.y * x.x), fmaf(w.x, s.y, w.y * x.y), fmaf(w.x, s.z, w.y * x.z), fmaf(w.x, s.w, w.y * x.w));
    }
    if (live) *reinterpret_cast<float4*>(p.S + sh * size + i) = s;
    return;
  }
  float s = !fresh && tid < p.dim_p ? p.n[sh * p.dim_p + tid] : 0.f;
  for (int c = c0; c < c1; ++c) {
    const long long ch = (long long)c * p.heads + h;
    if (tid == 0) p.m0[ch] = m;
    const float2 w = step(p.loc_m[ch]);
    if (tid < p.dim_p) {
      p.n0[ch * p.dim_p + tid] = s;
      s = fmaf(w.x, s, w.y * p.loc_n[ch * p.dim_p + tid]);
    }
  }
  if (tid < p.dim_p) p.n[sh * p.dim_p + tid] = s;
}

// ---------------------------------------------------------------------------------------------------------
// outputs: a thread of warps 0-3 has a token (a lane of tensor memory), warp 4 brings tiles, warp 5 issues the products
//
//   room 0   queries, then the output gates, then the results on their way out
//   room 1   starting state, high part, then keys          room 2   starting state, low part, then values
//   tensor memory: scores (columns 0 .. 127; a half's weights go over its scores, high and low parts side by side), sums
// ---------------------------------------------------------------------------------------------------------
constexpr int kMlstmOutSmem = 3 * kMlstmTile + 1024;

__global__ void __launch_bounds__(192, 2) mlstm_chunk_out_kernel(const __grid_constant__ MlstmMaps maps, const MlstmChunkParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  __shared__ __align__(16) float s_g[kMlstmChunk], s_n0[128], s_norm[128];
  __shared__ uint64_t bars[9];
  __shared__ uint32_t tmem_ptr;
  __shared__ int s_abort;
  uint64_t *q_full = bars, *s_full = bars + 1, *inter_done = bars + 2, *k_full = bars + 3, *v_full = bars + 4, *s_done = bars + 5, *p_ready = bars + 6,
           *o_done = bars + 7, *gate_full = bars + 8;
  constexpr uint32_t O_COL = 128;
  const int4 it = p.items[blockIdx.x];
  const int h = blockIdx.y, tid = threadIdx.x, warp = uniform_warp_idx(), lane = tid & 31;
  const long long ch = (long long)blockIdx.x * p.heads + h;
  const uint32_t r0 = smem_u32(smem), r1 = r0 + kMlstmTile, r2 = r1 + kMlstmTile;
  if (tid == 0) {
    for (int b = 0; b < 9; ++b) mbar_init(smem_u32(&bars[b]), b == 6 ? 128 : 1);
    s_abort = 0;
    fence_barrier_init();
  }
  if (warp == 5) {
    tmem_alloc(smem_u32(&tmem_ptr), 256);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_ptr;
  auto wait = [&](uint64_t* bar, int code) {
    const bool ok = mbar_wait(smem_u32(bar), 0, &s_abort, p.status, code);
    return __all_sync(0xffffffffu, ok) != 0;
  };
  if (warp == 4) {
    if (lane == 0) {
      mlstm_load(r0, &maps.q, q_full, it.x, h);
      mbar_arrive_expect_tx(smem_u32(s_full), 2 * kMlstmTile);
      bulk_load_1d(r1, p.s0 + ch * 2 * kMlstmTile, 2 * kMlstmTile, smem_u32(s_full));
    }
    __syncwarp();
    bool ok = wait(inter_done, RB_ERR_TIMEOUT_EMPTY);
    if (ok && lane == 0) {
      mlstm_load(r1, &maps.k, k_full, it.x, h);
      mlstm_load(r2, &maps.v, v_full, it.x, h);
    }
    __syncwarp();
    ok = ok && wait(p_ready, RB_ERR_TIMEOUT_EMPTY);       // every token has read its query, and the scores are done
    if (ok && lane == 0) mlstm_load(r0, &maps.gate, gate_full, it.x, h);
    __syncwarp();
    if (!ok)
      for (int i = 0; i < 64; ++i) __nanosleep(10000);
  } else if (warp == 5) {
    using F = UmmaFormat<__nv_bfloat16>;
    constexpr uint32_t by_row = make_idesc(F::value, 0, 0, 128, 128), by_col = make_idesc(F::value, 0, 1, 128, 128);
    bool ok = wait(q_full, RB_ERR_TIMEOUT_FULL) && wait(s_full, RB_ERR_TIMEOUT_FULL);
    if (ok) {
      tc_fence_after();
#pragma unroll
      for (int x = 0; x < 4; ++x)                       // 64 key numbers of the high, then of the low part
        umma_f16_w4<2, 128>(tmem + O_COL, make_smem_desc_sw128(r0 + (x & 1) * kMlstmSub, 16, 1024),
                            make_smem_desc_sw128(r1 + (x >> 1) * kMlstmTile + (x & 1) * 64 * 128, kMlstmSub, 1024), by_col, x != 0);
      umma_commit_w(smem_u32(inter_done));
      ok = wait(k_full, RB_ERR_TIMEOUT_FULL);
    }
    if (ok) {
      tc_fence_after();
#pragma unroll
      for (int x = 0; x < 2; ++x)
        umma_f16_w4<2, 2>(tmem, make_smem_desc_sw128(r0 + x * kMlstmSub, 16, 1024), make_smem_desc_sw128(r1 + x * kMlstmSub, 16, 1024), by_row,
                          x != 0);
      umma_commit_w(smem_u32(s_done));
      ok = wait(v_full, RB_ERR_TIMEOUT_FULL) && wait(p_ready, RB_ERR_TIMEOUT_FLAG);
    }
    if (ok) {
      tc_fence_after();
#pragma unroll
      for (int i = 0; i < 8; ++i)                       // 16 tokens at a time, high and low parts of their weights
#pragma unroll
        for (int x = 0; x < 2; ++x)
          umma_f16_ts_w(tmem + O_COL, tmem + (i >> 2) * 64 + x * 32 + (i & 3) * 8, make_smem_desc_sw128(r2 + i * 2048, kMlstmSub, 1024), by_col, 1u);
      umma_commit_w(smem_u32(o_done));
    }
  } else {
    const int t = tid;
    const uint32_t lane_addr = tmem + (static_cast<uint32_t>(warp * 32) << 16);
    const float4 tr = p.trace[ch * kMlstmChunk + t];    // {g, largest g so far, F}
    const float m0 = p.m0[ch];
    constexpr float LOG2E = 1.4426950408889634f;
    s_g[t] = tr.x * LOG2E;
    s_n0[t] = t < p.dim_p ? p.n0[ch * p.dim_p + t] : 0.f;
    s_norm[t] = t < p.vdim_p ? p.o.norm[h * p.o.norm_step + t] : 0.f;
    const float c = fmaxf(m0, tr.y), w = expf(m0 - c) * p.q_scale, floor_ = expf(-(tr.z + c)), c2 = c * LOG2E;
    // the last chunk leaves the state's m: the scan has read the old one
    if (t == kMlstmChunk - 1 && (int)blockIdx.x == p.first[it.z + 1] - 1) p.m[(long long)p.seqs[it.z].z * p.heads + h] = tr.z + c;
    asm volatile("bar.sync 1, 128;" ::: "memory");
    bool ok = wait(q_full, RB_ERR_TIMEOUT_FULL);
    float l = 0.f;
    if (ok) {
#pragma unroll 4
      for (int x = 0; x < 16; ++x) {
        const uint4 q = *reinterpret_cast<const uint4*>(smem + mlstm_at(t, x));
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 v = unpack2<__nv_bfloat16>(reinterpret_cast<const uint32_t*>(&q)[e]), n = *reinterpret_cast<const float2*>(s_n0 + x * 8 + e * 2);
          l = fmaf(v.x, n.x, fmaf(v.y, n.y, l));
        }
      }
      l *= w;
      ok = wait(inter_done, RB_ERR_TIMEOUT_TMEM_FULL);
    }
    if (ok) {                                           // the starting state's part in units of this token
      tc_fence_after();
#pragma unroll 1
      for (int x = 0; x < 128; x += 32) {
        uint32_t r[32];
        tmem_ld_32x32b_x32(lane_addr + O_COL + x, r);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * w);
        tmem_st_32x32b_x32(lane_addr + O_COL + x, r);
      }
      ok = wait(s_done, RB_ERR_TIMEOUT_TMEM_FULL);
    }
    if (ok) {
      tc_fence_after();
#pragma unroll 1
      for (int half = 0; half < 2; ++half) {
        const uint32_t addr = lane_addr + half * 64;
        uint32_t s[64];
        if (half * 64 <= warp * 32 + 31) {              // uniform over the warp: tokens before the half see none of it
          tmem_ld_32x32b_x32(addr, s);
          tmem_ld_32x32b_x32(addr + 32, s + 32);
          tmem_ld_wait();
          const int seen = t - half * 64;               // columns up to this one
#pragma unroll
          for (int i = 0; i < 64; i += 4) {
            const float4 g = *reinterpret_cast<const float4*>(s_g + half * 64 + i);
            const float gs[4] = {g.x, g.y, g.z, g.w};
            float pr[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              pr[e] = i + e <= seen ? __uint_as_float(s[i + e]) * p.q_scale * fast_exp2(gs[e] - c2) : 0.f;
              l += pr[e];
            }
            // in the registers of the scores: high parts, then low parts
            const SplitPair a = split2(pr[0], pr[1]), b = split2(pr[2], pr[3]);
            s[i] = a.hi; s[i + 1] = b.hi; s[i + 2] = a.lo; s[i + 3] = b.lo;
          }
        } else {
#pragma unroll
          for (int i = 0; i < 64; ++i) s[i] = 0u;
        }
        uint32_t hi[32], lo[32];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          hi[2 * i] = s[4 * i]; hi[2 * i + 1] = s[4 * i + 1];
          lo[2 * i] = s[4 * i + 2]; lo[2 * i + 1] = s[4 * i + 3];
        }
        tmem_st_32x32b_x32(addr, hi);
        tmem_st_32x32b_x32(addr + 32, lo);
      }
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(smem_u32(p_ready));
      ok = wait(o_done, RB_ERR_TIMEOUT_TMEM_EMPTY) && wait(gate_full, RB_ERR_TIMEOUT_FULL);
    }
    if (ok) {
      tc_fence_after();
      uint32_t o[128];
#pragma unroll
      for (int x = 0; x < 4; ++x) tmem_ld_32x32b_x32(lane_addr + O_COL + x * 32, o + x * 32);
      tmem_ld_wait();
      const float inv = 1.0f / (fmaxf(fabsf(l), floor_) + 1e-6f);
      float sum[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int i = 0; i < 128; ++i) {
        const float v = __uint_as_float(o[i]) * inv;
        o[i] = __float_as_uint(v);
        sum[i & 3] = fmaf(v, v, sum[i & 3]);
      }
      const float scale = 1.0f / sqrtf(((sum[0] + sum[1]) + (sum[2] + sum[3])) / p.vdim + p.o.eps);
#pragma unroll
      for (int x = 0; x < 16; ++x) {                    // a thread's gates give way to its results
        uint4* at = reinterpret_cast<uint4*>(smem + mlstm_at(t, x));
        uint4 g = *at;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 gate = unpack2<__nv_bfloat16>(reinterpret_cast<const uint32_t*>(&g)[e]), n = *reinterpret_cast<const float2*>(s_norm + x * 8 + e * 2);
          reinterpret_cast<uint32_t*>(&g)[e] =
              pack2<__nv_bfloat16>(__uint_as_float(o[x * 8 + 2 * e]) * scale * n.x * sigmoid_tanh(gate.x),
                                   __uint_as_float(o[x * 8 + 2 * e + 1]) * scale * n.y * sigmoid_tanh(gate.y));
        }
        *at = g;
      }
    }
    ok = __all_sync(0xffffffffu, ok);
    __syncwarp();
    // a warp's own 32 tokens, two whole rows at a time
    const int x = lane & 15;
    if (ok && x * 8 < p.vdim_p) {
#pragma unroll 4
      for (int i = lane >> 4; i < 32; i += 2) {
        const int row = warp * 32 + i;
        if (row < it.y)
          *reinterpret_cast<uint4*>(p.o.out + (long long)(it.x + row) * p.o.ldo + (long long)h * p.vdim_p + x * 8) =
              *reinterpret_cast<const uint4*>(smem + mlstm_at(row, x));
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 5) {
    tc_fence_after();
    tmem_dealloc(tmem, 256);
  }
}

}  // namespace rb

extern "C" {

// Whether the kernels cover these sizes (others run token by token).
int rb_mlstm_chunk_ok(int dtype, int dim_p, int vdim_p) {
  return dtype == rbh::DT_BF16 && dim_p <= 128 && vdim_p <= 128 && dim_p % 8 == 0 && vdim_p % 8 == 0;
}

// Bytes of scratch per chunk and head: two state tiles, per-token numbers, own sums, {F, g}, m.
struct MlstmScratch {
  long long s0, trace, loc, loc_n, n0, loc_m, m0;
};
static MlstmScratch mlstm_scratch(int dim_p, int vdim_p) {
  return {2LL * rb::kMlstmTile, rb::kMlstmChunk * 16LL, 4LL * dim_p * vdim_p, 4LL * dim_p, 4LL * dim_p, 8, 8};
}
long long rb_mlstm_chunk_scratch(int dim_p, int vdim_p) {
  const MlstmScratch n = mlstm_scratch(dim_p, vdim_p);
  return n.s0 + n.trace + n.loc + n.loc_n + n.n0 + n.loc_m + n.m0;
}

// tokens: rows of proj and gate; items: chunks of up to 128 tokens; first: [portions + 1]; scratch: rb_mlstm_chunk_scratch
// bytes per chunk and head.  Otherwise as rb_mlstm_rows.
int rb_mlstm_chunk(int dtype, const void* proj, long long ldp, int tokens, const float* gates, long long ldz, const int* items, int n_items,
                   const int* seqs, const int* first, int portions, float* S, float* n, float* m, const void* gate, long long ldg,
                   const float* norm, void* out, long long ldo, void* scratch, int heads, int dim_p, int vdim_p, int vdim, float q_scale,
                   float cap, float eps, void* stream) {
  using namespace rb;
  if (n_items <= 0) return 0;
  auto al = [](const void* x, int to) { return (reinterpret_cast<uintptr_t>(x) & (to - 1)) == 0; };
  if (!rb_mlstm_chunk_ok(dtype, dim_p, vdim_p) || heads > 65535 || portions > 65535) return 22;
  if (!al(proj, 16) || !al(gate, 16) || !al(out, 16) || !al(norm, 4) || !al(S, 16) || !al(scratch, 256) || ldp % 8 || ldg % 8 || ldo % 8) return 21;
  using T = __nv_bfloat16;
  MlstmChunkParams p{};
  p.gates = gates; p.ldz = ldz; p.items = (const int4*)items; p.seqs = (const int4*)seqs; p.first = first; p.S = S; p.n = n; p.m = m;
  p.heads = heads; p.dim_p = dim_p; p.vdim_p = vdim_p; p.vdim = vdim; p.q_scale = q_scale; p.cap = cap;
  p.o = RecOut<T>{(T*)out, ldo, (const T*)gate, ldg, norm, vdim_p, nullptr, eps};
  p.status = rbh::device_status_word();
  const MlstmScratch sz = mlstm_scratch(dim_p, vdim_p);
  char* at = (char*)scratch;
  auto take = [&](long long bytes) {
    char* x = at;
    at += (long long)n_items * heads * bytes;
    return x;
  };
  p.s0 = (uint8_t*)take(sz.s0);
  p.trace = (float4*)take(sz.trace);
  p.loc = (float*)take(sz.loc);
  p.loc_n = (float*)take(sz.loc_n);
  p.n0 = (float*)take(sz.n0);
  p.loc_m = (float2*)take(sz.loc_m);
  p.m0 = (float*)take(sz.m0);
  MlstmMaps maps;
  auto map = [&](CUtensorMap* x, const T* base, long long ld, int cols) {
    uint64_t dims[3] = {(uint64_t)cols, (uint64_t)tokens, (uint64_t)heads};
    uint64_t strides[3] = {2, (uint64_t)ld * 2, (uint64_t)cols * 2};
    uint32_t box[3] = {64, 64, 1};
    return rbh::encode_tensor_map(x, rbh::DT_BF16, 3, const_cast<T*>(base), dims, strides, box, 1);
  };
  const T* q = (const T*)proj;
  int rc = map(&maps.q, q, ldp, dim_p);
  if (!rc) rc = map(&maps.k, q + (long long)heads * dim_p, ldp, dim_p);
  if (!rc) rc = map(&maps.v, q + 2LL * heads * dim_p, ldp, vdim_p);
  if (!rc) rc = map(&maps.gate, (const T*)gate, ldg, vdim_p);
  if (rc) return 1000 + rc;
  cudaError_t e = cudaFuncSetAttribute(mlstm_chunk_states_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kMlstmStateSmem);
  if (e == cudaSuccess) e = cudaFuncSetAttribute(mlstm_chunk_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kMlstmOutSmem);
  if (e != cudaSuccess) return 2000 + (int)e;
  cudaStream_t st = (cudaStream_t)stream;
  mlstm_chunk_states_kernel<<<dim3(n_items, heads), 256, kMlstmStateSmem, st>>>(maps, p);
  mlstm_chunk_scan_kernel<<<dim3(17, heads, portions), 256, 0, st>>>(p);
  mlstm_chunk_out_kernel<<<dim3(n_items, heads), 192, kMlstmOutSmem, st>>>(maps, p);
  e = cudaGetLastError();
  return e == cudaSuccess ? 0 : 3000 + (int)e;
}
}
