// Matrix memory with exponential gates over prompt portions, sm_100a, 16-bit activations: chunks of 128 tokens in three
// passes instead of a loop over tokens.
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
// keep 16 bits of it.  The products are warp-level: a chunk is 128 x 128 x 128 at most, its operands change their form
// (weights, splits) between products, and fragments stay in registers for that.
#include "recurrent.cuh"
#include "warp_mma.cuh"

namespace rb {

constexpr int kMlstmChunk = 128;

// Tensor maps over the activations: [head][row][number], boxes of 64 rows x 64 numbers, 128-byte swizzle; numbers past a
// head's end arrive as zeros.
struct MlstmMaps {
  CUtensorMap q, k, v, gate;
};
constexpr int kMlstmBox = 64 * 128;          // bytes

// Byte offset of 16-byte chunk c of row r in a tile of such boxes: 64-number sub-tiles of ROWS rows.
template <int ROWS>
__device__ __forceinline__ uint32_t box_at(int r, int c) {
  return (c >> 3) * (ROWS * 128) + r * 128 + (((c & 7) ^ (r & 7)) << 4);
}

struct MlstmChunkParams {
  const __nv_bfloat16* proj;     // row: heads x dim_p queries, keys, heads x vdim_p values
  long long ldp;
  const float* gates;            // row: heads input gates, heads forget gates, before the cap
  long long ldz;
  const int4* items;             // chunks: {first row, tokens, portion}, a portion's chunks neighbours
  const int4* seqs;              // portions
  const int* first;              // [portions + 1] first chunk
  float *S, *n, *m;              // state by place
  // by chunk and head: sum of the chunk's own tokens [dim_p, vdim_p] and [dim_p], {sum of forget gates, largest g}
  float *loc, *loc_n;
  float2* loc_m;
  // what the chunk starts from: per 32 columns two planes (high and low parts) [dim_p][32] as they lie in shared memory
  // (tile_at), so that bulk copies bring them there; [dim_p]; m
  uint8_t* s0;
  float *n0, *m0;
  int heads, dim_p, vdim_p, vdim;
  float q_scale, cap;
  RecOut<__nv_bfloat16> o;
};

// First 128 threads of a CTA (and all of it at the barriers): running sums of a chunk's gates.  s_g[j] = i_j - F_j
// (-infinity past the end); returns {F_j, largest g up to and with j} of thread j.
__device__ __forceinline__ float2 mlstm_chunk_gates(const MlstmChunkParams& p, int4 it, int h, float* s_g, float* s_w) {
  const int j = threadIdx.x, lane = j & 31, warp = j >> 5;
  float f = 0.f, i = -INFINITY;
  if (j < it.y) {
    const float* z = p.gates + (long long)(it.x + j) * p.ldz;
    const float2 g = mlstm_gates(z[h], z[p.heads + h], p.cap);
    i = g.x;
    f = g.y;
  }
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float x = __shfl_up_sync(0xffffffffu, f, o);
    if (lane >= o) f += x;
  }
  if (j < kMlstmChunk && lane == 31) s_w[warp] = f;
  __syncthreads();
  if (j < kMlstmChunk)
    for (int w = 0; w < warp; ++w) f += s_w[w];
  float g = i - f;
  if (j < kMlstmChunk) s_g[j] = g;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float x = __shfl_up_sync(0xffffffffu, g, o);
    if (lane >= o) g = fmaxf(g, x);
  }
  if (j < kMlstmChunk && lane == 31) s_w[4 + warp] = g;
  __syncthreads();
  if (j < kMlstmChunk)
    for (int w = 0; w < warp; ++w) g = fmaxf(g, s_w[4 + w]);
  return make_float2(f, g);
}

// ---------------------------------------------------------------------------------------------------------
// states: sum over j of exp(g_j - max g) k_j v_j^T, relative to max g + (sum of forget gates)
// ---------------------------------------------------------------------------------------------------------
template <int KS, int VS>        // 64-column sub-tiles of keys and of values
struct MlstmStateCfg {
  static constexpr int K_BYTES = kMlstmChunk * KS * 128, V_BYTES = kMlstmChunk * VS * 128;
  static constexpr int SMEM_BYTES = K_BYTES + 2 * V_BYTES + 1024;
};

template <int KS, int VS>
__global__ void __launch_bounds__(256, 2)
    mlstm_chunk_states_kernel(const __grid_constant__ MlstmMaps maps, const MlstmChunkParams p, int* status) {
  using C = MlstmStateCfg<KS, VS>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  __shared__ float s_g[kMlstmChunk], s_w[12];
  __shared__ uint64_t full;
  __shared__ int s_abort;
  const int4 it = p.items[blockIdx.x];
  const int h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t sk = smem_u32(smem), sv = sk + C::K_BYTES;
  if (tid == 0) {
    mbar_init(smem_u32(&full), 1);
    s_abort = 0;
    fence_barrier_init();
    mbar_arrive_expect_tx(smem_u32(&full), C::K_BYTES + C::V_BYTES);
#pragma unroll
    for (int x = 0; x < 2 * KS; ++x)
      tma_load_3d(sk + x * kMlstmBox, &maps.k, smem_u32(&full), (x >> 1) * 64, it.x + (x & 1) * 64, h);
#pragma unroll
    for (int x = 0; x < 2 * VS; ++x)         // they become the high plane
      tma_load_3d(sv + x * kMlstmBox, &maps.v, smem_u32(&full), (x >> 1) * 64, it.x + (x & 1) * 64, h);
  }
  const float2 fg = mlstm_chunk_gates(p, it, h, s_g, s_w);
  if (tid == kMlstmChunk - 1) {
    s_w[8] = fg.y;
    p.loc_m[(long long)blockIdx.x * p.heads + h] = fg;
  }
  __syncthreads();
  const float top = s_w[8];
  if (tid < kMlstmChunk) s_g[tid] = expf(s_g[tid] - top);
  __syncthreads();
  const bool ok = mbar_wait(smem_u32(&full), 0, &s_abort, status, RB_ERR_TIMEOUT_FULL);
  if (!__syncthreads_and(ok)) return;
#pragma unroll 4
  for (int x = tid; x < kMlstmChunk * VS * 8; x += 256) {      // a thread's own chunks: in place
    const int r = x / (VS * 8);
    const uint32_t at = C::K_BYTES + box_at<kMlstmChunk>(r, x % (VS * 8));
    const uint4 v = *reinterpret_cast<const uint4*>(smem + at);
    const float w = s_g[r];
    uint4 hi, lo;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 q = unpack2<__nv_bfloat16>(reinterpret_cast<const uint32_t*>(&v)[e]);
      const SplitPair s = split2(q.x * w, q.y * w);
      reinterpret_cast<uint32_t*>(&hi)[e] = s.hi;
      reinterpret_cast<uint32_t*>(&lo)[e] = s.lo;
    }
    *reinterpret_cast<uint4*>(smem + at) = hi;
    *reinterpret_cast<uint4*>(smem + C::V_BYTES + at) = lo;
  }
  __syncthreads();
  const long long ch = (long long)blockIdx.x * p.heads + h;
  // keys alone: a thread per key number and half (quarter) of the tokens
  {
    constexpr int PARTS = 256 / (KS * 64);
    const int d = tid % (KS * 64), part = tid / (KS * 64);
    float s = 0.f;
    for (int r = part * (kMlstmChunk / PARTS); r < (part + 1) * (kMlstmChunk / PARTS); ++r)
      s = fmaf(s_g[r], __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(smem + box_at<kMlstmChunk>(r, d >> 3) + (d & 7) * 2)), s);
    __shared__ float s_n[256];
    s_n[tid] = s;
    __syncthreads();
    if (tid < KS * 64 && tid < p.dim_p) {
#pragma unroll
      for (int x = 1; x < PARTS; ++x) s += s_n[x * KS * 64 + tid];
      p.loc_n[ch * p.dim_p + tid] = s;
    }
  }
  constexpr int GROUPS = 8 / (KS * 4), NT = VS * 8 / GROUPS;   // column groups; 8-column tiles of a warp
  const int m0 = warp % (KS * 4) * 16, n0 = warp / (KS * 4) * NT * 8;
  float acc[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
#pragma unroll 2
  for (int ks = 0; ks < kMlstmChunk / 16; ++ks) {
    uint32_t a[4];
    ldmatrix_x4_trans(sk + box_at<kMlstmChunk>(ks * 16 + (lane >> 4) * 8 + (lane & 7), (m0 >> 3) + ((lane >> 3) & 1)), a);
    const int vr = ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7);
#pragma unroll
    for (int j = 0; j < NT / 2; ++j) {
      const uint32_t at = sv + box_at<kMlstmChunk>(vr, (n0 >> 3) + 2 * j + (lane >> 4));
      uint32_t b[4];
      ldmatrix_x4_trans(at, b);
      mma_bf16(acc[2 * j], a, b[0], b[1]);
      mma_bf16(acc[2 * j + 1], a, b[2], b[3]);
      ldmatrix_x4_trans(at + C::V_BYTES, b);
      mma_bf16(acc[2 * j], a, b[0], b[1]);
      mma_bf16(acc[2 * j + 1], a, b[2], b[3]);
    }
  }
  float* out = p.loc + ch * p.dim_p * p.vdim_p;
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    const int c = n0 + j * 8 + 2 * (lane & 3);
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int d = m0 + (lane >> 2) + 8 * x;
      if (d < p.dim_p && c < p.vdim_p) *reinterpret_cast<float2*>(out + (long long)d * p.vdim_p + c) = make_float2(acc[j][2 * x], acc[j][2 * x + 1]);
    }
  }
}

// ---------------------------------------------------------------------------------------------------------
// scan: grid (pieces of 1024 numbers of the state, rows rounded up to 32 columns; then one for n and m; heads; portions)
// ---------------------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) mlstm_chunk_scan_kernel(const MlstmChunkParams p) {
  const int h = blockIdx.y, tid = threadIdx.x;
  const int4 seq = p.seqs[blockIdx.z];
  const int c0 = p.first[blockIdx.z], c1 = p.first[blockIdx.z + 1];
  const long long sh = (long long)seq.z * p.heads + h;
  const bool fresh = seq.w == 0;
  const int size = p.dim_p * p.vdim_p, wide = (p.vdim_p + 31) / 32 * 32;
  float m = fresh ? 0.f : p.m[sh];
  // factors of a chunk: {state, chunk's own sum}
  auto step = [&](float2 fg) {
    const float c = fmaxf(m, fg.y);
    const float2 w = make_float2(expf(m - c), expf(fg.y - c));
    m = fg.x + c;
    return w;
  };
  if (blockIdx.x < gridDim.x - 1) {
    const int x4 = (blockIdx.x * 256 + tid) * 4, d = x4 / wide, col = x4 % wide, i = d * p.vdim_p + col;
    const bool inside = d < p.dim_p, live = inside && col < p.vdim_p;
    uint8_t* out = p.s0 + (col >> 5) * 2 * p.dim_p * 64 + tile_at<4>(d, (col & 31) >> 3) + (col & 7) * 2;
    float4 s = !fresh && live ? *reinterpret_cast<const float4*>(p.S + sh * size + i) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int c = c0; c < c1; ++c) {
      const long long ch = (long long)c * p.heads + h;
      const float4 x = live ? *reinterpret_cast<const float4*>(p.loc + ch * size + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      const float2 w = step(p.loc_m[ch]);
      if (inside) {
        const SplitPair a = split2(s.x, s.y), b = split2(s.z, s.w);
        uint8_t* at = out + ch * 4 * p.dim_p * wide;
        *reinterpret_cast<uint2*>(at) = make_uint2(a.hi, b.hi);
        *reinterpret_cast<uint2*>(at + p.dim_p * 64) = make_uint2(a.lo, b.lo);
      }
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
// outputs: a CTA has one half of a chunk's tokens, a warp 16 of them and half of the columns.  Three rooms in shared memory
// are used one after another:
//   1  starting state, first half of each warp's columns, then the values
//   2  queries (until they are in registers), starting state, second half, then the output gates
//   3  keys
// ---------------------------------------------------------------------------------------------------------
template <int KS, int VS>
struct MlstmOutCfg {
  static constexpr int PLANE = KS * 64 * 64, STATE = 4 * PLANE;                // 2 x 32 columns of the state
  static constexpr int most(int a, int b) { return a > b ? a : b; }
  static constexpr int ROOM1 = most(STATE, 2 * VS * kMlstmBox), ROOM2 = most(STATE, most(KS, VS) * kMlstmBox), ROOM3 = 2 * KS * kMlstmBox;
  static constexpr int SMEM_BYTES = ROOM1 + ROOM2 + ROOM3 + 1024;
};

template <int KS, int VS>
__global__ void __launch_bounds__(256, 2)
    mlstm_chunk_out_kernel(const __grid_constant__ MlstmMaps maps, const MlstmChunkParams p, int* status) {
  using C = MlstmOutCfg<KS, VS>;
  constexpr int NT = VS * 4;                          // 8-column tiles of a warp
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  __shared__ float s_g[kMlstmChunk], s_c[kMlstmChunk], s_em[kMlstmChunk], s_n0[128], s_w[12], s_norm[VS * 64], s_sum[2][64];
  __shared__ uint64_t bars[6];
  __shared__ int s_abort;
  uint64_t *q_full = bars, *s_full = bars + 1, *k_full = bars + 3, *v_full = bars + 4, *gate_full = bars + 5;
  const int4 it = p.items[blockIdx.x >> 1];
  const int first = (blockIdx.x & 1) * 64;            // of the chunk's tokens
  if (first >= it.y) return;
  const int h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r = lane >> 2, c2 = (lane & 3) * 2;
  const int mt = warp & 3, ch_ = warp >> 2;           // 16 tokens, half of the columns
  const uint32_t r1 = smem_u32(smem), r2 = r1 + C::ROOM1, r3 = r2 + C::ROOM2;
  const long long ch = (long long)(blockIdx.x >> 1) * p.heads + h;
  const int blocks = (p.vdim_p + 31) / 32, key_boxes = first ? 2 : 1;
  // one thread: 32 columns `step` of both halves' share of the starting state, each two planes
  auto state = [&](int step) {
    const uint32_t bar = smem_u32(&s_full[step]), bytes = p.dim_p * 64, dst = step ? r2 : r1;
    const int there = (step < blocks) + (VS + step < blocks);
    mbar_arrive_expect_tx(bar, there * 2 * bytes);
    for (int x = 0; x < 2; ++x) {
      const int b = x * VS + step;
      if (b >= blocks) continue;
      const uint8_t* src = p.s0 + ch * 4 * p.dim_p * blocks * 32 + (long long)b * 2 * bytes;
      bulk_load_1d(dst + x * 2 * C::PLANE, src, bytes, bar);
      bulk_load_1d(dst + x * 2 * C::PLANE + C::PLANE, src + bytes, bytes, bar);
    }
  };
  if (tid == 0) {
    for (int b = 0; b < 6; ++b) mbar_init(smem_u32(&bars[b]), 1);
    s_abort = 0;
    fence_barrier_init();
    mbar_arrive_expect_tx(smem_u32(q_full), KS * kMlstmBox);
#pragma unroll
    for (int x = 0; x < KS; ++x) tma_load_3d(r2 + x * kMlstmBox, &maps.q, smem_u32(q_full), x * 64, it.x + first, h);
    state(0);
    mbar_arrive_expect_tx(smem_u32(k_full), KS * key_boxes * kMlstmBox);
#pragma unroll
    for (int x = 0; x < KS; ++x)
      for (int y = 0; y < key_boxes; ++y) tma_load_3d(r3 + (2 * x + y) * kMlstmBox, &maps.k, smem_u32(k_full), x * 64, it.x + y * 64, h);
  }
  // rows of the planes past the key size: zeros (queries have zeros there, but what lies there must be numbers)
  auto clear = [&](uint8_t* room) {
    for (int i = tid; i < 4 * (KS * 64 - p.dim_p) * 4; i += 256) {
      const int rest = (KS * 64 - p.dim_p) * 4, plane = i / rest, at = i % rest;
      *reinterpret_cast<uint4*>(room + plane * C::PLANE + p.dim_p * 64 + at * 16) = make_uint4(0, 0, 0, 0);
    }
  };
  clear(smem);
  if (tid < VS * 64) s_norm[tid] = tid < p.vdim_p ? p.o.norm[h * p.o.norm_step + tid] : 0.f;
  const float m0 = p.m0[ch];
  if (tid < 128) s_n0[tid] = tid < p.dim_p ? p.n0[ch * p.dim_p + tid] : 0.f;
  {
    const float2 fg = mlstm_chunk_gates(p, it, h, s_g, s_w);
    if (tid < kMlstmChunk) {
      const float c = fmaxf(m0, fg.y);
      s_c[tid] = c;
      s_em[tid] = expf(-(fg.x + c));
      // the last chunk leaves the state's m: the scan has read the old one
      if (tid == kMlstmChunk - 1 && first == 0 && (int)(blockIdx.x >> 1) == p.first[it.z + 1] - 1)
        p.m[(long long)p.seqs[it.z].z * p.heads + h] = fg.x + c;
    }
  }
  __syncthreads();
  bool ok = mbar_wait(smem_u32(q_full), 0, &s_abort, status, RB_ERR_TIMEOUT_FULL);
  uint32_t qa[KS * 4][4];
  float qn[2] = {0.f, 0.f};      // query . starting n, rows r and r + 8
#pragma unroll
  for (int k = 0; k < KS * 4; ++k) {
    ldmatrix_x4(r2 + box_at<64>(mt * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), k * 2 + (lane >> 4)), qa[k]);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 q = unpack2<__nv_bfloat16>(qa[k][e]);
      const int d = k * 16 + (e >> 1) * 8 + c2;
      qn[e & 1] = fmaf(q.x, s_n0[d], fmaf(q.y, s_n0[d + 1], qn[e & 1]));
    }
  }
  ok = __syncthreads_and(ok);
  if (VS == 2 && ok) {
    clear(smem + C::ROOM1);
    if (tid == 0) {
      fence_proxy_async_smem();
      state(1);
    }
  }
  float acc[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
#pragma unroll
  for (int step = 0; step < VS; ++step) {
    if (ok) ok = mbar_wait(smem_u32(&s_full[step]), 0, &s_abort, status, RB_ERR_TIMEOUT_FULL);
    if (step == 1) ok = __syncthreads_and(ok);       // the zeros below the planes are there
    const uint32_t sb = (step ? r2 : r1) + ch_ * 2 * C::PLANE;
    if (ok && ch_ * VS + step < blocks) {
#pragma unroll
      for (int k = 0; k < KS * 4; ++k) {
        const int d = k * 16 + ((lane >> 3) & 1) * 8 + (lane & 7);
        uint32_t x[4][4];                            // tiles 0 1 and 2 3, high and low planes
#pragma unroll
        for (int j = 0; j < 4; ++j) ldmatrix_x4_trans(sb + (j & 1) * C::PLANE + tile_at<4>(d, (j >> 1) * 2 + (lane >> 4)), x[j]);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          mma_bf16(acc[step * 4 + (j >> 1) * 2], qa[k], x[j][0], x[j][1]);
          mma_bf16(acc[step * 4 + (j >> 1) * 2 + 1], qa[k], x[j][2], x[j][3]);
        }
      }
    }
    ok = __syncthreads_and(ok);
    if (tid == 0 && ok) {
      if (step == 0) {
        mbar_arrive_expect_tx(smem_u32(v_full), VS * key_boxes * kMlstmBox);
#pragma unroll
        for (int x = 0; x < VS; ++x)
          for (int y = 0; y < key_boxes; ++y) tma_load_3d(r1 + (2 * x + y) * kMlstmBox, &maps.v, smem_u32(v_full), x * 64, it.x + y * 64, h);
      }
      if (step == VS - 1) {
        mbar_arrive_expect_tx(smem_u32(gate_full), VS * kMlstmBox);
#pragma unroll
        for (int x = 0; x < VS; ++x) tma_load_3d(r2 + x * kMlstmBox, &maps.gate, smem_u32(gate_full), x * 64, it.x + first, h);
      }
    }
  }
  const int t0 = first + mt * 16 + r;                 // this lane's tokens: t0 and t0 + 8
  float c[2], l[2];
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    c[x] = s_c[t0 + 8 * x];
    const float w = expf(m0 - c[x]) * p.q_scale;
    l[x] = qn[x] * w;
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      acc[j][2 * x] *= w;
      acc[j][2 * x + 1] *= w;
    }
  }
  if (ok) ok = mbar_wait(smem_u32(k_full), 0, &s_abort, status, RB_ERR_TIMEOUT_FULL);
  if (ok) ok = mbar_wait(smem_u32(v_full), 0, &s_abort, status, RB_ERR_TIMEOUT_FULL);
  ok = __all_sync(0xffffffffu, ok);
  const int last = ok ? (first >> 4) + mt : -1;
#pragma unroll 1
  for (int kb = 0; kb <= last; ++kb) {
    float s[2][2][4];                                 // even and odd steps apart: shorter chains
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[0][n][e] = s[1][n][e] = 0.f;
#pragma unroll
    for (int k = 0; k < KS * 4; ++k) {
      uint32_t x[4];
      ldmatrix_x4(r3 + box_at<kMlstmChunk>(kb * 16 + (lane >> 4) * 8 + (lane & 7), k * 2 + ((lane >> 3) & 1)), x);
      mma_bf16(s[k & 1][0], qa[k], x[0], x[1]);
      mma_bf16(s[k & 1][1], qa[k], x[2], x[3]);
    }
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      const float2 g = *reinterpret_cast<const float2*>(s_g + kb * 16 + n * 8 + c2);
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        float w[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int j = kb * 16 + n * 8 + c2 + e;
          w[e] = j <= t0 + 8 * x ? (s[0][n][2 * x + e] + s[1][n][2 * x + e]) * p.q_scale * __expf((e ? g.y : g.x) - c[x]) : 0.f;
          l[x] += w[e];
        }
        const SplitPair pr = split2(w[0], w[1]);
        hi[2 * n + x] = pr.hi;
        lo[2 * n + x] = pr.lo;
      }
    }
#pragma unroll
    for (int j = 0; j < NT / 2; ++j) {
      uint32_t x[4];
      ldmatrix_x4_trans(r1 + box_at<kMlstmChunk>(kb * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), ch_ * NT + 2 * j + (lane >> 4)), x);
      mma_bf16(acc[2 * j], hi, x[0], x[1]);
      mma_bf16(acc[2 * j + 1], hi, x[2], x[3]);
      mma_bf16(acc[2 * j], lo, x[0], x[1]);
      mma_bf16(acc[2 * j + 1], lo, x[2], x[3]);
    }
  }
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    l[x] += __shfl_xor_sync(0xffffffffu, l[x], 1);
    l[x] += __shfl_xor_sync(0xffffffffu, l[x], 2);
    const float inv = 1.0f / (fmaxf(fabsf(l[x]), s_em[t0 + 8 * x]) + 1e-6f);
    float sum = 0.f;
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        acc[j][2 * x + e] *= inv;
        sum = fmaf(acc[j][2 * x + e], acc[j][2 * x + e], sum);
      }
    sum += __shfl_xor_sync(0xffffffffu, sum, 1);
    sum += __shfl_xor_sync(0xffffffffu, sum, 2);
    if ((lane & 3) == 0) s_sum[ch_][mt * 16 + r + 8 * x] = sum;
  }
  if (ok) ok = mbar_wait(smem_u32(gate_full), 0, &s_abort, status, RB_ERR_TIMEOUT_FULL);
  if (!__syncthreads_and(ok)) return;
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const int tr = mt * 16 + r + 8 * x;               // row of the CTA
    if (first + tr >= it.y) continue;
    const float scale = 1.0f / sqrtf((s_sum[0][tr] + s_sum[1][tr]) / p.vdim + p.o.eps);
    __nv_bfloat16* out = p.o.out + (long long)(it.x + first + tr) * p.o.ldo + (long long)h * p.vdim_p;
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int col = (ch_ * NT + j) * 8 + c2;
      if (col >= p.vdim_p) break;
      const float2 g = unpack2<__nv_bfloat16>(*reinterpret_cast<const uint32_t*>(smem + C::ROOM1 + box_at<64>(tr, col >> 3) + (col & 7) * 2));
      const float2 w = *reinterpret_cast<const float2*>(s_norm + col);
      *reinterpret_cast<uint32_t*>(out + col) = pack2<__nv_bfloat16>(acc[j][2 * x] * scale * w.x * sigmoid_tanh(g.x),
                                                                     acc[j][2 * x + 1] * scale * w.y * sigmoid_tanh(g.y));
    }
  }
}

template <int KS, int VS>
int launch_mlstm_chunk(const MlstmChunkParams& p, int tokens, int n_items, int portions, cudaStream_t st) {
  MlstmMaps maps;
  auto map = [&](CUtensorMap* m, const __nv_bfloat16* base, long long ld, int cols) {
    uint64_t dims[3] = {(uint64_t)cols, (uint64_t)tokens, (uint64_t)p.heads};
    uint64_t strides[3] = {2, (uint64_t)ld * 2, (uint64_t)cols * 2};
    uint32_t box[3] = {64, 64, 1};
    return rbh::encode_tensor_map(m, rbh::DT_BF16, 3, const_cast<__nv_bfloat16*>(base), dims, strides, box, 1);
  };
  int rc = map(&maps.q, p.proj, p.ldp, p.dim_p);
  if (!rc) rc = map(&maps.k, p.proj + (long long)p.heads * p.dim_p, p.ldp, p.dim_p);
  if (!rc) rc = map(&maps.v, p.proj + 2LL * p.heads * p.dim_p, p.ldp, p.vdim_p);
  if (!rc) rc = map(&maps.gate, p.o.gate, p.o.ldg, p.vdim_p);
  if (rc) return 1000 + rc;
  auto states = mlstm_chunk_states_kernel<KS, VS>;
  auto outputs = mlstm_chunk_out_kernel<KS, VS>;
  cudaError_t e = cudaFuncSetAttribute(states, cudaFuncAttributeMaxDynamicSharedMemorySize, MlstmStateCfg<KS, VS>::SMEM_BYTES);
  if (e == cudaSuccess) e = cudaFuncSetAttribute(outputs, cudaFuncAttributeMaxDynamicSharedMemorySize, MlstmOutCfg<KS, VS>::SMEM_BYTES);
  if (e != cudaSuccess) return 2000 + (int)e;
  int* status = rbh::device_status_word();
  states<<<dim3(n_items, p.heads), 256, MlstmStateCfg<KS, VS>::SMEM_BYTES, st>>>(maps, p, status);
  mlstm_chunk_scan_kernel<<<dim3((p.dim_p * ((p.vdim_p + 31) / 32 * 32) + 1023) / 1024 + 1, p.heads, portions), 256, 0, st>>>(p);
  outputs<<<dim3(2 * n_items, p.heads), 256, MlstmOutCfg<KS, VS>::SMEM_BYTES, st>>>(maps, p, status);
  e = cudaGetLastError();
  return e == cudaSuccess ? 0 : 3000 + (int)e;
}

}  // namespace rb

extern "C" {

// Whether the kernels cover these sizes (others run token by token).
int rb_mlstm_chunk_ok(int dtype, int dim_p, int vdim_p) {
  return dtype == rbh::DT_BF16 && dim_p <= 128 && vdim_p <= 128 && dim_p % 8 == 0 && vdim_p % 8 == 0;
}

// tokens: rows of proj and gate; items: chunks of up to 128 tokens; first: [portions + 1].  Scratch by chunk and head: loc dim_p * vdim_p floats, loc_n and
// n0 dim_p, loc_m 2, m0 1, s0 4 * dim_p * (vdim_p rounded up to 32) bytes.  Otherwise as rb_mlstm_rows.
int rb_mlstm_chunk(int dtype, const void* proj, long long ldp, int tokens, const float* gates, long long ldz, const int* items, int n_items,
                   const int* seqs, const int* first, int portions, float* S, float* n, float* m, const void* gate, long long ldg,
                   const float* norm, void* out, long long ldo, float* loc, float* loc_n, float* loc_m, void* s0, float* n0, float* m0,
                   int heads, int dim_p, int vdim_p, int vdim, float q_scale, float cap, float eps, void* stream) {
  using namespace rb;
  if (n_items <= 0) return 0;
  auto al = [](const void* x, int to) { return (reinterpret_cast<uintptr_t>(x) & (to - 1)) == 0; };
  if (!rb_mlstm_chunk_ok(dtype, dim_p, vdim_p) || heads > 65535 || portions > 65535) return 22;
  if (!al(proj, 16) || !al(gate, 16) || !al(out, 4) || !al(norm, 8) || !al(loc, 16) || !al(s0, 16) || !al(loc_m, 8) || ldp % 8 || ldg % 8 || ldo % 2)
    return 21;
  using T = __nv_bfloat16;
  const MlstmChunkParams p{(const T*)proj, ldp, gates, ldz, (const int4*)items, (const int4*)seqs, first, S, n, m, loc, loc_n, (float2*)loc_m,
                           (uint8_t*)s0, n0, m0, heads, dim_p, vdim_p, vdim, q_scale, cap,
                           {(T*)out, ldo, (const T*)gate, ldg, norm, vdim_p, nullptr, eps}};
  cudaStream_t st = (cudaStream_t)stream;
  if (dim_p <= 64) return vdim_p <= 64 ? launch_mlstm_chunk<1, 1>(p, tokens, n_items, portions, st) : launch_mlstm_chunk<1, 2>(p, tokens, n_items, portions, st);
  return vdim_p <= 64 ? launch_mlstm_chunk<2, 1>(p, tokens, n_items, portions, st) : launch_mlstm_chunk<2, 2>(p, tokens, n_items, portions, st);
}
}
