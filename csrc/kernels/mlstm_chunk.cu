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
  static constexpr int SMEM_BYTES = K_BYTES + 2 * V_BYTES + 128;
};

template <int KS, int VS>
__global__ void __launch_bounds__(256, 2) mlstm_chunk_states_kernel(const MlstmChunkParams p) {
  using C = MlstmStateCfg<KS, VS>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 127) & ~static_cast<uintptr_t>(127));
  __shared__ float s_g[kMlstmChunk], s_w[12];
  const int4 it = p.items[blockIdx.x];
  const int h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t sk = smem_u32(smem), sv = sk + C::K_BYTES;
  const __nv_bfloat16* base = p.proj + (long long)it.x * p.ldp;
  for (int i = tid; i < kMlstmChunk * KS * 8; i += 256) {
    const int r = i / (KS * 8), c = i % (KS * 8);
    const bool live = r < it.y && c * 8 < p.dim_p;
    copy16(sk + tile_at<KS * 8>(r, c), base + (live ? r * p.ldp + (p.heads + h) * p.dim_p + c * 8 : 0), live);
  }
  copy_commit();
  // values wait in registers for their weights
  constexpr int NV = kMlstmChunk * VS * 8 / 256;
  uint4 v[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int x = i * 256 + tid, r = x / (VS * 8), c = x % (VS * 8);
    v[i] = r < it.y && c * 8 < p.vdim_p
               ? *reinterpret_cast<const uint4*>(base + r * p.ldp + 2LL * p.heads * p.dim_p + (long long)h * p.vdim_p + c * 8)
               : make_uint4(0, 0, 0, 0);
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
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int x = i * 256 + tid, r = x / (VS * 8), c = x % (VS * 8);
    const float w = s_g[r];
    uint4 hi, lo;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 q = unpack2<__nv_bfloat16>(reinterpret_cast<const uint32_t*>(&v[i])[e]);
      const SplitPair s = split2(q.x * w, q.y * w);
      reinterpret_cast<uint32_t*>(&hi)[e] = s.hi;
      reinterpret_cast<uint32_t*>(&lo)[e] = s.lo;
    }
    const uint32_t at = tile_at<VS * 8>(r, c);
    *reinterpret_cast<uint4*>(smem + C::K_BYTES + at) = hi;
    *reinterpret_cast<uint4*>(smem + C::K_BYTES + C::V_BYTES + at) = lo;
  }
  copy_wait<0>();
  __syncthreads();
  const long long ch = (long long)blockIdx.x * p.heads + h;
  // keys alone: a thread per key number and half (quarter) of the tokens
  {
    constexpr int PARTS = 256 / (KS * 64);
    const int d = tid % (KS * 64), part = tid / (KS * 64);
    float s = 0.f;
    for (int r = part * (kMlstmChunk / PARTS); r < (part + 1) * (kMlstmChunk / PARTS); ++r)
      s = fmaf(s_g[r], __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(smem + tile_at<KS * 8>(r, d >> 3) + (d & 7) * 2)), s);
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
    ldmatrix_x4_trans(sk + tile_at<KS * 8>(ks * 16 + (lane >> 4) * 8 + (lane & 7), (m0 >> 3) + ((lane >> 3) & 1)), a);
    const int vr = ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7);
#pragma unroll
    for (int j = 0; j < NT / 2; ++j) {
      const uint32_t at = sv + tile_at<VS * 8>(vr, (n0 >> 3) + 2 * j + (lane >> 4));
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
// outputs: a warp has 16 of the chunk's tokens
// ---------------------------------------------------------------------------------------------------------
template <int KS, int VS>
struct MlstmOutCfg {
  static constexpr int Q_BYTES = kMlstmChunk * KS * 128, V_BYTES = kMlstmChunk * VS * 128;
  static constexpr int QV_BYTES = Q_BYTES > V_BYTES ? Q_BYTES : V_BYTES;       // values go where the queries were
  static constexpr int PLANE = KS * 64 * 64;                                   // 32 columns of the state, two stages
  static constexpr int RING = 4 * PLANE > V_BYTES ? 4 * PLANE : V_BYTES;       // the output gates go there at the end
  static constexpr int SMEM_BYTES = QV_BYTES + Q_BYTES + RING + 128;
};

template <int KS, int VS>
__global__ void __launch_bounds__(256, 2) mlstm_chunk_out_kernel(const MlstmChunkParams p, int* status) {
  using C = MlstmOutCfg<KS, VS>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 127) & ~static_cast<uintptr_t>(127));
  __shared__ float s_g[kMlstmChunk], s_c[kMlstmChunk], s_em[kMlstmChunk], s_n0[128], s_w[12], s_norm[VS * 64];
  __shared__ uint64_t full[VS * 2];
  __shared__ int s_abort;
  const int4 it = p.items[blockIdx.x];
  const int h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r = lane >> 2, c2 = (lane & 3) * 2;
  const uint32_t sq = smem_u32(smem), sk = sq + C::QV_BYTES, ss = sk + C::Q_BYTES;
  const long long ch = (long long)blockIdx.x * p.heads + h;
  const int blocks = (p.vdim_p + 31) / 32;
  const __nv_bfloat16* base = p.proj + (long long)it.x * p.ldp;
  auto rows = [&](uint32_t dst, const __nv_bfloat16* src, long long ld, long long col, int cols, auto chunks) {
    constexpr int N = decltype(chunks)::value;
    for (int i = tid; i < kMlstmChunk * N; i += 256) {
      const int row = i / N, c = i % N;
      const bool live = row < it.y && c * 8 < cols;
      copy16(dst + tile_at<N>(row, c), src + (live ? row * ld + col + c * 8 : 0), live);
    }
  };
  if (tid == 0) {
    for (int b = 0; b < VS * 2; ++b) mbar_init(smem_u32(&full[b]), 1);
    s_abort = 0;
    fence_barrier_init();
  }
  for (int i = tid; i < 4 * (KS * 64 - p.dim_p) * 4; i += 256) {       // rows of the planes past the key size: zeros
    const int rest = (KS * 64 - p.dim_p) * 4, plane = i / rest, at = i % rest;
    *reinterpret_cast<uint4*>(smem + C::QV_BYTES + C::Q_BYTES + plane * C::PLANE + p.dim_p * 64 + at * 16) = make_uint4(0, 0, 0, 0);
  }
  if (tid < VS * 64) s_norm[tid] = tid < p.vdim_p ? p.o.norm[h * p.o.norm_step + tid] : 0.f;
  __syncthreads();
  // one thread: columns 32 b .. 32 b + 31 of both planes of the starting state
  auto state = [&](int b) {
    const uint32_t bar = smem_u32(&full[b]), dst = ss + (b & 1) * 2 * C::PLANE, bytes = p.dim_p * 64;
    const uint8_t* src = p.s0 + ch * 4 * p.dim_p * blocks * 32 + (long long)b * 2 * bytes;
    mbar_arrive_expect_tx(bar, 2 * bytes);
    bulk_load_1d(dst, src, bytes, bar);
    bulk_load_1d(dst + C::PLANE, src + bytes, bytes, bar);
  };
  if (tid == 0) {
    state(0);
    if (blocks > 1) state(1);
  }
  rows(sq, base, p.ldp, (long long)h * p.dim_p, p.dim_p, std::integral_constant<int, KS * 8>{});
  copy_commit();
  rows(sk, base, p.ldp, (long long)(p.heads + h) * p.dim_p, p.dim_p, std::integral_constant<int, KS * 8>{});
  copy_commit();
  const float m0 = p.m0[ch];
  if (tid < 128) s_n0[tid] = tid < p.dim_p ? p.n0[ch * p.dim_p + tid] : 0.f;
  {
    const float2 fg = mlstm_chunk_gates(p, it, h, s_g, s_w);
    if (tid < kMlstmChunk) {
      const float c = fmaxf(m0, fg.y);
      s_c[tid] = c;
      s_em[tid] = expf(-(fg.x + c));
      // the last chunk leaves the state's m: the scan has read the old one
      if (tid == kMlstmChunk - 1 && (int)blockIdx.x == p.first[it.z + 1] - 1) p.m[(long long)p.seqs[it.z].z * p.heads + h] = fg.x + c;
    }
  }
  copy_wait<1>();
  __syncthreads();
  uint32_t qa[KS * 4][4];
  float qn[2] = {0.f, 0.f};      // query . starting n, rows r and r + 8
#pragma unroll
  for (int k = 0; k < KS * 4; ++k) {
    ldmatrix_x4(sq + tile_at<KS * 8>(warp * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), k * 2 + (lane >> 4)), qa[k]);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 q = unpack2<__nv_bfloat16>(qa[k][e]);
      const int d = k * 16 + (e >> 1) * 8 + c2;
      qn[e & 1] = fmaf(q.x, s_n0[d], fmaf(q.y, s_n0[d + 1], qn[e & 1]));
    }
  }
  __syncthreads();
  rows(sq, base, p.ldp, 2LL * p.heads * p.dim_p + (long long)h * p.vdim_p, p.vdim_p, std::integral_constant<int, VS * 8>{});
  copy_commit();
  float acc[VS * 8][4];
  bool ok = true;
#pragma unroll
  for (int b = 0; b < VS * 2; ++b) {
#pragma unroll
    for (int j = b * 4; j < b * 4 + 4; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
    if (b >= blocks || !ok) continue;
    ok = mbar_wait(smem_u32(&full[b]), 0, &s_abort, status, RB_ERR_TIMEOUT_FULL);
    const uint32_t sb = ss + (b & 1) * 2 * C::PLANE;
#pragma unroll
    for (int k = 0; k < KS * 4; ++k) {
      const int d = k * 16 + ((lane >> 3) & 1) * 8 + (lane & 7);
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const uint32_t at = sb + tile_at<4>(d, 2 * j + (lane >> 4));
        uint32_t x[4];
        ldmatrix_x4_trans(at, x);
        mma_bf16(acc[b * 4 + 2 * j], qa[k], x[0], x[1]);
        mma_bf16(acc[b * 4 + 2 * j + 1], qa[k], x[2], x[3]);
        ldmatrix_x4_trans(at + C::PLANE, x);
        mma_bf16(acc[b * 4 + 2 * j], qa[k], x[0], x[1]);
        mma_bf16(acc[b * 4 + 2 * j + 1], qa[k], x[2], x[3]);
      }
    }
    ok = __syncthreads_and(ok);
    if (ok && tid == 0 && b + 2 < blocks) state(b + 2);
  }
  // the gates come while the chunk's own part is computed
  rows(ss, p.o.gate + (long long)it.x * p.o.ldg, p.o.ldg, (long long)h * p.vdim_p, p.vdim_p, std::integral_constant<int, VS * 8>{});
  copy_commit();
  copy_wait<1>();
  __syncthreads();
  const int t0 = warp * 16 + r;                       // this lane's tokens: t0 and t0 + 8
  float c[2], l[2];
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    c[x] = s_c[t0 + 8 * x];
    const float w = expf(m0 - c[x]) * p.q_scale;
    l[x] = qn[x] * w;
#pragma unroll
    for (int j = 0; j < VS * 8; ++j) {
      acc[j][2 * x] *= w;
      acc[j][2 * x + 1] *= w;
    }
  }
  for (int kb = 0; kb <= warp; ++kb) {
    float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
    for (int k = 0; k < KS * 4; ++k) {
      uint32_t x[4];
      ldmatrix_x4(sk + tile_at<KS * 8>(kb * 16 + (lane >> 4) * 8 + (lane & 7), k * 2 + ((lane >> 3) & 1)), x);
      mma_bf16(s[0], qa[k], x[0], x[1]);
      mma_bf16(s[1], qa[k], x[2], x[3]);
    }
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        float w[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int j = kb * 16 + n * 8 + c2 + e;
          w[e] = j <= t0 + 8 * x ? s[n][2 * x + e] * p.q_scale * __expf(s_g[j] - c[x]) : 0.f;
          l[x] += w[e];
        }
        const SplitPair pr = split2(w[0], w[1]);
        hi[2 * n + x] = pr.hi;
        lo[2 * n + x] = pr.lo;
      }
#pragma unroll
    for (int j = 0; j < VS * 4; ++j) {
      uint32_t x[4];
      ldmatrix_x4_trans(sq + tile_at<VS * 8>(kb * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), 2 * j + (lane >> 4)), x);
      mma_bf16(acc[2 * j], hi, x[0], x[1]);
      mma_bf16(acc[2 * j + 1], hi, x[2], x[3]);
      mma_bf16(acc[2 * j], lo, x[0], x[1]);
      mma_bf16(acc[2 * j + 1], lo, x[2], x[3]);
    }
  }
  copy_wait<0>();
  __syncthreads();
  if (!ok) return;
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    l[x] += __shfl_xor_sync(0xffffffffu, l[x], 1);
    l[x] += __shfl_xor_sync(0xffffffffu, l[x], 2);
    const int t = t0 + 8 * x;
    const float inv = 1.0f / (fmaxf(fabsf(l[x]), s_em[t]) + 1e-6f);
    float sum = 0.f;
#pragma unroll
    for (int j = 0; j < VS * 8; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        acc[j][2 * x + e] *= inv;
        sum = fmaf(acc[j][2 * x + e], acc[j][2 * x + e], sum);
      }
    sum += __shfl_xor_sync(0xffffffffu, sum, 1);
    sum += __shfl_xor_sync(0xffffffffu, sum, 2);
    const float scale = 1.0f / sqrtf(sum / p.vdim + p.o.eps);
    if (t >= it.y) continue;
    const long long row = it.x + t;
    __nv_bfloat16* out = p.o.out + row * p.o.ldo + (long long)h * p.vdim_p;
#pragma unroll
    for (int j = 0; j < VS * 8; ++j) {
      const int col = j * 8 + c2;
      if (col >= p.vdim_p) break;
      const float2 g = unpack2<__nv_bfloat16>(
          *reinterpret_cast<const uint32_t*>(smem + C::QV_BYTES + C::Q_BYTES + tile_at<VS * 8>(t, col >> 3) + (col & 7) * 2));
      *reinterpret_cast<uint32_t*>(out + col) =
          pack2<__nv_bfloat16>(acc[j][2 * x] * scale * s_norm[col] * rec_sigmoid<__nv_bfloat16>(g.x),
                               acc[j][2 * x + 1] * scale * s_norm[col + 1] * rec_sigmoid<__nv_bfloat16>(g.y));
    }
  }
}

template <int KS, int VS>
int launch_mlstm_chunk(const MlstmChunkParams& p, int n_items, int portions, cudaStream_t st) {
  auto states = mlstm_chunk_states_kernel<KS, VS>;
  auto outputs = mlstm_chunk_out_kernel<KS, VS>;
  cudaError_t e = cudaFuncSetAttribute(states, cudaFuncAttributeMaxDynamicSharedMemorySize, MlstmStateCfg<KS, VS>::SMEM_BYTES);
  if (e == cudaSuccess) e = cudaFuncSetAttribute(outputs, cudaFuncAttributeMaxDynamicSharedMemorySize, MlstmOutCfg<KS, VS>::SMEM_BYTES);
  if (e != cudaSuccess) return 2000 + (int)e;
  states<<<dim3(n_items, p.heads), 256, MlstmStateCfg<KS, VS>::SMEM_BYTES, st>>>(p);
  mlstm_chunk_scan_kernel<<<dim3((p.dim_p * ((p.vdim_p + 31) / 32 * 32) + 1023) / 1024 + 1, p.heads, portions), 256, 0, st>>>(p);
  outputs<<<dim3(n_items, p.heads), 256, MlstmOutCfg<KS, VS>::SMEM_BYTES, st>>>(p, rbh::device_status_word());
  e = cudaGetLastError();
  return e == cudaSuccess ? 0 : 3000 + (int)e;
}

}  // namespace rb

extern "C" {

// Whether the kernels cover these sizes (others run token by token).
int rb_mlstm_chunk_ok(int dtype, int dim_p, int vdim_p) {
  return dtype == rbh::DT_BF16 && dim_p <= 128 && vdim_p <= 128 && dim_p % 8 == 0 && vdim_p % 8 == 0;
}

// items: chunks of up to 128 tokens; first: [portions + 1].  Scratch by chunk and head: loc dim_p * vdim_p floats, loc_n and
// n0 dim_p, loc_m 2, m0 1, s0 4 * dim_p * (vdim_p rounded up to 32) bytes.  Otherwise as rb_mlstm_rows.
int rb_mlstm_chunk(int dtype, const void* proj, long long ldp, const float* gates, long long ldz, const int* items, int n_items,
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
  if (dim_p <= 64) return vdim_p <= 64 ? launch_mlstm_chunk<1, 1>(p, n_items, portions, st) : launch_mlstm_chunk<1, 2>(p, n_items, portions, st);
  return vdim_p <= 64 ? launch_mlstm_chunk<2, 1>(p, n_items, portions, st) : launch_mlstm_chunk<2, 2>(p, n_items, portions, st);
}
}
