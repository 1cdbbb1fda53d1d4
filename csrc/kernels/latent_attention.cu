// Attention over a compressed key/value latent, sm_100a: everything around the tensor-core kernels
// (latent_prefill.cu, latent_decode.cu), and a plain kernel that covers every size and type.
//
// A token leaves one cache row [latent (rank) | key part shared by all heads (rot)] per layer, both parts
// padded to multiples of eight numbers with zeros.  Per head, the key is W_uk c next to the shared part and
// the value is W_uv c.  Decoding never writes keys or values out: q . (W_uk c) = (W_uk^T q) . c, so a query
// is carried into latent space once, all heads attend to the same rows, and the weighted sum of latents goes
// through W_uv at the end.
//
// Cache layout: pool [num_blocks, block_size, row]; token t of a sequence is in block table[t / block_size].
#include "attn_merge.cuh"

namespace rb {

// ---------------------------------------------------------------------------------------------------------
// rotation table: tab[t][i] = (cos, sin)(pos[t] * freq[i]) * mscale
// ---------------------------------------------------------------------------------------------------------
__global__ void rotary_table_kernel(const long long* __restrict__ pos, const float* __restrict__ freq,
                                    float2* __restrict__ tab, long long n, int pairs, float mscale) {
  const long long stride = (long long)gridDim.x * blockDim.x;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += stride) {
    const long long t = i / pairs;
    float s, c;
    sincosf((float)pos[t] * freq[i - t * pairs], &s, &c);
    tab[i] = make_float2(c * mscale, s * mscale);
  }
}

// ---------------------------------------------------------------------------------------------------------
// after the input projection: rotate the queries' rotated parts in place; norm the latent, rotate the shared
// key part and put both into the cache.  One CTA per token.
//   proj row: [heads x (dim_p + rot_p)] queries, then (own latents only) [rank_p + rot_p]
// ---------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(128)
    latent_post_kernel(T* __restrict__ proj, long long ldp, const float2* __restrict__ tab,
                       const float* __restrict__ norm_w, const long long* __restrict__ slots, T* __restrict__ pool,
                       int heads, int dim_p, int rot, int rot_p, int kv_col, int rank, int rank_p, float eps) {
  __shared__ float red[4];
  const long long t = blockIdx.x;
  T* row = proj + t * ldp;
  const int half = rot >> 1, tid = threadIdx.x;
  const float2* tb = tab + t * half;
  for (int i = tid; i < heads * half; i += 128) {
    const int h = i / half, p = i - h * half;
    T* b = row + (long long)h * (dim_p + rot_p) + dim_p + 2 * p;
    const float u = to_f32<T>(b[0]), v = to_f32<T>(b[1]);
    const float2 cs = tb[p];
    b[0] = from_f32<T>(u * cs.x - v * cs.y);
    b[1] = from_f32<T>(v * cs.x + u * cs.y);
  }
  if (kv_col < 0) return;
  const T* z = row + kv_col;
  float s = 0.f;
  for (int c = tid; c < rank; c += 128) {
    const float v = to_f32<T>(z[c]);
    s += v * v;
  }
  s = warp_sum(s);
  if ((tid & 31) == 0) red[tid >> 5] = s;
  __syncthreads();
  s = red[0] + red[1] + red[2] + red[3];
  const float r = 1.0f / sqrtf(s / rank + eps);
  const long long slot = slots[t];
  if (slot < 0) return;
  T* o = pool + slot * (rank_p + rot_p);
  for (int c = tid; c < rank_p; c += 128) o[c] = from_f32<T>(c < rank ? to_f32<T>(z[c]) * r * norm_w[c] : 0.f);
  for (int c = 2 * tid; c < rot_p; c += 256) {
    const int p = c >> 1;
    float a = 0.f, b = 0.f;
    if (p < half) {
      const float u = to_f32<T>(z[rank_p + c]), v = to_f32<T>(z[rank_p + c + 1]);
      const float2 cs = tb[p];
      a = u * cs.x - v * cs.y;
      b = v * cs.x + u * cs.y;
    }
    o[rank_p + c] = from_f32<T>(a);
    o[rank_p + c + 1] = from_f32<T>(b);
  }
}

// ---------------------------------------------------------------------------------------------------------
// rows of several sequences' prefixes, one behind the other: out[i] = pool row of token i of its segment
//   seg_off[s] = first output row of segment s (seg_off[n_seg] = total)
// ---------------------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256)
    latent_gather_kernel(const uint4* __restrict__ pool, const int* __restrict__ tables, const int* __restrict__ seg_off,
                         uint4* __restrict__ out, int n_seg, int max_blocks, int block_size, int vecs, long long total) {
  const long long n = total * vecs;
  const long long stride = (long long)gridDim.x * blockDim.x;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += stride) {
    const long long r = i / vecs;
    const int c = (int)(i - r * vecs);
    int s = 0;
    while (s + 1 < n_seg && r >= seg_off[s + 1]) ++s;
    const int t = (int)(r - seg_off[s]);
    const long long blk = tables[(long long)s * max_blocks + t / block_size];
    out[i] = pool[(blk * block_size + t % block_size) * vecs + c];
  }
}

// ---------------------------------------------------------------------------------------------------------
// plain attention of single query rows over latent rows: any sizes, any type; fp32 scores and sums.
// grid (heads, rows, splits), 4 warps; a warp takes one key at a time, lanes share the row's numbers.
//   qa [rows, heads, rank_p] queries in latent space, qr: rotated parts (row stride ldq, head stride hq)
//   part_o [rows, heads, splits, rank_p], part_ml [rows, heads, splits, 2] (maximum in log2 units, sum)
// ---------------------------------------------------------------------------------------------------------
template <typename T, int NR>
__global__ void __launch_bounds__(128)
    latent_rows_kernel(const T* __restrict__ qa, const T* __restrict__ qr, long long ldq, int hq,
                       const T* __restrict__ pool, const int* __restrict__ tables, const int* __restrict__ ctx_lens,
                       float* __restrict__ part_o, float* __restrict__ part_ml, int heads, int rank_p, int rot_p,
                       int block_size, int max_blocks, int splits, float scale_log2) {
  extern __shared__ float sm[];            // query [rank_p + rot_p], then per-warp sums [4][rank_p]
  __shared__ float s_m[4], s_l[4];
  const int h = blockIdx.x, sp = blockIdx.z;
  const long long b = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row = rank_p + rot_p;
  const int ctx = ctx_lens[b];
  const int per = (ctx + splits - 1) / splits;
  const int t0 = sp * per, t1 = min(ctx, t0 + per);
  for (int c = threadIdx.x; c < row; c += 128)
    sm[c] = (c < rank_p ? to_f32<T>(qa[(b * heads + h) * rank_p + c]) : to_f32<T>(qr[b * ldq + (long long)h * hq + c - rank_p])) * scale_log2;
  __syncthreads();
  const int* table = tables + b * max_blocks;
  float m = -INFINITY, l = 0.f, acc[NR];
#pragma unroll
  for (int j = 0; j < NR; ++j) acc[j] = 0.f;
  for (int t = t0 + warp; t < t1; t += 4) {
    const T* kv = pool + ((long long)table[t / block_size] * block_size + t % block_size) * row;
    float s = 0.f, c[NR];
#pragma unroll
    for (int j = 0; j < NR; ++j) {
      const int d = j * 32 + lane;
      c[j] = d < rank_p ? to_f32<T>(kv[d]) : 0.f;
      if (d < rank_p) s = fmaf(sm[d], c[j], s);
    }
    for (int d = rank_p + lane; d < row; d += 32) s = fmaf(sm[d], to_f32<T>(kv[d]), s);
    s = warp_sum(s);
    const float mn = fmaxf(m, s);
    const float corr = exp2f(m - mn), p = exp2f(s - mn);
    l = l * corr + p;
#pragma unroll
    for (int j = 0; j < NR; ++j) acc[j] = acc[j] * corr + p * c[j];
    m = mn;
  }
  float* so = sm + row + warp * rank_p;
#pragma unroll
  for (int j = 0; j < NR; ++j)
    if (j * 32 + lane < rank_p) so[j * 32 + lane] = acc[j];
  if (lane == 0) { s_m[warp] = m; s_l[warp] = l; }
  __syncthreads();
  const float gm = fmaxf(fmaxf(s_m[0], s_m[1]), fmaxf(s_m[2], s_m[3]));
  float f[4], gl = 0.f;
#pragma unroll
  for (int w = 0; w < 4; ++w) {
    f[w] = s_m[w] == -INFINITY ? 0.f : exp2f(s_m[w] - gm);
    gl += s_l[w] * f[w];
  }
  const long long pi = (b * heads + h) * splits + sp;
  for (int d = threadIdx.x; d < rank_p; d += 128) {
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) o += sm[row + w * rank_p + d] * f[w];
    part_o[pi * rank_p + d] = o;
  }
  if (threadIdx.x == 0) { part_ml[pi * 2] = gm; part_ml[pi * 2 + 1] = gl; }
}

// x[r, c] *= sigmoid(g[r, c]) in place
template <typename T>
__global__ void __launch_bounds__(256)
    sigmoid_gate_kernel(T* __restrict__ x, long long ldx, const T* __restrict__ g, long long ldg, long long rows, int n) {
  const long long total = rows * n, stride = (long long)gridDim.x * blockDim.x;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += stride) {
    const long long r = i / n;
    const int c = (int)(i - r * n);
    const float z = to_f32<T>(g[r * ldg + c]);
    x[r * ldx + c] = from_f32<T>(to_f32<T>(x[r * ldx + c]) / (1.0f + expf(-z)));
  }
}

static unsigned grid_for(long long n, int threads) {
  const long long b = (n + threads - 1) / threads;
  return (unsigned)(b < 1 ? 1 : b < 148 * 32 ? b : 148 * 32);
}

template <typename T>
int launch_latent_rows(const T* qa, const T* qr, long long ldq, int hq, const T* pool, const int* tables,
                       const int* ctx, float* part_o, float* part_ml, int rows, int heads, int rank_p, int rot_p,
                       int block_size, int max_blocks, int splits, float scale, cudaStream_t st) {
  const size_t smem = (size_t)(rank_p + rot_p + 4 * rank_p) * 4;
  if (smem > 200 * 1024) return 22;
  const float sl2 = scale * 1.4426950408889634f;
  dim3 grid(heads, rows, splits);
  auto go = [&](auto kern) -> int {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return 2000 + (int)e;
    kern<<<grid, 128, smem, st>>>(qa, qr, ldq, hq, pool, tables, ctx, part_o, part_ml, heads, rank_p, rot_p,
                                  block_size, max_blocks, splits, sl2);
    e = cudaGetLastError();
    return e == cudaSuccess ? 0 : 3000 + (int)e;
  };
  if (rank_p <= 64) return go(latent_rows_kernel<T, 2>);
  if (rank_p <= 128) return go(latent_rows_kernel<T, 4>);
  if (rank_p <= 256) return go(latent_rows_kernel<T, 8>);
  if (rank_p <= 512) return go(latent_rows_kernel<T, 16>);
  if (rank_p <= 1024) return go(latent_rows_kernel<T, 32>);
  if (rank_p <= 2048) return go(latent_rows_kernel<T, 64>);
  return 22;
}

}  // namespace rb

#define RB_BY_DTYPE(CALL)                                       \
  if (dtype == rbh::DT_BF16) { using T = __nv_bfloat16; CALL; } \
  else if (dtype == rbh::DT_F16) { using T = __half; CALL; }    \
  else if (dtype == rbh::DT_F32) { using T = float; CALL; }     \
  else return 20;
#define RB_LAUNCH_STATUS()             \
  cudaError_t e_ = cudaGetLastError(); \
  return e_ == cudaSuccess ? 0 : 3000 + (int)e_

extern "C" {

int rb_rotary_table(const long long* pos, const float* freq, float* tab, long long tokens, int pairs, float mscale,
                    void* stream) {
  using namespace rb;
  if (tokens <= 0 || pairs <= 0) return 0;
  rotary_table_kernel<<<grid_for(tokens * pairs, 256), 256, 0, (cudaStream_t)stream>>>(pos, freq, (float2*)tab, tokens * pairs, pairs, mscale);
  RB_LAUNCH_STATUS();
}

// kv_col: column of the latents in proj, or -1 when the layer keeps none
int rb_latent_post(int dtype, void* proj, long long ldp, const float* tab, const float* norm_w, const long long* slots,
                   void* pool, long long tokens, int heads, int dim_p, int rot, int rot_p, int kv_col, int rank,
                   int rank_p, float eps, void* stream) {
  using namespace rb;
  if (tokens <= 0) return 0;
  if ((rot & 1) || rot > rot_p || (rot_p & 1) || rank > rank_p) return 21;
  RB_BY_DTYPE((latent_post_kernel<T><<<(unsigned)tokens, 128, 0, (cudaStream_t)stream>>>(
      (T*)proj, ldp, (const float2*)tab, norm_w, slots, (T*)pool, heads, dim_p, rot, rot_p, kv_col, rank, rank_p, eps)))
  RB_LAUNCH_STATUS();
}

// row_bytes must be a multiple of 16; tables [n_seg, max_blocks]; seg_off [n_seg + 1] on the device
int rb_latent_gather(const void* pool, const int* tables, const int* seg_off, void* out, int n_seg, int max_blocks,
                     int block_size, int row_bytes, long long total, void* stream) {
  using namespace rb;
  if (total <= 0) return 0;
  if (row_bytes % 16) return 21;
  latent_gather_kernel<<<grid_for(total * (row_bytes / 16), 256), 256, 0, (cudaStream_t)stream>>>(
      (const uint4*)pool, tables, seg_off, (uint4*)out, n_seg, max_blocks, block_size, row_bytes / 16, total);
  RB_LAUNCH_STATUS();
}

// scratch: part_o rows*heads*splits*rank_p floats, part_ml rows*heads*splits*2 floats; sink may be null
int rb_latent_rows_attn(int dtype, const void* qa, const void* qr, long long ldq, int hq, const void* pool,
                        const int* tables, const int* ctx, const float* sink, void* out, float* part_o,
                        float* part_ml, int rows, int heads, int rank_p, int rot_p, int block_size, int max_blocks,
                        int splits, float scale, void* stream) {
  using namespace rb;
  if (rows <= 0) return 0;
  if (rows > 65535 || splits > 65535) return 22;
  cudaStream_t st = (cudaStream_t)stream;
  int rc = 0;
  RB_BY_DTYPE((rc = launch_latent_rows<T>((const T*)qa, (const T*)qr, ldq, hq, (const T*)pool, tables, ctx, part_o, part_ml,
                                          rows, heads, rank_p, rot_p, block_size, max_blocks, splits, scale, st)))
  if (rc) return rc;
  RB_BY_DTYPE((launch_attn_merge<T>(part_o, part_ml, sink, nullptr, 0, ATTN_GATE_NONE, (T*)out, (long long)heads * rank_p, rows, heads, rank_p, splits, st)))
  RB_LAUNCH_STATUS();
}

// The merge alone, for partial results another kernel wrote.
int rb_latent_merge(int dtype, const float* part_o, const float* part_ml, const float* sink, void* out, int rows,
                    int heads, int rank_p, int splits, void* stream) {
  using namespace rb;
  if (rows <= 0) return 0;
  RB_BY_DTYPE((launch_attn_merge<T>(part_o, part_ml, sink, nullptr, 0, ATTN_GATE_NONE, (T*)out, (long long)heads * rank_p, rows, heads, rank_p, splits, (cudaStream_t)stream)))
  RB_LAUNCH_STATUS();
}

int rb_sigmoid_gate(int dtype, void* x, long long ldx, const void* g, long long ldg, long long rows, int n, void* stream) {
  using namespace rb;
  if (rows <= 0 || n <= 0) return 0;
  RB_BY_DTYPE((sigmoid_gate_kernel<T><<<grid_for(rows * n, 256), 256, 0, (cudaStream_t)stream>>>((T*)x, ldx, (const T*)g, ldg, rows, n)))
  RB_LAUNCH_STATUS();
}
}
