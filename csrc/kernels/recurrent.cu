// Recurrent mixers whose state is a matrix per head, token by token, sm_100a: the matrix memory with exponential gates
// (mLSTM) and the gated delta rule with a decay per key channel or per head.  Decoded tokens, short portions, and everything in
// 32-bit runs; long prompts are in mlstm_chunk.cu and delta_chunk.cu.
//
// A CTA takes one head of one sequence at a time.  The state (fp32, [dim, vdim]) comes into registers once, all tokens of
// the portion pass over it, and it goes back: 16 warps share the rows, the lanes of a warp the columns.  With more heads
// than CTAs fit, a CTA goes on to another head whose state has been on its way to shared memory meanwhile (STAGED).  A portion that
// starts at position 0 starts from zeros whatever its place holds.  The output norm over a head, its weight and its gate
// are the last step of a token, so the mixer leaves what the output product takes.
//
// A sequence's portion: {first row, tokens, place of its state, position of the first token}; no tokens: nothing to do.
#include "recurrent.cuh"

namespace rb {

constexpr int kRecThreads = 512, kRecWarps = 16, kRecMaxDim = 512;

template <int VEC>
__device__ __forceinline__ void rec_load(const float* p, float (&v)[VEC]) {
  if constexpr (VEC == 4) *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(p);
  else if constexpr (VEC == 2) *reinterpret_cast<float2*>(v) = *reinterpret_cast<const float2*>(p);
  else v[0] = *p;
}
template <int VEC>
__device__ __forceinline__ void rec_store(float* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = *reinterpret_cast<const float4*>(v);
  else if constexpr (VEC == 2) *reinterpret_cast<float2*>(p) = *reinterpret_cast<const float2*>(v);
  else *p = v[0];
}

// Weight and gate of thread c's number, asked for before the token's arithmetic; used when the head has one block of columns.
template <typename T>
__device__ __forceinline__ float rec_factor(const RecOut<T>& p, long long row, int h, int vdim_p, bool whole) {
  const int c = threadIdx.x;
  if (!whole || c >= vdim_p) return 0.f;
  return p.norm[h * p.norm_step + c] * rec_gate<T>(to_f32<T>(p.gate[row * p.ldg + (long long)h * vdim_p + c]), p.silu);
}
// All threads; o: the head's result of thread c < COLS (0 for others) when the head has one block of columns, else
// columns chunk * COLS + c of `tmp` take it.
template <typename T, int COLS>
__device__ __forceinline__ void rec_finish(const RecOut<T>& p, long long row, int h, int heads, int chunk, bool whole, int vdim, int vdim_p,
                                           float o, float factor, float* s_red) {
  const int c = threadIdx.x;
  if (!whole) {
    if (c < COLS && chunk * COLS + c < vdim_p) p.tmp[row * heads * vdim_p + (long long)h * vdim_p + chunk * COLS + c] = o;
    return;
  }
  if (c < COLS) {
    const float s = warp_sum(o * o);
    if ((c & 31) == 0) s_red[c >> 5] = s;
  }
  __syncthreads();
  if (c >= vdim_p) return;
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < COLS / 32; ++i) s += s_red[i];
  p.out[row * p.ldo + (long long)h * vdim_p + c] = from_f32<T>(o * factor / sqrtf(s / vdim + p.eps));
}
// All threads, after all blocks of columns: norm and gate of the rows in `tmp`.
template <typename T>
__device__ __forceinline__ void rec_finish_rows(const RecOut<T>& p, int row0, int n, int h, int heads, int vdim, int vdim_p) {
  __syncthreads();
  for (int t = threadIdx.x >> 5; t < n; t += kRecWarps) {
    const long long row = row0 + t;
    const float* o = p.tmp + row * heads * vdim_p + (long long)h * vdim_p;
    float s = 0.f;
    for (int c = threadIdx.x & 31; c < vdim_p; c += 32) s += o[c] * o[c];
    const float r = 1.0f / sqrtf(warp_sum(s) / vdim + p.eps);
    for (int c = threadIdx.x & 31; c < vdim_p; c += 32) rec_write(p, row, h, c, vdim_p, o[c], r);
  }
}

// ---------------------------------------------------------------------------------------------------------
// S <- exp(f + m - m') S + exp(i - m') k v^T, n the same with k alone, m' = max(f + m, i);
// o = S^T q / (max(|n . q|, exp(-m')) + 1e-6)
// ---------------------------------------------------------------------------------------------------------
// The heads a CTA takes: numbers blockIdx.x, + gridDim.x, ... of (sequence, head), sequences without tokens left out.
struct RecItems {
  const int4* seqs;
  int heads, total;
  __device__ __forceinline__ int next(int i) const {
    while (i < total && seqs[i / heads].y <= 0) i += gridDim.x;
    return i;
  }
};
// One thread: the state of an item into shared memory (nothing for a sequence that starts).
__device__ __forceinline__ void rec_request(const RecItems& it, int i, const float* S, int size, float* stage, uint64_t* full) {
  if (i >= it.total) return;
  const int4 seq = it.seqs[i / it.heads];
  if (seq.w == 0) {
    mbar_arrive(smem_u32(full));
    return;
  }
  mbar_arrive_expect_tx(smem_u32(full), size * 4);
  bulk_load_1d(smem_u32(stage), S + ((long long)seq.z * it.heads + i % it.heads) * size, size * 4, smem_u32(full));
}

template <typename T>
struct MlstmRowsParams {
  const T* proj;                 // row: heads x dim_p queries, keys, heads x vdim_p values
  long long ldp;
  const float* gates;            // row: heads input gates, heads forget gates, before the cap
  long long ldz;
  const int4* seqs;
  float *S, *n, *m;              // [places, heads, dim_p, vdim_p], [places, heads, dim_p], [places, heads]
  int heads, dim_p, vdim_p, vdim;
  float q_scale, cap;
  RecOut<T> o;
};

template <typename T, int RPW, int VEC, bool STAGED>
__global__ void __launch_bounds__(kRecThreads, RPW * VEC <= 32 ? 2 : 1) mlstm_rows_kernel(const MlstmRowsParams<T> p, int n_seqs, int* status) {
  constexpr int COLS = 32 * VEC;
  extern __shared__ __align__(128) float s_stage[];
  __shared__ uint64_t full;
  __shared__ int s_abort;
  __shared__ float s_k[kRecMaxDim], s_q[kRecMaxDim], s_nq[kRecWarps], s_red[4];
  __shared__ __align__(16) float s_o[kRecWarps][COLS], s_v[COLS];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r0 = warp * RPW;
  const int chunks = (p.vdim_p + COLS - 1) / COLS;
  const RecItems items{p.seqs, p.heads, p.heads * n_seqs};
  int item = items.next(blockIdx.x), phase = 0;
  if (STAGED && threadIdx.x == 0) {
    mbar_init(smem_u32(&full), 1);
    s_abort = 0;
    fence_barrier_init();
    rec_request(items, item, p.S, p.dim_p * p.vdim_p, s_stage, &full);
  }
  if (STAGED) __syncthreads();
  for (; item < items.total; item = items.next(item + gridDim.x)) {
    const int4 seq = p.seqs[item / p.heads];
    const int h = item % p.heads;
    const long long sh = (long long)seq.z * p.heads + h;
    const bool fresh = seq.w == 0, mine = lane < RPW && r0 + lane < p.dim_p;
    for (int chunk = 0; chunk < chunks; ++chunk) {
      const int col = chunk * COLS + lane * VEC;
      const bool live = col < p.vdim_p;
      float S[RPW][VEC];
      float* state = p.S + (sh * p.dim_p + r0) * p.vdim_p + col;
      auto load_state = [&](const float* from) {
#pragma unroll
        for (int i = 0; i < RPW; ++i) {
          if (!fresh && live && r0 + i < p.dim_p) {
            rec_load<VEC>(from + (long long)i * p.vdim_p, S[i]);
          } else {
#pragma unroll
            for (int e = 0; e < VEC; ++e) S[i][e] = 0.f;
          }
        }
      };
      if (!STAGED) load_state(state);
      float n = !fresh && mine ? p.n[sh * p.dim_p + r0 + lane] : 0.f;
      float m = fresh ? 0.f : p.m[sh];
      for (int t = 0; t < seq.y; ++t) {
        const long long row = seq.x + t;
        const T* pr = p.proj + row * p.ldp;
        for (int d = threadIdx.x; d < p.dim_p; d += kRecThreads) {
          s_q[d] = to_f32<T>(pr[h * p.dim_p + d]) * p.q_scale;
          s_k[d] = to_f32<T>(pr[(p.heads + h) * p.dim_p + d]);
        }
        if (threadIdx.x < COLS) {
          const int c = chunk * COLS + threadIdx.x;
          s_v[threadIdx.x] = c < p.vdim_p ? to_f32<T>(pr[2LL * p.heads * p.dim_p + (long long)h * p.vdim_p + c]) : 0.f;
        }
        const float factor = rec_factor(p.o, row, h, p.vdim_p, chunks == 1);
        const float2 g = mlstm_gates(p.gates[row * p.ldz + h], p.gates[row * p.ldz + p.heads + h], p.cap);
        const float m_new = fmaxf(g.y + m, g.x), keep = expf(g.y + m - m_new), put = expf(g.x - m_new);
        m = m_new;
        if (STAGED && t == 0) {                  // the token's vectors were asked for before the wait
          const bool ok = mbar_wait(smem_u32(&full), phase, &s_abort, status, RB_ERR_TIMEOUT_FULL);
          if (!__syncthreads_and(ok)) return;
          phase ^= 1;
          load_state(s_stage + r0 * p.vdim_p + col);
        }
        __syncthreads();
        if (STAGED && t == 0 && threadIdx.x == 0)          // the stage has been read: the next head's state may come
          rec_request(items, items.next(item + gridDim.x), p.S, p.dim_p * p.vdim_p, s_stage, &full);
        float o[VEC], v[VEC];
        rec_load<VEC>(&s_v[lane * VEC], v);
#pragma unroll
        for (int e = 0; e < VEC; ++e) o[e] = 0.f;
#pragma unroll
        for (int i = 0; i < RPW; ++i)
          if (r0 + i < p.dim_p) {
            const float k = put * s_k[r0 + i], q = s_q[r0 + i];
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
              S[i][e] = fmaf(keep, S[i][e], k * v[e]);
              o[e] = fmaf(S[i][e], q, o[e]);
            }
          }
        float nq = 0.f;
        if (mine) {
          n = fmaf(keep, n, put * s_k[r0 + lane]);
          nq = n * s_q[r0 + lane];
        }
        nq = warp_sum(nq);
        if (lane == 0) s_nq[warp] = nq;
        rec_store<VEC>(&s_o[warp][lane * VEC], o);
        __syncthreads();
        float sum = 0.f;
        if (threadIdx.x < COLS) {
          nq = 0.f;
#pragma unroll
          for (int w = 0; w < kRecWarps; ++w) {
            nq += s_nq[w];
            sum += s_o[w][threadIdx.x];
          }
          sum /= fmaxf(fabsf(nq), expf(-m)) + 1e-6f;
        }
        rec_finish<T, COLS>(p.o, row, h, p.heads, chunk, chunks == 1, p.vdim, p.vdim_p, sum, factor, s_red);
      }
      if (live) {
#pragma unroll
        for (int i = 0; i < RPW; ++i)
          if (r0 + i < p.dim_p) rec_store<VEC>(state + (long long)i * p.vdim_p, S[i]);
      }
      if (chunk == chunks - 1) {              // every block of columns starts from the old ones
        if (mine) p.n[sh * p.dim_p + r0 + lane] = n;
        __syncthreads();
        if (threadIdx.x == 0) p.m[sh] = m;
      }
    }
    if (chunks > 1) rec_finish_rows<T>(p.o, seq.x, seq.y, h, p.heads, p.vdim, p.vdim_p);
  }
}

// ---------------------------------------------------------------------------------------------------------
// Short causal convolutions over time with silu (queries, keys, values), unit queries and keys, decays
// g = exp(-exp(A) softplus(a + dt)), write strengths beta = sigmoid(b); then S <- diag(g) S, u = beta (v - S^T k),
// S <- S + k u^T, o = S^T q.  With the old S: S^T k = S_old^T (g k) and o = S_old^T (g q) + (k . q) u, so one pass over the
// state and one exchange between the warps do for a token.
// ---------------------------------------------------------------------------------------------------------
template <typename T>
struct DeltaRowsParams {
  const T* raw;                  // row: kv_heads x dim_p queries, keys, heads x vdim_p values, before their convolutions
  long long ldr;
  const float* taps_w;           // [taps][channels], the last one is the current token's
  T* conv;                       // [places, heads, taps - 1, 2 dim_p + vdim_p] inputs before the portion
  const float *a, *dt, *decay;   // steps [tokens, heads * dim_p] and [heads * dim_p], or [tokens, heads] and [heads] (per_head); [heads]: exp(A)
  long long lda;
  int per_head;
  const float* b;                // [tokens, ldb]
  long long ldb;
  const int4* seqs;
  float* S;                      // [places, heads, dim_p, vdim_p]
  int heads, kv_heads, dim_p, vdim_p, vdim, taps;
  float q_scale;
  RecOut<T> o;
};

template <typename T, int RPW, int VEC, bool STAGED>
__global__ void __launch_bounds__(kRecThreads, RPW * VEC <= 32 ? 2 : 1) delta_rows_kernel(const DeltaRowsParams<T> p, int n_seqs, int* status) {
  constexpr int COLS = 32 * VEC;
  extern __shared__ __align__(128) float s_stage[];
  __shared__ uint64_t full;
  __shared__ int s_abort;
  __shared__ float4 s_x[kRecMaxDim];           // {decay, key, query} of every key channel
  __shared__ __align__(16) float s_v[COLS], s_r[kRecWarps][COLS], s_p[kRecWarps][COLS];
  __shared__ float s_red[4];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r0 = warp * RPW;
  const int chunks = (p.vdim_p + COLS - 1) / COLS, past = p.taps - 1, own = 2 * p.dim_p + p.vdim_p;
  const int channels = 2 * p.kv_heads * p.dim_p + p.heads * p.vdim_p;
  const RecItems items{p.seqs, p.heads, p.heads * n_seqs};
  int item = items.next(blockIdx.x), phase = 0;
  if (STAGED && threadIdx.x == 0) {
    mbar_init(smem_u32(&full), 1);
    s_abort = 0;
    fence_barrier_init();
    rec_request(items, item, p.S, p.dim_p * p.vdim_p, s_stage, &full);
  }
  if (STAGED) __syncthreads();
  for (; item < items.total; item = items.next(item + gridDim.x)) {
    const int4 seq = p.seqs[item / p.heads];
    const int h = item % p.heads;
    const long long sh = (long long)seq.z * p.heads + h;
    const bool fresh = seq.w == 0;
    T* conv = p.conv + sh * past * own;
    // channel c of the head at token t of the portion; with the last token it leaves the inputs that the next portion needs
    // (a channel is one thread's throughout)
    auto convolved = [&](int c, int t) {
      const int ch = delta_channel(c, h, p.heads, p.kv_heads, p.dim_p, p.vdim_p);
      const T* raw = p.raw + (long long)(seq.x + t) * p.ldr + ch;
      const bool keep = chunks == 1 && t == seq.y - 1;
      float s = 0.f;
      for (int j0 = 0; j0 < p.taps; j0 += 4) {   // four inputs at a time: all loads before the stores
        T x[4];
        float w[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int j = j0 + i, back = past - j;               // tokens ago
          x[i] = from_f32<T>(0.f);
          w[i] = 0.f;
          if (j >= p.taps) continue;
          if (back <= t) x[i] = raw[-back * p.ldr];
          else if (!fresh) x[i] = conv[(long long)(j + t) * own + c];
          w[i] = p.taps_w[(long long)j * channels + ch];
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          s = fmaf(w[i], to_f32<T>(x[i]), s);
          if (keep && j0 + i > 0 && j0 + i < p.taps) conv[(long long)(j0 + i - 1) * own + c] = x[i];
        }
      }
      return s * rec_sigmoid<T>(s);
    };
    for (int chunk = 0; chunk < chunks; ++chunk) {
      const int col = chunk * COLS + lane * VEC;
      const bool live = col < p.vdim_p;
      float S[RPW][VEC];
      float* state = p.S + (sh * p.dim_p + r0) * p.vdim_p + col;
      auto load_state = [&](const float* from) {
#pragma unroll
        for (int i = 0; i < RPW; ++i) {
          if (!fresh && live && r0 + i < p.dim_p) {
            rec_load<VEC>(from + (long long)i * p.vdim_p, S[i]);
          } else {
#pragma unroll
            for (int e = 0; e < VEC; ++e) S[i][e] = 0.f;
          }
        }
      };
      if (!STAGED) load_state(state);
      for (int t = 0; t < seq.y; ++t) {
        const long long row = seq.x + t;
        for (int c = threadIdx.x; c < 3 * p.dim_p + COLS; c += kRecThreads) {
          if (c < 2 * p.dim_p) {
            float x = convolved(c, t);
            if (p.per_head) x = to_f32<T>(from_f32<T>(x));       // as prompts have them (delta_chunk.cu)
            if (c < p.dim_p) s_x[c].z = x;
            else s_x[c - p.dim_p].y = x;
          } else if (c < 3 * p.dim_p) {
            const int d = p.per_head ? h : h * p.dim_p + c - 2 * p.dim_p;
            s_x[c - 2 * p.dim_p].x = expf(-p.decay[h] * softplus_f(p.a[row * p.lda + d] + p.dt[d]));
          } else {
            const int v = c - 3 * p.dim_p;
            s_v[v] = chunk * COLS + v < p.vdim_p ? to_f32<T>(from_f32<T>(convolved(2 * p.dim_p + chunk * COLS + v, t))) : 0.f;
          }
        }
        const float beta = 1.0f / (1.0f + expf(-p.b[row * p.ldb + h])), factor = rec_factor(p.o, row, h, p.vdim_p, chunks == 1);
        if (STAGED && t == 0) {                  // the token's vectors were asked for before the wait
          const bool ok = mbar_wait(smem_u32(&full), phase, &s_abort, status, RB_ERR_TIMEOUT_FULL);
          if (!__syncthreads_and(ok)) return;
          phase ^= 1;
          load_state(s_stage + r0 * p.vdim_p + col);
        }
        __syncthreads();
        if (STAGED && t == 0 && threadIdx.x == 0)          // the stage has been read: the next head's state may come
          rec_request(items, items.next(item + gridDim.x), p.S, p.dim_p * p.vdim_p, s_stage, &full);
        float r[VEC], po[VEC], qq = 0.f, kk = 0.f, kq = 0.f;
#pragma unroll
        for (int e = 0; e < VEC; ++e) r[e] = po[e] = 0.f;
#pragma unroll
        for (int i = 0; i < RPW; ++i)
          if (r0 + i < p.dim_p) {
            const float4 x = s_x[r0 + i];
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
              S[i][e] *= x.x;
              r[e] = fmaf(S[i][e], x.y, r[e]);
              po[e] = fmaf(S[i][e], x.z, po[e]);
            }
          }
        rec_store<VEC>(&s_r[warp][lane * VEC], r);
        rec_store<VEC>(&s_p[warp][lane * VEC], po);
        for (int d = lane; d < p.dim_p; d += 32) {
          const float4 x = s_x[d];
          kk = fmaf(x.y, x.y, kk);
          qq = fmaf(x.z, x.z, qq);
          kq = fmaf(x.y, x.z, kq);
        }
        const float rk = 1.0f / sqrtf(warp_sum(kk) + 1e-6f), rq = p.q_scale / sqrtf(warp_sum(qq) + 1e-6f);
        kq = warp_sum(kq) * rk * rq;
        __syncthreads();
        float o = 0.f;
        if (threadIdx.x < COLS) {
          float rs = 0.f;
#pragma unroll
          for (int w = 0; w < kRecWarps; ++w) {
            rs += s_r[w][threadIdx.x];
            o += s_p[w][threadIdx.x];
          }
          const float u = beta * (s_v[threadIdx.x] - rs * rk);
          o = fmaf(kq, u, o * rq);
          s_v[threadIdx.x] = u * rk;
        }
        rec_finish<T, COLS>(p.o, row, h, p.heads, chunk, chunks == 1, p.vdim, p.vdim_p, o, factor, s_red);
        if (chunks > 1) __syncthreads();
        float u[VEC];
        rec_load<VEC>(&s_v[lane * VEC], u);
#pragma unroll
        for (int i = 0; i < RPW; ++i)
          if (r0 + i < p.dim_p) {
            const float k = s_x[r0 + i].y;
#pragma unroll
            for (int e = 0; e < VEC; ++e) S[i][e] = fmaf(k, u[e], S[i][e]);
          }
        if (t + 1 < seq.y || chunk + 1 < chunks) __syncthreads();      // the vectors of this token have been read
      }
      if (live) {
#pragma unroll
        for (int i = 0; i < RPW; ++i)
          if (r0 + i < p.dim_p) rec_store<VEC>(state + (long long)i * p.vdim_p, S[i]);
      }
    }
    __syncthreads();
    if (chunks > 1) {
      delta_keep_inputs<T>(p.raw, p.ldr, p.conv, seq, h, p.heads, p.kv_heads, p.dim_p, p.vdim_p, p.taps, threadIdx.x, kRecThreads);
      rec_finish_rows<T>(p.o, seq.x, seq.y, h, p.heads, p.vdim, p.vdim_p);
    }
  }
}

// ---------------------------------------------------------------------------------------------------------
// A product with few outputs per token, kept in fp32 (gates of a recurrence): out[t][n] = h[t] . w[n] + bias[n].  One CTA
// per token and 16 outputs, a warp per output.
// ---------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(512)
    few_outputs_kernel(const T* __restrict__ h, long long ldh, const T* __restrict__ w, const float* __restrict__ bias,
                       float* __restrict__ out, int K, int N) {
  constexpr int V = 16 / sizeof(T);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* x = h + (long long)blockIdx.x * ldh;
  const int n = blockIdx.y * 16 + warp;
  if (n < N) {
    float s = 0.f;
#pragma unroll 4
    for (int c = lane * V; c < K; c += 32 * V) {
      const uint4 a = *reinterpret_cast<const uint4*>(x + c), b = *reinterpret_cast<const uint4*>(w + (long long)n * K + c);
#pragma unroll
      for (int j = 0; j < V; ++j) s = fmaf(to_f32<T>(reinterpret_cast<const T*>(&a)[j]), to_f32<T>(reinterpret_cast<const T*>(&b)[j]), s);
    }
    s = warp_sum(s);
    if (lane == 0) out[(long long)blockIdx.x * N + n] = s + (bias ? bias[n] : 0.f);
  }
}

// calls go(rows per warp, numbers per lane) with the smallest that fit
template <typename F>
int rec_by_size(int dim_p, int vdim_p, F go) {
#define RB_REC(RPW)                                                       \
  if (dim_p <= kRecWarps * RPW) {                                         \
    if (vdim_p > 64 && RPW <= 16) return go.template operator()<RPW, (RPW <= 16 ? 4 : 2)>(); \
    if (vdim_p > 32) return go.template operator()<RPW, 2>();             \
    return go.template operator()<RPW, 1>();                              \
  }
  RB_REC(2)
  RB_REC(4)
  RB_REC(8)
  RB_REC(16)
  RB_REC(32)
#undef RB_REC
  return 22;
}

// One CTA per head, or CTAs that stay (two per SM) when there are several heads for each and a state fits shared memory.
template <typename P, typename K>
int rec_launch(const P& p, int n_seqs, int cols, K plain, K staged, cudaStream_t st) {
  const long long total = (long long)p.heads * n_seqs;
  const int bytes = p.dim_p * p.vdim_p * 4, resident = 2 * rbh::sm_count();
  int* status = rbh::device_status_word();
  if (total > resident && bytes <= 64 * 1024 && p.vdim_p <= cols) {
    const cudaError_t e = cudaFuncSetAttribute(staged, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) return 2000 + (int)e;
    staged<<<resident, kRecThreads, bytes, st>>>(p, n_seqs, status);
  } else {
    plain<<<(unsigned)total, kRecThreads, 0, st>>>(p, n_seqs, status);
  }
  return 0;
}
template <typename T>
struct MlstmRowsLaunch {
  MlstmRowsParams<T> p;
  int n_seqs;
  cudaStream_t st;
  template <int RPW, int VEC>
  int operator()() {
    return rec_launch(p, n_seqs, 32 * VEC, mlstm_rows_kernel<T, RPW, VEC, false>, mlstm_rows_kernel<T, RPW, VEC, true>, st);
  }
};
template <typename T>
struct DeltaRowsLaunch {
  DeltaRowsParams<T> p;
  int n_seqs;
  cudaStream_t st;
  template <int RPW, int VEC>
  int operator()() {
    return rec_launch(p, n_seqs, 32 * VEC, delta_rows_kernel<T, RPW, VEC, false>, delta_rows_kernel<T, RPW, VEC, true>, st);
  }
};

}  // namespace rb

#define RB_BY_DTYPE(...)                                               \
  if (dtype == rbh::DT_BF16) { using T = __nv_bfloat16; __VA_ARGS__; } \
  else if (dtype == rbh::DT_F32) { using T = float; __VA_ARGS__; }     \
  else return 20;
#define RB_LAUNCH_STATUS()             \
  cudaError_t e_ = cudaGetLastError(); \
  return e_ == cudaSuccess ? 0 : 3000 + (int)e_

extern "C" {

// Whether a head has more columns than one pass takes (the caller then passes `tmp`).
int rb_recurrent_blocks(int dim_p, int vdim_p) {
  const int cols = dim_p <= 256 && vdim_p > 64 ? 128 : vdim_p > 32 ? 64 : 32;
  return (vdim_p + cols - 1) / cols;
}

// Sizes ending in _p are multiples of eight; dim_p at most 512.  Scales, layouts: see MlstmRowsParams and RecOut.
int rb_mlstm_rows(int dtype, const void* proj, long long ldp, const float* gates, long long ldz, const int* seqs, int n_seqs, float* S,
                  float* n, float* m, const void* gate, long long ldg, const float* norm, void* out, long long ldo, float* tmp, int heads,
                  int dim_p, int vdim_p, int vdim, float q_scale, float cap, float eps, void* stream) {
  using namespace rb;
  if (n_seqs <= 0) return 0;
  if (n_seqs > 65535 || dim_p % 8 || vdim_p % 8 || dim_p > kRecMaxDim || (!tmp && rb_recurrent_blocks(dim_p, vdim_p) > 1)) return 22;
  RB_BY_DTYPE({
    MlstmRowsLaunch<T> go{{(const T*)proj, ldp, gates, ldz, (const int4*)seqs, S, n, m, heads, dim_p, vdim_p, vdim, q_scale, cap,
                           {(T*)out, ldo, (const T*)gate, ldg, norm, vdim_p, tmp, eps, 0}}, n_seqs, (cudaStream_t)stream};
    const int rc = rec_by_size(dim_p, vdim_p, go);
    if (rc) return rc;
  })
  RB_LAUNCH_STATUS();
}

// norm [vdim_p], shared by the heads.  See DeltaRowsParams.
int rb_delta_rows(int dtype, const void* raw, long long ldr, const float* taps_w, void* conv, const float* a, long long lda, int per_head,
                  const float* dt, const float* decay, const float* b, long long ldb, const int* seqs, int n_seqs, float* S, const void* gate, long long ldg,
                  const float* norm, void* out, long long ldo, float* tmp, int heads, int kv_heads, int dim_p, int vdim_p, int vdim, int taps,
                  float q_scale, float eps, int silu, void* stream) {
  using namespace rb;
  if (n_seqs <= 0) return 0;
  if (n_seqs > 65535 || heads % kv_heads || dim_p % 8 || vdim_p % 8 || dim_p > kRecMaxDim || taps < 1 ||
      (!tmp && rb_recurrent_blocks(dim_p, vdim_p) > 1))
    return 22;
  RB_BY_DTYPE({
    DeltaRowsLaunch<T> go{{(const T*)raw, ldr, taps_w, (T*)conv, a, dt, decay, lda, per_head, b, ldb, (const int4*)seqs, S, heads, kv_heads, dim_p, vdim_p,
                           vdim, taps, q_scale, {(T*)out, ldo, (const T*)gate, ldg, norm, 0, tmp, eps, silu}}, n_seqs, (cudaStream_t)stream};
    const int rc = rec_by_size(dim_p, vdim_p, go);
    if (rc) return rc;
  })
  RB_LAUNCH_STATUS();
}

// w [N, K] (rows 16-byte aligned), out [tokens, N] fp32, bias fp32 or null
int rb_few_outputs(int dtype, const void* h, long long ldh, const void* w, const float* bias, float* out, long long tokens, int K, int N,
                   void* stream) {
  using namespace rb;
  if (tokens <= 0) return 0;
  if (K % 8 || ldh % 8 || ((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(w)) & 15)) return 21;
  RB_BY_DTYPE((few_outputs_kernel<T><<<dim3((unsigned)tokens, (N + 15) / 16), 512, 0, (cudaStream_t)stream>>>((const T*)h, ldh, (const T*)w, bias, out, K, N)))
  RB_LAUNCH_STATUS();
}
}
