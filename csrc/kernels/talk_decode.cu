// Attention of single query rows whose heads talk, sm_100a, 16-bit: all heads of a row attend in one CTA, so that every page
// crosses HBM once although every head's softmax needs all heads' scores.
//
// As in window_decode.cu the kernel is bound by the pages' bytes, and a row has too few queries for a tile of tcgen05, so
// products are warp-level ones with fragments that go from one to the next in registers.  Heads stand in slots of eight,
// those of a key/value head together.  A CTA takes a slice of one row's tiles of 64 keys:
//
//   warp 4      brings keys, then values of a tile, one key/value head after the other, through a ring (TMA)
//   warps 0-3   scores: warp w has keys 16 w .. 16 w + 15 of every head.  Products are keys x heads, whose accumulators, split
//               into high and low 16-bit parts, are the left operand of the product with the mixing matrix (three products,
//               about 16 bits).  Mixed scores go to shared memory.
//               values: warp w has slots w, w + 4 and all 64 keys: softmax, then (numbers x keys) x (keys x heads)
//
// One barrier a tile separates the two (scores alternate between two buffers); slices meet in attn_merge.
#include "attn_merge.cuh"
#include "warp_mma.cuh"

namespace rb {

constexpr int kTdKeys = 64, kTdLd = 72, kTdUnits = 16;

struct TalkDecodeParams {
  const __nv_bfloat16* q;        // row b, head h at q[b * ldq + h * dim]
  long long ldq;
  const int *tables, *ctx;       // [rows, max_blocks], [rows]: keys up to and with the row's own
  const float *mix, *sink;       // [heads, heads]; [heads] or null
  const __nv_bfloat16* gate;
  long long ldg, ldo;
  __nv_bfloat16* out;
  float *part_o, *part_ml;       // used when splits > 1
  int heads, kv_heads, dim, vdim, window, block_size, box_rows, max_blocks, splits, gate_kind;
  int per_kv, n_slots, units;    // slots per key/value head, slots, units of the ring
  float scale_log2;
  int* status;
};

template <int KS, int NS>        // 64-column sub-tiles of a head; slots, rounded up
struct TalkDecodeCfg {
  static constexpr int SUB = kTdKeys * 128, UNIT = KS * SUB;
  static constexpr int Q_LD = (KS * 64 + 8) * 2, Q_BYTES = NS * 8 * Q_LD;
  static constexpr int M_BYTES = NS / 2 * NS * 512, S_FLOATS = NS * 8 * kTdLd;
  static constexpr int FIXED = Q_BYTES + M_BYTES + 2 * S_FLOATS * 4 + 1024;
};

template <int KS, int NS>
__global__ void __launch_bounds__(160, 1)
    talk_decode_kernel(const __grid_constant__ CUtensorMap tk, const __grid_constant__ CUtensorMap tv, const TalkDecodeParams p) {
  using C = TalkDecodeCfg<KS, NS>;
  using T = __nv_bfloat16;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                             ~static_cast<uintptr_t>(1023));
  uint8_t* s_m = smem + p.units * C::UNIT;
  float* s_s = reinterpret_cast<float*>(s_m + C::M_BYTES);       // [2][head][kTdLd]
  uint8_t* s_q = reinterpret_cast<uint8_t*>(s_s + 2 * C::S_FLOATS);
  __shared__ uint64_t full[kTdUnits], empty[kTdUnits];
  __shared__ int s_abort;
  volatile int* abort_flag = &s_abort;
  const int warp = uniform_warp_idx(), lane = threadIdx.x & 31;
  const int b = blockIdx.x, sp = blockIdx.y, rep = p.heads / p.kv_heads;
  const int ctx = p.ctx[b], lo = max(0, ctx - p.window), first = lo / kTdKeys;
  // slices are whole tiles; a tile at either end of the window is masked
  const int all = (ctx + kTdKeys - 1) / kTdKeys - first, per = (all + p.splits - 1) / p.splits;
  const int tile0 = first + sp * per, n_tiles = min(per, all - sp * per);
  if (n_tiles <= 0) {                          // nothing of this row falls into the slice (splits > 1)
    for (int h = threadIdx.x; h < p.heads; h += 160) {
      float* ml = p.part_ml + (((long long)b * p.heads + h) * p.splits + sp) * 2;
      ml[0] = -INFINITY;
      ml[1] = 0.f;
    }
    return;
  }
  // head of place i of slot s; -1: none
  auto head_of = [&](int s, int i) {
    const int c = s / p.per_kv, x = (s - c * p.per_kv) * 8 + i;
    return s < p.n_slots && x < rep ? c * rep + x : -1;
  };
  if (threadIdx.x == 0) {
    for (int u = 0; u < p.units; ++u) {
      mbar_init(smem_u32(&full[u]), 1);
      mbar_init(smem_u32(&empty[u]), 4);
    }
    s_abort = 0;
    fence_barrier_init();
  } else if (threadIdx.x == 32) {
    prefetch_tensormap(&tk);
    prefetch_tensormap(&tv);
  }
  __syncthreads();

  if (warp == 4) {
    const int* table = p.tables + (long long)b * p.max_blocks;
    const int boxes = kTdKeys / p.box_rows;    // at most 8
    // row of the pools (key/value head 0) where box `lane` of tile i starts.  Boxes past the context are read from its last one.
    auto lookup = [&](int i) -> int {
      const int t = min((tile0 + i) * kTdKeys + min(lane, boxes - 1) * p.box_rows, (ctx - 1) / p.box_rows * p.box_rows);
      return table[min(t / p.block_size, p.max_blocks - 1)] * p.kv_heads * p.block_size + t % p.block_size;
    };
    int unit = 0, phase = 1, rows = lookup(0);
    bool ok = true;
    for (int i = 0; i < n_tiles && ok; ++i) {
      const int next = i + 1 < n_tiles ? lookup(i + 1) : 0;
      for (int x = 0; x < 2 * p.kv_heads; ++x) {
        ok = mbar_wait(smem_u32(&empty[unit]), phase, abort_flag, p.status, RB_ERR_TIMEOUT_EMPTY);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        const bool keys = x < p.kv_heads;
        const int c = keys ? x : x - p.kv_heads;
        const uint32_t bar = smem_u32(&full[unit]), dst = smem_u32(smem + unit * C::UNIT);
        if (lane == 0) mbar_arrive_expect_tx(bar, C::UNIT);
        for (int y = 0; y < boxes; ++y) {
          const int row = __shfl_sync(0xffffffffu, rows, y) + c * p.block_size;
          if (lane == 0) {
#pragma unroll
            for (int s = 0; s < KS; ++s) tma_load_2d(dst + s * C::SUB + y * p.box_rows * 128, keys ? &tk : &tv, bar, s * 64, row);
          }
        }
        if (++unit == p.units) {
          unit = 0;
          phase ^= 1;
        }
      }
      rows = next;
    }
    if (!ok)                                   // copies in flight land before the shared memory gets another use
      for (int i = 0; i < 64; ++i) __nanosleep(10000);
    return;
  }

  // fragments: this lane has row r (and r + 8) and columns 2 c, 2 c + 1 of an accumulator
  const int r = lane >> 2, c = lane & 3;
  // queries by slot; the mixing matrix, in units of log2, as right operands: [16 heads listened to][slot][lane], high and low parts
  for (int i = threadIdx.x; i < NS * 8 * (KS * 8); i += 128) {
    const int at = i / (KS * 8), d = (i - at * (KS * 8)) * 8, h = head_of(at >> 3, at & 7);
    *reinterpret_cast<uint4*>(s_q + at * C::Q_LD + d * 2) =
        h >= 0 && d < p.dim ? *reinterpret_cast<const uint4*>(p.q + b * p.ldq + (long long)h * p.dim + d) : make_uint4(0, 0, 0, 0);
  }
  for (int i = warp; i < NS / 2 * NS; i += 4) {
    const int ki = i / NS, h = head_of(i - ki * NS, r);
    float m[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int g = head_of(2 * ki + (e >> 1), 2 * c + (e & 1));
      m[e] = h >= 0 && g >= 0 ? p.mix[h * p.heads + g] * p.scale_log2 : 0.f;
    }
    const SplitPair x = split2(m[0], m[1]), y = split2(m[2], m[3]);
    reinterpret_cast<uint4*>(s_m)[i * 32 + lane] = make_uint4(x.hi, y.hi, x.lo, y.lo);
  }
  asm volatile("bar.sync 1, 128;" ::: "memory");

  constexpr int NW = NS > 4 ? NS / 4 : 1;      // slots of a warp
  float acc[NW][KS * 4][4], m[NW], l[NW];
#pragma unroll
  for (int i = 0; i < NW; ++i) {
    m[i] = -INFINITY;
    l[i] = 0.f;
#pragma unroll
    for (int x = 0; x < KS * 4; ++x)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][x][e] = 0.f;
  }
  int unit = 0, phase = 0;
  auto arrived = [&]() {
    const bool ok = mbar_wait(smem_u32(&full[unit]), phase, abort_flag, p.status, RB_ERR_TIMEOUT_FULL);
    return __all_sync(0xffffffffu, ok) != 0;
  };
  auto release = [&]() {
    __syncwarp();
    if (lane == 0) mbar_arrive(smem_u32(&empty[unit]));
    if (++unit == p.units) {
      unit = 0;
      phase ^= 1;
    }
  };
  // rows of a unit that this lane points ldmatrix at
  const int k_row = warp * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), k_half = lane >> 4;
  const int v_row = (lane >> 4) * 8 + (lane & 7), v_half = (lane >> 3) & 1;
  bool ok = true;
  for (int i = 0; i < n_tiles; ++i) {
    float* buf = s_s + (i & 1) * C::S_FLOATS;
    // ---- scores of 16 keys and all heads
    uint32_t hi[NS][2], lw[NS][2];
    int x = 0;                                 // slot of its key/value head
#pragma unroll
    for (int s = 0; s < NS; ++s) {
      float raw[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};      // even and odd steps
      if (ok && s < p.n_slots) {
        if (x == 0) ok = arrived();
        if (ok) {
          const uint32_t ks = smem_u32(smem + unit * C::UNIT), qs = smem_u32(s_q) + (s * 8 + (lane & 7)) * C::Q_LD + (lane >> 3) * 16;
#pragma unroll
          for (int k = 0; k < KS * 4; k += 2) {
            uint32_t kb[4], qb[4];
            ldmatrix_x4(qs + k * 32, qb);
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              const int chunk = (k + e) * 2 + k_half;
              ldmatrix_x4(ks + (chunk >> 3) * C::SUB + k_row * 128 + (((chunk & 7) ^ (k_row & 7)) << 4), kb);
              mma_bf16(raw[e], kb, qb[2 * e], qb[2 * e + 1]);
            }
          }
          if (++x == p.per_kv) {
            x = 0;
            release();
          }
        }
      }
      const SplitPair a = split2(raw[0][0] + raw[1][0], raw[0][1] + raw[1][1]), d = split2(raw[0][2] + raw[1][2], raw[0][3] + raw[1][3]);
      hi[s][0] = a.hi; hi[s][1] = d.hi;
      lw[s][0] = a.lo; lw[s][1] = d.lo;
    }
    // ---- mixed
#pragma unroll
    for (int n = 0; n < NS; ++n) {
      if (n >= p.n_slots) break;
      float o[3][4];
#pragma unroll
      for (int y = 0; y < 3; ++y)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[y][e] = 0.f;
#pragma unroll
      for (int k = 0; k < NS / 2; ++k) {
        const uint4 w = reinterpret_cast<const uint4*>(s_m)[(k * NS + n) * 32 + lane];
        const uint32_t ah[4] = {hi[2 * k][0], hi[2 * k][1], hi[2 * k + 1][0], hi[2 * k + 1][1]};
        const uint32_t al[4] = {lw[2 * k][0], lw[2 * k][1], lw[2 * k + 1][0], lw[2 * k + 1][1]};
        mma_bf16(o[0], ah, w.x, w.y);
        mma_bf16(o[1], al, w.x, w.y);
        mma_bf16(o[2], ah, w.z, w.w);
      }
      float* to = buf + (n * 8 + 2 * c) * kTdLd + warp * 16 + r;
#pragma unroll
      for (int e = 0; e < 4; ++e) to[(e & 1) * kTdLd + (e >> 1) * 8] = o[0][e] + (o[1][e] + o[2][e]);
    }
    asm volatile("bar.sync 1, 128;" ::: "memory");
    // ---- softmax and values, slot by slot
    const int key0 = (tile0 + i) * kTdKeys;
    const bool edge = key0 < lo || key0 + kTdKeys > ctx;
    x = 0;
#pragma unroll
    for (int j = 0; j < NW; ++j)
      for (int y = 0; y < 4; ++y) {
        const int s = j * 4 + y;
        if (!ok || s >= p.n_slots) break;
        if (x == 0) ok = arrived();
        if (!ok) break;
        if (y == warp) {
          const float* from = buf + (s * 8 + r) * kTdLd + 2 * c;      // this lane: head r of the slot, keys 2 c, 2 c + 1, + 8, ...
          float v[16];
          float mx = -INFINITY;
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            const float2 z = *reinterpret_cast<const float2*>(from + e * 8);
            v[2 * e] = z.x;
            v[2 * e + 1] = z.y;
          }
          if (edge) {
#pragma unroll
            for (int e = 0; e < 16; ++e) {
              const int at = key0 + (e >> 1) * 8 + 2 * c + (e & 1);
              if (at < lo || at >= ctx) v[e] = -INFINITY;
            }
          }
#pragma unroll
          for (int e = 0; e < 16; ++e) mx = fmaxf(mx, v[e]);
          mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
          mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
          if (__any_sync(0xffffffffu, mx > m[j] + 8.0f)) {            // rare after the first tiles
            float alpha = 1.f;
            if (mx > m[j]) {
              alpha = m[j] == -INFINITY ? 0.f : fast_exp2(m[j] - mx);
              m[j] = mx;
              l[j] *= alpha;
            }
            const float a0 = __shfl_sync(0xffffffffu, alpha, c * 8), a1 = __shfl_sync(0xffffffffu, alpha, c * 8 + 4);
#pragma unroll
            for (int t = 0; t < KS * 4; ++t) {
              acc[j][t][0] *= a0; acc[j][t][1] *= a1; acc[j][t][2] *= a0; acc[j][t][3] *= a1;
            }
          }
          const float neg = m[j] == -INFINITY ? 0.f : -m[j];
          uint32_t w[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            const float w0 = fast_exp2(v[2 * e] + neg), w1 = fast_exp2(v[2 * e + 1] + neg);
            l[j] += w0 + w1;
            w[e] = pack2<T>(w0, w1);
          }
          const uint32_t vs = smem_u32(smem + unit * C::UNIT);
#pragma unroll
          for (int k = 0; k < 4; ++k)
#pragma unroll
            for (int t = 0; t < KS * 4; ++t) {
              const int chunk = t * 2 + v_half, row = k * 16 + v_row;
              uint32_t va[4];
              ldmatrix_x4_trans(vs + (chunk >> 3) * C::SUB + row * 128 + (((chunk & 7) ^ (row & 7)) << 4), va);
              mma_bf16(acc[j][t], va, w[2 * k], w[2 * k + 1]);
            }
        }
        if (++x == p.per_kv) {
          x = 0;
          release();
        }
      }
    // after a wait that ran out a warp does no more work, but takes part in the barriers that the others wait at
  }
  if (!ok) {                                   // copies in flight land before the shared memory gets another use
    for (int i = 0; i < 64; ++i) __nanosleep(10000);
    return;
  }
#pragma unroll
  for (int j = 0; j < NW; ++j) {
    const int s = j * 4 + warp;
    if (s >= p.n_slots) break;
    l[j] += __shfl_xor_sync(0xffffffffu, l[j], 1);
    l[j] += __shfl_xor_sync(0xffffffffu, l[j], 2);
    const int h_row = head_of(s, r);
    float f = 1.f;
    if (p.splits > 1) {
      if (c == 0 && h_row >= 0) {
        float* ml = p.part_ml + (((long long)b * p.heads + h_row) * p.splits + sp) * 2;
        ml[0] = m[j];
        ml[1] = l[j];
      }
    } else if (h_row >= 0) {
      const float sk = p.sink ? p.sink[h_row] * 1.4426950408889634f : -INFINITY, gm = fmaxf(m[j], sk), f0 = fast_exp2(m[j] - gm);
      f = f0 / (l[j] * f0 + (p.sink ? fast_exp2(sk - gm) : 0.f));
      if (p.gate_kind == ATTN_GATE_HEAD) f *= sigmoid_f<T>(to_f32<T>(p.gate[b * p.ldg + h_row]));
    }
    const float f0 = __shfl_sync(0xffffffffu, f, c * 8), f1 = __shfl_sync(0xffffffffu, f, c * 8 + 4);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int h = head_of(s, 2 * c + e);
      if (h < 0) continue;
#pragma unroll
      for (int t = 0; t < KS * 4; ++t)
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int d = t * 16 + r + 8 * x;
          if (d >= p.vdim) continue;
          float v = acc[j][t][2 * x + e] * (e ? f1 : f0);
          if (p.splits > 1) {
            p.part_o[(((long long)b * p.heads + h) * p.splits + sp) * p.vdim + d] = v;
          } else {
            if (p.gate_kind == ATTN_GATE_ELEMENT) v *= sigmoid_f<T>(to_f32<T>(p.gate[b * p.ldg + (long long)h * p.vdim + d]));
            p.out[b * p.ldo + (long long)h * p.vdim + d] = from_f32<T>(v);
          }
        }
    }
  }
}

// Units of the ring and CTAs per SM: two where each has at least four units.
template <int KS, int NS>
int talk_decode_units(int& ctas) {
  using C = TalkDecodeCfg<KS, NS>;
  auto fit = [](int bytes) { return bytes <= C::FIXED ? 0 : (bytes - C::FIXED) / C::UNIT < kTdUnits ? (bytes - C::FIXED) / C::UNIT : kTdUnits; };
  ctas = fit(112 * 1024) >= 4 ? 2 : 1;
  return fit(ctas == 2 ? 112 * 1024 : 226 * 1024);
}

template <int KS, int NS>
int launch_talk_decode(TalkDecodeParams& p, const void* k_pool, const void* v_pool, long long pool_rows, int rows, cudaStream_t st) {
  using C = TalkDecodeCfg<KS, NS>;
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
  int ctas;
  p.units = talk_decode_units<KS, NS>(ctas);
  const int smem = C::FIXED + p.units * C::UNIT;
  auto kern = talk_decode_kernel<KS, NS>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return 2000 + (int)e;
  kern<<<dim3(rows, p.splits), 160, smem, st>>>(tk, tv, p);
  e = cudaGetLastError();
  return e == cudaSuccess ? 0 : 3000 + (int)e;
}

static int talk_slots(int heads, int kv_heads) { return kv_heads * ((heads / kv_heads + 7) / 8); }

template <typename F>
int talk_by_size(int dim_p, int slots, F go) {
  if (dim_p <= 64) return slots <= 2 ? go.template operator()<1, 2>() : slots <= 4 ? go.template operator()<1, 4>() : go.template operator()<1, 8>();
  return slots <= 2 ? go.template operator()<2, 2>() : slots <= 4 ? go.template operator()<2, 4>() : go.template operator()<2, 8>();
}

struct TalkDecodeCtas {
  template <int KS, int NS>
  int operator()() {
    int ctas;
    talk_decode_units<KS, NS>(ctas);
    return ctas;
  }
};
struct TalkDecodeLaunch {
  TalkDecodeParams& p;
  const void *k_pool, *v_pool;
  long long pool_rows;
  int rows;
  cudaStream_t st;
  template <int KS, int NS>
  int operator()() {
    return launch_talk_decode<KS, NS>(p, k_pool, v_pool, pool_rows, rows, st);
  }
};

}  // namespace rb

extern "C" {

// Whether the kernel covers these sizes (others run on rb_talk_rows): 16-bit, heads of up to 128 whose keys and values take
// equally many sub-tiles, at most eight slots of eight heads that share a key/value head.
int rb_talk_decode_ok(int dtype, int heads, int kv_heads, int dim_p, int vdim_p, int block_size) {
  return dtype == rbh::DT_BF16 && dim_p <= 128 && vdim_p <= 128 && dim_p % 8 == 0 && vdim_p % 8 == 0 && (dim_p > 64) == (vdim_p > 64) &&
         rb::talk_slots(heads, kv_heads) <= 8 && (block_size % 64 == 0 || (block_size >= 8 && 64 % block_size == 0));
}

// Slices of a row's visible keys (at most max_keys of them): whole waves of the resident CTAs.
int rb_talk_decode_splits(int heads, int kv_heads, int dim_p, int rows, int max_keys) {
  const int ctas = rb::talk_by_size(dim_p, rb::talk_slots(heads, kv_heads), rb::TalkDecodeCtas{});
  const long long slots = (long long)ctas * rbh::sm_count();
  const int tiles = (max_keys + rb::kTdKeys - 1) / rb::kTdKeys + 1;
  int best = 1;
  double best_cost = 1e30;
  for (int s = 1; s <= 256 && s <= tiles; ++s) {
    const long long waves = (rows * (long long)s + slots - 1) / slots;
    const double cost = (double)waves * ((tiles + s - 1) / s + 1.5) + (s > 1 ? 1.0 + s / 64.0 : 0.0);   // set-up and tail, merge
    if (cost < best_cost - 1e-9) {
      best_cost = cost;
      best = s;
    }
  }
  return best;
}

// Arguments as rb_talk_rows; num_blocks: blocks of the pools.
int rb_talk_decode(int dtype, const void* q, long long ldq, const void* k_pool, const void* v_pool, int num_blocks, const int* tables,
                   const int* ctx, const float* mix, const float* sink, const void* gate, long long ldg, int gate_kind, void* out,
                   long long ldo, float* part_o, float* part_ml, int rows, int heads, int kv_heads, int dim_p, int vdim_p, int window,
                   int block_size, int max_blocks, int splits, float scale, void* stream) {
  using namespace rb;
  if (rows <= 0) return 0;
  if (!rb_talk_decode_ok(dtype, heads, kv_heads, dim_p, vdim_p, block_size) || splits < 1 || splits > 256 || heads % kv_heads || window < 1)
    return 22;
  auto al = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
  if (!al(q) || !al(k_pool) || !al(v_pool) || ldq % 8) return 21;
  using T = __nv_bfloat16;
  TalkDecodeParams p{};
  p.q = (const T*)q; p.ldq = ldq; p.tables = tables; p.ctx = ctx; p.mix = mix; p.sink = sink; p.gate = (const T*)gate; p.ldg = ldg; p.ldo = ldo;
  p.out = (T*)out; p.part_o = part_o; p.part_ml = part_ml; p.heads = heads; p.kv_heads = kv_heads; p.dim = dim_p; p.vdim = vdim_p;
  p.window = window; p.block_size = block_size; p.box_rows = block_size < kTdKeys ? block_size : kTdKeys; p.max_blocks = max_blocks;
  p.splits = splits; p.gate_kind = gate ? gate_kind : ATTN_GATE_NONE; p.per_kv = (heads / kv_heads + 7) / 8;
  p.n_slots = talk_slots(heads, kv_heads); p.scale_log2 = scale * 1.4426950408889634f; p.status = rbh::device_status_word();
  cudaStream_t st = (cudaStream_t)stream;
  const int rc = talk_by_size(dim_p, p.n_slots, TalkDecodeLaunch{p, k_pool, v_pool, (long long)num_blocks * kv_heads * block_size, rows, st});
  if (rc || splits == 1) return rc;
  launch_attn_merge<T>(part_o, part_ml, sink, (const T*)gate, ldg, p.gate_kind, (T*)out, ldo, rows, heads, vdim_p, splits, st);
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : 3000 + (int)e;
}
}
