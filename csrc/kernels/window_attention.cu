// Sliding-window attention with grouped key/value heads over a paged cache, sm_100a: what follows the input
// projection, and single query rows of any size and type (32-bit runs, large heads).  16-bit rows are in
// window_decode.cu, prompt tiles in window_prefill.cu.
//
// Cache layout, keys and values each: pool [num_blocks, kv_heads, block_size, dim]; token t of a sequence is in
// block table[t / block_size], so a head's tokens of a block are one contiguous run.  Head sizes are padded to
// multiples of eight numbers with zeros.
#include <type_traits>

#include "attn_merge.cuh"

namespace rb {

// ---------------------------------------------------------------------------------------------------------
// after the input projection [q | k | v | ...]: optional RMS norm and rotation of every query and key head (norm
// first; pair i = elements i and i + half, or neighbours 2i and 2i + 1), then keys and values into their cache rows.  Queries change in place.
// One CTA per token, one warp per head at a time.  QUAD: heads of up to 128 numbers whose rotation is made of whole
// groups of four: a lane keeps four neighbouring numbers and gets their partners from another lane.
// ---------------------------------------------------------------------------------------------------------
template <typename T>
struct WindowPostParams {
  T* proj;
  long long ldp;
  const float2* tab;          // [tokens, half] (cos, sin), or null: no rotation
  const float *q_norm, *k_norm;   // [dim] or null
  const long long* slots;     // cache slot (block * block_size + offset) of every token, -1: keep nothing
  T *k_pool, *v_pool;
  int heads, kv_heads, dim, dim_p, vdim_p, half, block_size;
  int neighbours;             // pair i = elements 2i, 2i + 1
  float eps;
};

template <typename T>
__device__ __forceinline__ void load4(const T* p, float* f) {
  if constexpr (sizeof(T) == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  } else {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    const float2 lo = unpack2<T>(a.x), hi = unpack2<T>(a.y);
    f[0] = lo.x; f[1] = lo.y; f[2] = hi.x; f[3] = hi.y;
  }
}
template <typename T>
__device__ __forceinline__ void store4(T* p, const float* f) {
  if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  else *reinterpret_cast<uint2*>(p) = make_uint2(pack2<T>(f[0], f[1]), pack2<T>(f[2], f[3]));
}

template <typename T, bool QUAD>
__global__ void __launch_bounds__(256) window_post_kernel(const WindowPostParams<T> p) {
  const long long t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  T* row = p.proj + t * p.ldp;
  const long long slot = p.slots[t];
  const long long blk = slot / p.block_size;
  const int off = (int)(slot - blk * p.block_size);
  const bool plain_q = p.tab == nullptr && p.q_norm == nullptr;
  constexpr int V = 16 / sizeof(T);
  for (int i = warp + (plain_q ? p.heads : 0); i < p.heads + 2 * p.kv_heads; i += 8) {
    const bool is_q = i < p.heads, is_v = i >= p.heads + p.kv_heads;
    T* src = row + (is_v ? (long long)(p.heads + p.kv_heads) * p.dim_p + (long long)(i - p.heads - p.kv_heads) * p.vdim_p
                         : (long long)i * p.dim_p);
    T* dst = src;
    if (!is_q) {
      if (slot < 0) continue;
      const int g = i - p.heads - (is_v ? p.kv_heads : 0);
      const int w = is_v ? p.vdim_p : p.dim_p;
      dst = (is_v ? p.v_pool : p.k_pool) + ((blk * p.kv_heads + g) * p.block_size + off) * w;
    }
    if (is_v || plain_q) {
      const int n = (is_v ? p.vdim_p : p.dim_p) / V;
      for (int c = lane; c < n; c += 32) reinterpret_cast<uint4*>(dst)[c] = reinterpret_cast<const uint4*>(src)[c];
      continue;
    }
    const float* nw = is_q ? p.q_norm : p.k_norm;
    if constexpr (QUAD) {
      const int c = lane * 4, reach = p.tab ? p.half >> 2 : 0;      // lanes between the two halves of a pair
      float x[4] = {0.f, 0.f, 0.f, 0.f};
      if (c < p.dim_p) load4<T>(src + c, x);                        // zeros between dim and dim_p
      if (nw) {
        const float r = 1.0f / sqrtf(warp_sum(x[0] * x[0] + x[1] * x[1] + x[2] * x[2] + x[3] * x[3]) / p.dim + p.eps);
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (c + e < p.dim) x[e] *= r * nw[c + e];
      }
      if (p.neighbours) {
        if (lane < 2 * reach) {
          const float2* tb = p.tab + t * p.half + lane * 2;
#pragma unroll
          for (int e = 0; e < 4; e += 2) {
            const float2 cs = tb[e / 2];
            const float u = x[e], v = x[e + 1];
            x[e] = u * cs.x - v * cs.y;
            x[e + 1] = v * cs.x + u * cs.y;
          }
        }
        if (c < p.dim_p) store4<T>(dst + c, x);
        continue;
      }
      const bool low = lane < reach, high = !low && lane < 2 * reach;
      float other[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) other[e] = __shfl_sync(0xffffffffu, x[e], low ? lane + reach : high ? lane - reach : lane);
      if (low || high) {
        const float2* tb = p.tab + t * p.half + (low ? c : c - p.half);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 cs = tb[e];
          x[e] = low ? x[e] * cs.x - other[e] * cs.y : x[e] * cs.x + other[e] * cs.y;
        }
      }
      if (c < p.dim_p) store4<T>(dst + c, x);
      continue;
    }
    float r = 1.f;
    if (nw) {
      float s = 0.f;
      for (int c = lane; c < p.dim; c += 32) {
        const float v = to_f32<T>(src[c]);
        s += v * v;
      }
      s = warp_sum(s);
      r = 1.0f / sqrtf(s / p.dim + p.eps);
    }
    const float2* tb = p.tab + t * p.half;
    const int half = p.tab ? p.half : 0;
    // a pair belongs to one lane, so writing in place is safe
    for (int c = lane; c < half; c += 32) {
      const int a = p.neighbours ? 2 * c : c, b = p.neighbours ? 2 * c + 1 : c + half;
      float u = to_f32<T>(src[a]), v = to_f32<T>(src[b]);
      if (nw) {
        u *= r * nw[a];
        v *= r * nw[b];
      }
      const float2 cs = tb[c];
      dst[a] = from_f32<T>(u * cs.x - v * cs.y);
      dst[b] = from_f32<T>(v * cs.x + u * cs.y);
    }
    for (int c = 2 * half + lane; c < p.dim_p; c += 32) {
      float v = c < p.dim ? to_f32<T>(src[c]) : 0.f;
      if (nw && c < p.dim) v *= r * nw[c];
      dst[c] = from_f32<T>(v);
    }
  }
}

// ---------------------------------------------------------------------------------------------------------
// single query rows.  A CTA takes a slice of one row's visible keys for up to HPW * hgc query heads of one
// key/value head: four warps attend, and take turns at bringing tiles of keys and values into a ring with bulk
// copies (tiles start at multiples of their size, so a page holds whole ones).  Eight lanes share a key, each with
// chunks of eight numbers of it in registers for HPW heads; the HPW x KP scores of a trip are reduced so that each
// of the eight lanes ends up with one of them (two or four lanes with the same one when there are fewer), which it
// exponentiates and hands round.  All sums are fp32; maxima move only when they grow by more than 8 (in log2 units),
// so accumulators are rarely rescaled.
// ---------------------------------------------------------------------------------------------------------
struct WindowRowsParams {
  const void *q, *k_pool, *v_pool;
  long long ldq;                 // query row stride; head h at h * dim
  const int *tables, *ctx;       // [rows, max_blocks], [rows]: keys up to and with the row's own
  const float* sink;             // [heads] or null
  const void* gate;
  long long ldg, ldo;
  void* out;
  float *part_o, *part_ml;       // used when splits > 1
  int heads, kv_heads, dim, vdim, window, block_size, max_blocks, splits, gate_kind;
  int hgc, blocks_per_kv, tile, stages;
  int keep;                      // the first tokens stay visible outside the window
  float scale_log2, scale, cap, out_scale;   // cap 0: none
  int* status;
};

__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  float2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;"
      : "=l"(reinterpret_cast<unsigned long long&>(d))
      : "l"(reinterpret_cast<unsigned long long&>(a)), "l"(reinterpret_cast<unsigned long long&>(b)),
        "l"(reinterpret_cast<unsigned long long&>(c)));
  return d;
}

// eight numbers as four pairs
template <typename T>
__device__ __forceinline__ void load8(const T* p, float2* f) {
  if constexpr (sizeof(T) == 4) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    f[0] = make_float2(a.x, a.y); f[1] = make_float2(a.z, a.w);
    f[2] = make_float2(b.x, b.y); f[3] = make_float2(b.z, b.w);
  } else {
    const uint4 a = *reinterpret_cast<const uint4*>(p);
    f[0] = unpack2<T>(a.x); f[1] = unpack2<T>(a.y); f[2] = unpack2<T>(a.z); f[3] = unpack2<T>(a.w);
  }
}

// adds 2 HALF values of two lanes `o` apart; the lane with that bit set keeps the upper half of the sums
template <int HALF, int N>
__device__ __forceinline__ void fold_lanes(float (&s)[N], int sub, int o) {
  const bool up = sub & o;
#pragma unroll
  for (int e = 0; e < HALF; ++e) {
    const float keep = up ? s[e + HALF] : s[e], give = up ? s[e] : s[e + HALF];
    s[e] = keep + __shfl_xor_sync(0xffffffffu, give, o);
  }
}

template <typename T, int NJ, int HPW, int KP>     // KP: keys per trip and group of lanes
__global__ void __launch_bounds__(128, NJ * HPW <= 4 ? 4 : 2)
    window_rows_kernel(const WindowRowsParams p) {
  constexpr int NS = HPW * KP, DUP = 8 / NS;  // scores of a trip; lanes that end up with the same one
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ uint64_t bars[8];
  __shared__ int s_abort;
  __shared__ float s_ml[4][HPW][2];
  uint64_t *full = bars, *empty = bars + 4;
  volatile int* abort_flag = &s_abort;
  const int g = blockIdx.x / p.blocks_per_kv, bx = blockIdx.x - g * p.blocks_per_kv;
  const int b = blockIdx.y, sp = blockIdx.z;
  const int warp = uniform_warp_idx(), lane = threadIdx.x & 31;
  const int rep = p.heads / p.kv_heads;
  const int head0 = bx * p.hgc * HPW;         // first head of the CTA inside the group
  const int ctx = p.ctx[b];
  // keys are numbered as if the kept ones lay directly before the window: lo .. win are tokens 0 .. kept, from win on a
  // key's number is its token's
  const int win = max(0, ctx - p.window), kept = min(p.keep, win), lo = win - kept, n = ctx - lo;
  const int per = (n + p.splits - 1) / p.splits;
  const int t0 = lo + sp * per, t1 = min(ctx, t0 + per);
  if (t0 >= t1) {                             // nothing of this row falls into the slice (splits > 1)
    for (int i = threadIdx.x; i < p.hgc * HPW; i += 128)
      if (head0 + i < rep) {
        float* ml = p.part_ml + (((long long)b * p.heads + g * rep + head0 + i) * p.splits + sp) * 2;
        ml[0] = -INFINITY;
        ml[1] = 0.f;
      }
    return;
  }
  const int base0 = t0 / p.tile * p.tile;     // tile i holds keys max(t0, base0 + i tile) .. min(t1, base0 + (i + 1) tile)
  const int n_tiles = (t1 - base0 + p.tile - 1) / p.tile;
  const int k_bytes = p.tile * p.dim * (int)sizeof(T), stage_bytes = k_bytes + p.tile * p.vdim * (int)sizeof(T);
  const int* table = p.tables + (long long)b * p.max_blocks;
  auto block_at = [&](int page) -> int { return table[min(page, p.max_blocks - 1)]; };
  auto token_of = [&](int t) { return t < win ? t - lo : t; };
  auto page_of = [&](int i) -> int {          // block of the first key of tile i
    return i < n_tiles ? block_at(token_of(max(t0, base0 + i * p.tile)) / p.block_size) : 0;
  };
  if (threadIdx.x == 0) {
    for (int s = 0; s < p.stages; ++s) {
      mbar_init(smem_u32(&full[s]), 1);
      mbar_init(smem_u32(&empty[s]), 4);
    }
    s_abort = 0;
    fence_barrier_init();
  }
  __syncthreads();

  // one lane: tile i into its stage; `page` is page_of(i)
  auto bring = [&](int i, int page) {
    const int st = i % p.stages;
    const int first = max(t0, base0 + i * p.tile), last = min(t1, base0 + (i + 1) * p.tile);
    const uint32_t bar = smem_u32(&full[st]), dst = smem_u32(smem + st * stage_bytes);
    mbar_arrive_expect_tx(bar, (last - first) * (p.dim + p.vdim) * (int)sizeof(T));
    for (int t = first; t < last;) {
      const int tok = token_of(t), pg = tok / p.block_size, off = tok - pg * p.block_size;
      const int run = min((t < win ? min(last, win) : last) - t, p.block_size - off);
      const long long blk = t == first ? page : block_at(pg);
      const long long r = (blk * p.kv_heads + g) * p.block_size + off;
      bulk_load_1d(dst + (t - first) * p.dim * (int)sizeof(T), reinterpret_cast<const T*>(p.k_pool) + r * p.dim,
                   run * p.dim * (int)sizeof(T), bar);
      bulk_load_1d(dst + k_bytes + (t - first) * p.vdim * (int)sizeof(T), reinterpret_cast<const T*>(p.v_pool) + r * p.vdim,
                   run * p.vdim * (int)sizeof(T), bar);
      t += run;
    }
  };
  // warp w brings tiles w, w + 4, ...; the first `stages` of them need no room made for them
  if (lane == 0 && warp < p.stages && warp < n_tiles) bring(warp, page_of(warp));
  int duty = warp < p.stages ? warp + 4 : warp;
  int duty_page = lane == 0 ? page_of(duty) : 0;

  {
    const int grp = lane >> 3, sub = lane & 7;
    const int hg = warp % p.hgc, wi = warp / p.hgc;           // which heads; which of the warps that share them
    const int groups = 16 / p.hgc, gid = wi * 4 + grp;
    const int h0 = head0 + hg * HPW;
    const int kc = p.dim >> 3, vc = p.vdim >> 3;              // chunks of eight numbers
    float2 q[HPW][NJ * 4], acc[HPW][NJ * 4];
    const float q_scale = p.cap > 0.f ? p.scale : p.scale_log2;
#pragma unroll
    for (int h = 0; h < HPW; ++h) {
      const T* qp = reinterpret_cast<const T*>(p.q) + b * p.ldq + (long long)(g * rep + min(h0 + h, rep - 1)) * p.dim;
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const int c = sub + 8 * j;
        if (c < kc) load8<T>(qp + c * 8, &q[h][j * 4]);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          q[h][j * 4 + e] = c < kc ? make_float2(q[h][j * 4 + e].x * q_scale, q[h][j * 4 + e].y * q_scale)
                                   : make_float2(0.f, 0.f);
          acc[h][j * 4 + e] = make_float2(0.f, 0.f);
        }
      }
    }
    auto ex2 = [](float x) { return sizeof(T) == 4 ? exp2f(x) : fast_exp2(x); };
    // this lane's score of a trip is number sub / DUP: head (sub / DUP) % HPW, key (sub / DUP) / HPW
    float m = -INFINITY, l = 0.f;
    bool ok = true;
    for (int i = 0; i < n_tiles; ++i) {
      const int st = i % p.stages;
      // the stage that tile i - 1 had is for tile i - 1 + stages
      if (i > 0 && duty == i - 1 + p.stages) {
        if (duty < n_tiles) {
          if (lane == 0) {
            ok = mbar_wait(smem_u32(&empty[(i - 1) % p.stages]), ((i - 1) / p.stages) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_EMPTY);
            if (ok) bring(duty, duty_page);
            duty_page = page_of(duty + 4);
          }
          ok = __shfl_sync(0xffffffffu, (int)ok, 0) != 0;
          if (!ok) break;
        }
        duty += 4;
      }
      ok = mbar_wait(smem_u32(&full[st]), (i / p.stages) & 1, abort_flag, p.status, RB_ERR_TIMEOUT_FULL);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      const int cnt = min(t1, base0 + (i + 1) * p.tile) - max(t0, base0 + i * p.tile);
      const T* sk = reinterpret_cast<const T*>(smem + st * stage_bytes);
      const T* sv = reinterpret_cast<const T*>(smem + st * stage_bytes + k_bytes);
      // keys base + gid, base + groups + gid, ...; whole trips need no bounds
      auto trip = [&](int base, auto whole) {
        constexpr bool WHOLE = decltype(whole)::value;
        auto key = [&](int kx) { return WHOLE ? base + kx * groups + gid : min(base + kx * groups + gid, cnt - 1); };
        float s[NS];
#pragma unroll
        for (int kx = 0; kx < KP; ++kx) {
          float2 d[HPW];
#pragma unroll
          for (int h = 0; h < HPW; ++h) d[h] = make_float2(0.f, 0.f);
          const T* kr = sk + key(kx) * p.dim;
#pragma unroll
          for (int j = 0; j < NJ; ++j)
            if (sub + 8 * j < kc) {
              float2 k[4];
              load8<T>(kr + (sub + 8 * j) * 8, k);
#pragma unroll
              for (int h = 0; h < HPW; ++h)
#pragma unroll
                for (int e = 0; e < 4; ++e) d[h] = fma2(q[h][j * 4 + e], k[e], d[h]);
            }
#pragma unroll
          for (int h = 0; h < HPW; ++h) s[kx * HPW + h] = d[h].x + d[h].y;
        }
        // sums over the eight lanes, scattered: lane sub keeps score number sub / DUP
        if constexpr (NS == 8) {
          fold_lanes<4>(s, sub, 4);
          fold_lanes<2>(s, sub, 2);
          fold_lanes<1>(s, sub, 1);
        } else if constexpr (NS == 4) {
          fold_lanes<2>(s, sub, 4);
          fold_lanes<1>(s, sub, 2);
          s[0] += __shfl_xor_sync(0xffffffffu, s[0], 1);
        } else {
          fold_lanes<1>(s, sub, 4);
          s[0] += __shfl_xor_sync(0xffffffffu, s[0], 2);
          s[0] += __shfl_xor_sync(0xffffffffu, s[0], 1);
        }
        float v = s[0];
        if (p.cap > 0.f) v = (sizeof(T) == 4 ? p.cap * tanhf(v / p.cap) : soft_cap(v, 2.8853900817779268f / p.cap, p.cap)) * 1.4426950408889634f;
        if (!WHOLE && base + (sub / DUP / HPW) * groups + gid >= cnt) v = -INFINITY;
        float mx = v;
#pragma unroll
        for (int o = HPW * DUP; o < 8; o <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        const bool need = mx > m + 8.0f;
        if (__any_sync(0xffffffffu, need)) {
          float alpha = 1.f;
          if (need) {
            alpha = m == -INFINITY ? 0.f : ex2(m - mx);
            m = mx;
            l *= alpha;
          }
#pragma unroll
          for (int h = 0; h < HPW; ++h) {
            const float a = __shfl_sync(0xffffffffu, alpha, (lane & 24) + h * DUP);
#pragma unroll
            for (int e = 0; e < NJ * 4; ++e) acc[h][e] = make_float2(acc[h][e].x * a, acc[h][e].y * a);
          }
        }
        const float pr = !WHOLE && v == -INFINITY ? 0.f : ex2(v - m);
        l += pr;
#pragma unroll
        for (int kx = 0; kx < KP; ++kx) {
          float2 w[HPW];
#pragma unroll
          for (int h = 0; h < HPW; ++h) {
            const float a = __shfl_sync(0xffffffffu, pr, (lane & 24) + (kx * HPW + h) * DUP);
            w[h] = make_float2(a, a);
          }
          const T* vr = sv + key(kx) * p.vdim;
#pragma unroll
          for (int j = 0; j < NJ; ++j)
            if (sub + 8 * j < vc) {
              float2 vv[4];
              load8<T>(vr + (sub + 8 * j) * 8, vv);
#pragma unroll
              for (int h = 0; h < HPW; ++h)
#pragma unroll
                for (int e = 0; e < 4; ++e) acc[h][j * 4 + e] = fma2(w[h], vv[e], acc[h][j * 4 + e]);
            }
        }
      };
      int base = 0;
      for (; base + groups * KP <= cnt; base += groups * KP) trip(base, std::true_type{});
      if (base < cnt) trip(base, std::false_type{});
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&empty[st]));
    }
    if (!ok)                                   // copies in flight land before the shared memory gets another use
      for (int i = 0; i < 64; ++i) __nanosleep(10000);
    // the four groups of lanes of a warp
    float mw = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 8));
    mw = fmaxf(mw, __shfl_xor_sync(0xffffffffu, mw, 16));
    const float f = m == -INFINITY ? 0.f : ex2(m - mw);
    l *= f;
#pragma unroll
    for (int o = HPW * DUP; o < 32; o <<= 1) l += __shfl_xor_sync(0xffffffffu, l, o);   // keys of a trip, then groups
#pragma unroll
    for (int h = 0; h < HPW; ++h) {
      const float a = __shfl_sync(0xffffffffu, f, (lane & 24) + h * DUP);
#pragma unroll
      for (int e = 0; e < NJ * 4; ++e) {
        float2 x = make_float2(acc[h][e].x * a, acc[h][e].y * a);
#pragma unroll
        for (int o = 8; o < 32; o <<= 1) {
          x.x += __shfl_xor_sync(0xffffffffu, x.x, o);
          x.y += __shfl_xor_sync(0xffffffffu, x.y, o);
        }
        acc[h][e] = x;
      }
    }
    if (lane < HPW * DUP && lane % DUP == 0) {
      s_ml[warp][lane / DUP][0] = mw;
      s_ml[warp][lane / DUP][1] = l;
    }
    // every warp is through with the ring before sums go over it; all four get here on every path
    asm volatile("bar.sync 1, 128;" ::: "memory");
    float* so = reinterpret_cast<float*>(smem);               // [4 warps][HPW][vdim]
    if (grp == 0) {
#pragma unroll
      for (int h = 0; h < HPW; ++h)
#pragma unroll
        for (int j = 0; j < NJ; ++j)
          if (sub + 8 * j < vc)
#pragma unroll
            for (int e = 0; e < 4; ++e)
              *reinterpret_cast<float2*>(so + (warp * HPW + h) * p.vdim + (sub + 8 * j) * 8 + 2 * e) = acc[h][j * 4 + e];
    }
    asm volatile("bar.sync 1, 128;" ::: "memory");
    for (int x = threadIdx.x; x < p.hgc * HPW * p.vdim; x += 128) {
      const int hl = x / p.vdim, d = x - hl * p.vdim;         // head of the CTA, number
      if (head0 + hl >= rep) break;
      const int w0 = hl / HPW, hh = hl - w0 * HPW;            // warps w0, w0 + hgc, ... have it
      const int h = g * rep + head0 + hl;
      float gm = -INFINITY;
      for (int w = w0; w < 4; w += p.hgc) gm = fmaxf(gm, s_ml[w][hh][0]);
      const float sk = p.splits == 1 && p.sink ? p.sink[h] * 1.4426950408889634f : -INFINITY;
      gm = fmaxf(gm, sk);
      float gl = 0.f, o = 0.f;
      for (int w = w0; w < 4; w += p.hgc) {
        const float mv = s_ml[w][hh][0];
        const float fw = mv == -INFINITY ? 0.f : ex2(mv - gm);
        gl += s_ml[w][hh][1] * fw;
        o += so[(w * HPW + hh) * p.vdim + d] * fw;
      }
      if (p.splits > 1) {
        const long long pi = ((long long)b * p.heads + h) * p.splits + sp;
        p.part_o[pi * p.vdim + d] = o;
        if (d == 0) {
          p.part_ml[pi * 2] = gm;
          p.part_ml[pi * 2 + 1] = gl;
        }
      } else {
        if (sk != -INFINITY) gl += ex2(sk - gm);
        float v = gl > 0.f ? o / gl * p.out_scale : 0.f;
        if (p.gate_kind == ATTN_GATE_ELEMENT) v *= sigmoid_f<T>(to_f32<T>(reinterpret_cast<const T*>(p.gate)[b * p.ldg + (long long)h * p.vdim + d]));
        else if (p.gate_kind == ATTN_GATE_HEAD) v *= sigmoid_f<T>(to_f32<T>(reinterpret_cast<const T*>(p.gate)[b * p.ldg + h]));
        reinterpret_cast<T*>(p.out)[b * p.ldo + (long long)h * p.vdim + d] = from_f32<T>(v);
      }
    }
  }
}

// Heads a warp carries, for the sizes of a head and the query heads that share a key/value head; 0: too large.
static int window_rows_heads(int dim, int vdim, int rep) {
  const int d = dim > vdim ? dim : vdim;
  const int most = d <= 64 ? 4 : d <= 256 ? 2 : d <= 512 ? 1 : 0;
  const int want = rep >= 3 ? 4 : rep;
  return want < most ? want : most;
}

template <typename T, int NJ, int HPW, int KP>
int launch_window_rows(WindowRowsParams& p, int rows, cudaStream_t st) {
  const int rep = p.heads / p.kv_heads;
  const int hgs = (rep + HPW - 1) / HPW;
  p.hgc = hgs >= 3 ? 4 : hgs;
  p.blocks_per_kv = (rep + p.hgc * HPW - 1) / (p.hgc * HPW);
  const int key_bytes = (p.dim + p.vdim) * (int)sizeof(T);
  p.tile = 64;
  while (p.tile > 8 && p.tile * key_bytes > 16 * 1024) p.tile /= 2;
  const int stage = p.tile * key_bytes;
  p.stages = 3 * stage <= 48 * 1024 ? 3 : 2;
  int smem = p.stages * stage;
  if (smem < 4 * HPW * p.vdim * 4) smem = 4 * HPW * p.vdim * 4;
  auto kern = window_rows_kernel<T, NJ, HPW, KP>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return 2000 + (int)e;
  kern<<<dim3(p.kv_heads * p.blocks_per_kv, rows, p.splits), 128, smem, st>>>(p);
  e = cudaGetLastError();
  return e == cudaSuccess ? 0 : 3000 + (int)e;
}

template <typename T>
int window_rows_by_size(WindowRowsParams& p, int rows, cudaStream_t st) {
  const int d = p.dim > p.vdim ? p.dim : p.vdim;
  const int hpw = window_rows_heads(p.dim, p.vdim, p.heads / p.kv_heads);
  // a trip of all 16 groups of lanes should not be longer than a tile of 32 keys
  const bool pairs = p.heads / p.kv_heads > 2;               // two heads a warp: two warps or more share keys
  if (d <= 64) {
    if (hpw == 4) return launch_window_rows<T, 1, 4, 2>(p, rows, st);
    if (hpw == 2) return launch_window_rows<T, 1, 2, 2>(p, rows, st);
    return launch_window_rows<T, 1, 1, 2>(p, rows, st);
  }
  if (d <= 128) {
    if (hpw == 2) return pairs ? launch_window_rows<T, 2, 2, 4>(p, rows, st) : launch_window_rows<T, 2, 2, 2>(p, rows, st);
    return launch_window_rows<T, 2, 1, 2>(p, rows, st);
  }
  if (d <= 256) {
    if (hpw == 2) return launch_window_rows<T, 4, 2, 2>(p, rows, st);
    return launch_window_rows<T, 4, 1, 2>(p, rows, st);
  }
  return launch_window_rows<T, 8, 1, 2>(p, rows, st);
}

}  // namespace rb

#define RB_BY_DTYPE(...)                                               \
  if (dtype == rbh::DT_BF16) { using T = __nv_bfloat16; __VA_ARGS__; } \
  else if (dtype == rbh::DT_F32) { using T = float; __VA_ARGS__; }     \
  else return 20;
#define RB_LAUNCH_STATUS()             \
  cudaError_t e_ = cudaGetLastError(); \
  return e_ == cudaSuccess ? 0 : 3000 + (int)e_

extern "C" {

// proj row: heads x dim_p queries, kv_heads x dim_p keys, kv_heads x vdim_p values; tab, q_norm / k_norm may be null
int rb_window_post(int dtype, void* proj, long long ldp, const float* tab, const float* q_norm, const float* k_norm,
                   const long long* slots, void* k_pool, void* v_pool, long long tokens, int heads, int kv_heads, int dim,
                   int dim_p, int vdim_p, int rot, int neighbours, int block_size, float eps, void* stream) {
  using namespace rb;
  if (tokens <= 0) return 0;
  if ((rot & 1) || rot > dim || dim > dim_p || dim_p % 8 || vdim_p % 8 || ldp % 8 || (q_norm == nullptr) != (k_norm == nullptr)) return 21;
  const bool quad = dim_p <= 128 && (!tab || rot % 8 == 0);
  RB_BY_DTYPE({
    const WindowPostParams<T> p{(T*)proj, ldp, (const float2*)tab, q_norm, k_norm, slots, (T*)k_pool, (T*)v_pool, heads, kv_heads,
                                dim, dim_p, vdim_p, rot / 2, block_size, neighbours, eps};
    if (quad) window_post_kernel<T, true><<<(unsigned)tokens, 256, 0, (cudaStream_t)stream>>>(p);
    else window_post_kernel<T, false><<<(unsigned)tokens, 256, 0, (cudaStream_t)stream>>>(p);
  })
  RB_LAUNCH_STATUS();
}

// Slices of a row's visible keys (at most max_keys of them).
int rb_window_rows_splits(int heads, int kv_heads, int dim_p, int vdim_p, int rows, int max_keys) {
  const int hpw = rb::window_rows_heads(dim_p, vdim_p, heads / kv_heads);
  if (hpw == 0 || rows <= 0) return 1;
  const int hgs = (heads / kv_heads + hpw - 1) / hpw, hgc = hgs >= 3 ? 4 : hgs;
  const long long ctas = (long long)kv_heads * ((hgs + hgc - 1) / hgc) * rows;
  // whole waves of four CTAs per SM; a slice costs about two tiles' worth of set-up and tail
  const long long slots = 4LL * rbh::sm_count();
  const int tiles = (max_keys + 31) / 32;
  int best = 1;
  double best_cost = 1e30;
  for (int s = 1; s <= 64 && 2 * s <= tiles + 1; ++s) {
    const long long waves = (ctas * s + slots - 1) / slots;
    const double cost = (double)waves * ((tiles + s - 1) / s + 2.0) + (s > 1 ? 4.0 : 0.0);
    if (cost < best_cost - 1e-9) {
      best_cost = cost;
      best = s;
    }
  }
  return best;
}

// q: row t, head h at q[t * ldq + h * dim_p]; out the same with ldo and vdim_p.  gate_kind: see attn_merge.cuh.
// Every row sees the last `window` of its keys and the sequence's first `keep`.  cap > 0: soft cap of the scaled
// scores.  out_scale: factor on the result.  Scratch for splits > 1: part_o rows*heads*splits*vdim_p floats, part_ml rows*heads*splits*2.
int rb_window_rows(int dtype, const void* q, long long ldq, const void* k_pool, const void* v_pool, const int* tables,
                   const int* ctx, const float* sink, const void* gate, long long ldg, int gate_kind, void* out,
                   long long ldo, float* part_o, float* part_ml, int rows, int heads, int kv_heads, int dim_p, int vdim_p,
                   int window, int keep, int block_size, int max_blocks, int splits, float scale, float cap, float out_scale,
                   void* stream) {
  using namespace rb;
  if (rows <= 0) return 0;
  if (rows > 65535 || splits < 1 || splits > 64 || heads % kv_heads || window < 1 || keep < 0 || block_size < 1 ||
      window_rows_heads(dim_p, vdim_p, heads / kv_heads) == 0)
    return 22;
  auto al = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
  if (!al(q) || !al(k_pool) || !al(v_pool) || ldq % 8 || dim_p % 8 || vdim_p % 8) return 21;
  WindowRowsParams p{};
  p.q = q; p.k_pool = k_pool; p.v_pool = v_pool; p.ldq = ldq; p.tables = tables; p.ctx = ctx; p.sink = sink; p.gate = gate;
  p.ldg = ldg; p.ldo = ldo; p.out = out; p.part_o = part_o; p.part_ml = part_ml; p.heads = heads; p.kv_heads = kv_heads;
  p.dim = dim_p; p.vdim = vdim_p; p.window = window; p.block_size = block_size; p.max_blocks = max_blocks; p.splits = splits;
  p.gate_kind = gate ? gate_kind : ATTN_GATE_NONE; p.scale_log2 = scale * 1.4426950408889634f; p.scale = scale;
  p.keep = keep; p.cap = cap; p.out_scale = out_scale;
  p.status = rbh::device_status_word();
  cudaStream_t st = (cudaStream_t)stream;
  int rc = 0;
  RB_BY_DTYPE((rc = window_rows_by_size<T>(p, rows, st)))
  if (rc || splits == 1) return rc;
  RB_BY_DTYPE((launch_attn_merge<T>(part_o, part_ml, sink, (const T*)gate, ldg, p.gate_kind, (T*)out, ldo, rows, heads, vdim_p, splits, st, out_scale)))
  RB_LAUNCH_STATUS();
}
}
