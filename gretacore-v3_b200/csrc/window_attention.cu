// Windowed attention with kept first tokens, per-head temperature, soft cap, logarithmic distance bias and a softmax sink,
// behind a short causal convolution of q, k and v and a per-head normalisation of q and k.
//   conv_norm_kernel / conv_history_kernel   portions: convolution, norm, cache write; then the convolution's history
//   window_rows_kernel     one thread-block cluster per row and group of query heads, the keys split over its CTAs.  In the
//                          decode form the kernel convolves and normalises the new token itself (its q in every CTA, its k and v
//                          in the CTA that owns the last key, which writes them to the cache): one kernel per decode step
//   window_mma_kernel      prompts: 64 query positions of a head per CTA on the tensor cores (mma.sync, fp16 operands)
// Key list of position i: the kept positions in front of the window, then the window.  Scores, weights and sums are fp32.
#include <cooperative_groups.h>

#include <algorithm>

#include "dense_device.cuh"
#include "mma_device.cuh"

using namespace greta;

namespace {

namespace cg = cooperative_groups;

__host__ __device__ constexpr uint32_t up8(uint32_t d) { return (d + 7u) & ~7u; }

struct WinArgs {
  greta_window_attn a;
  greta_rows rows;
};

__device__ __forceinline__ uint32_t cache_row(const greta_window_attn &a, uint32_t p) {
  return p < a.keep_first ? p : a.keep_first + (p - a.keep_first) % a.ring;
}
// Keys that a row (or a tile of rows from position i0 on, up to i1) may see, as a list: the kept positions in front of the
// window, then the window; and where they lie in the cache (one division per list, none per key).
struct KeyList {
  uint32_t kept, lo, total, keep, ring, p0, base;
  __device__ __forceinline__ KeyList(const greta_window_attn &a, uint32_t i0, uint32_t i1) {
    lo = a.window && i0 + 1 > a.window ? i0 + 1 - a.window : 0;
    kept = min(a.keep_first, lo);
    total = kept + (i1 - lo + 1);
    keep = a.keep_first;
    ring = a.ring;
    p0 = max(lo, keep);
    base = (p0 - keep) % ring;
  }
  __device__ __forceinline__ uint32_t position(uint32_t t) const { return t < kept ? t : lo + (t - kept); }
  __device__ __forceinline__ uint32_t row(uint32_t t) const {
    const uint32_t p = position(t);
    if (p < keep) return p;
    const uint32_t o = base + (p - p0);  // p - p0 < ring: a ring holds every position that is seen
    return keep + (o >= ring ? o - ring : o);
  }
};
template <typename CT>
__device__ __forceinline__ CT to_cache(float v);
template <>
__device__ __forceinline__ float to_cache<float>(float v) { return v; }
template <>
__device__ __forceinline__ __half to_cache<__half>(float v) { return __float2half_rn(v); }
__device__ __forceinline__ void load8(const __half *p, float (&f)[8]) {
  const uint4 u = *reinterpret_cast<const uint4 *>(p);
  const float2 a = h2_to_f2(u.x), b = h2_to_f2(u.y), c = h2_to_f2(u.z), d = h2_to_f2(u.w);
  f[0] = a.x, f[1] = a.y, f[2] = b.x, f[3] = b.y, f[4] = c.x, f[5] = c.y, f[6] = d.x, f[7] = d.y;
}
__device__ __forceinline__ void load8(const float *p, float (&f)[8]) {
  const float4 a = *reinterpret_cast<const float4 *>(p), b = *reinterpret_cast<const float4 *>(p + 4);
  f[0] = a.x, f[1] = a.y, f[2] = a.z, f[3] = a.w, f[4] = b.x, f[5] = b.y, f[6] = b.z, f[7] = b.w;
}
__device__ __forceinline__ float4 load4(const __half *p) {
  const uint2 u = *reinterpret_cast<const uint2 *>(p);
  const float2 a = h2_to_f2(u.x), b = h2_to_f2(u.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ float4 load4(const float *p) { return *reinterpret_cast<const float4 *>(p); }

// Convolved channel c of the token at position p, activation row m of the launch; rows of the launch that belong to the same
// sequence start at position first.
__device__ __forceinline__ float conv_channel(const greta_window_attn &a, uint32_t m, uint32_t slot, uint32_t p, uint32_t first, uint32_t c) {
  const float cur = a.proj[(size_t)m * a.ld_proj + c];
  if (!a.conv) return cur;
  const uint32_t C = (a.heads + a.kv_heads) * a.dim + a.kv_heads * a.vdim;
  const float *w = a.conv + (size_t)c * a.taps;
  float y = 0.f;
  for (uint32_t back = a.taps - 1; back >= 1; --back) {
    if (back > p) continue;
    const uint32_t q = p - back;
    const float u = q >= first ? a.proj[(size_t)(m - back) * a.ld_proj + c] : a.history[((size_t)slot * a.taps + q % a.taps) * C + c];
    y = fmaf(w[a.taps - 1 - back], u, y);
  }
  return fmaf(w[a.taps - 1], cur, y);
}
// One warp: the d channels from column c0, convolved, optionally divided by their root mean square; lane holds channels
// lane + 32 i.
__device__ __forceinline__ void conv_head(const greta_window_attn &a, uint32_t m, uint32_t slot, uint32_t p, uint32_t first, uint32_t c0, uint32_t d,
                                          bool norm, int lane, float (&v)[8]) {
  float q = 0.f;
  if (a.conv && a.taps <= 4) {  // all loads in flight before the first is used
    const uint32_t C = (a.heads + a.kv_heads) * a.dim + a.kv_heads * a.vdim;
    float u[8][4], cw[8][4];
    const float *past[4];
#pragma unroll
    for (int back = 0; back < 4; ++back) {
      const bool on = back < (int)a.taps && back <= (int)p;
      const uint32_t at = p - back;
      past[back] = !on ? nullptr : at >= first ? a.proj + (size_t)(m - back) * a.ld_proj + c0 : a.history + ((size_t)slot * a.taps + at % a.taps) * C + c0;
    }
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int back = 0; back < 4; ++back) {
        const uint32_t c = lane + 32 * i;
        const bool on = c < d && past[back];
        u[i][back] = on ? past[back][c] : 0.f;
        cw[i][back] = on ? a.conv[(size_t)(c0 + c) * a.taps + a.taps - 1 - back] : 0.f;
      }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      v[i] = fmaf(cw[i][0], u[i][0], fmaf(cw[i][1], u[i][1], fmaf(cw[i][2], u[i][2], cw[i][3] * u[i][3])));
      q = fmaf(v[i], v[i], q);
    }
  } else {
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const uint32_t c = lane + 32 * i;
      v[i] = c < d ? conv_channel(a, m, slot, p, first, c0 + c) : 0.f;
      q = fmaf(v[i], v[i], q);
    }
  }
  if (norm) {
    const float inv = 1.f / sqrtf(warp_sum(q) / (float)d + a.eps);
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] *= inv;
  }
}
// Where head unit u (query heads, then key heads, then value heads) starts among the projected columns.
__device__ __forceinline__ uint32_t unit_col(const greta_window_attn &a, uint32_t u) {
  const uint32_t HK = a.heads + a.kv_heads;
  return u < HK ? u * a.dim : HK * a.dim + (u - HK) * a.vdim;
}
template <typename CT>
__device__ __forceinline__ void store_cache(const greta_window_attn &a, uint32_t slot, uint32_t p, uint32_t g, bool is_v, int lane, const float (&v)[8]) {
  const uint32_t d8 = up8(is_v ? a.vdim : a.dim), rows = a.keep_first + a.ring;
  CT *dst = static_cast<CT *>(is_v ? a.v_cache : a.k_cache) + (((size_t)slot * a.kv_heads + g) * rows + cache_row(a, p)) * d8;
#pragma unroll
  for (int i = 0; i < 8; ++i)
    if (lane + 32 * i < d8) dst[lane + 32 * i] = to_cache<CT>(v[i]);
}

// A warp takes one head unit through CV_ROWS consecutive rows: the convolution's weights and its window of projected rows
// stay in registers, every projected value is read once.  TAPS 0: no convolution; CH: 32-channel groups of the widest head.
constexpr int CV_ROWS = 16;
template <typename CT, int TAPS, int CH>
__global__ void __launch_bounds__(256) conv_norm_kernel(const __grid_constant__ WinArgs w, float *__restrict__ q_out) {
  constexpr int W = TAPS > 1 ? TAPS : 1;
  pdl_launch_dependents();
  pdl_wait();
  const greta_window_attn &a = w.a;
  const uint32_t u = blockIdx.x * 8 + (threadIdx.x >> 5), m0 = blockIdx.y * CV_ROWS, m1 = min(m0 + CV_ROWS, w.rows.M), slot = w.rows.slot0;
  const int lane = threadIdx.x & 31;
  const uint32_t HK = a.heads + a.kv_heads, C = HK * a.dim + a.kv_heads * a.vdim;
  if (u >= HK + a.kv_heads) return;
  const bool is_v = u >= HK;
  const uint32_t d = is_v ? a.vdim : a.dim, d8 = up8(d), c0 = unit_col(a, u) + lane;
  float cw[CH][W], win[CH][W];  // win[.][j]: the projected value W - 1 - j rows back
#pragma unroll
  for (int i = 0; i < CH; ++i)
#pragma unroll
    for (int j = 0; j < W; ++j) {
      const bool on = lane + 32 * i < (int)d;
      cw[i][j] = TAPS && on ? a.conv[(size_t)(c0 + 32 * i) * TAPS + j] : 1.f;
      win[i][j] = 0.f;
      const uint32_t back = W - 1 - j, p = w.rows.pos0 + m0;
      if (back && on && back <= p) {
        const uint32_t q = p - back;
        win[i][j] = back <= m0 ? a.proj[(size_t)(m0 - back) * a.ld_proj + c0 + 32 * i] : a.history[((size_t)slot * W + q % W) * C + c0 + 32 * i];
      }
    }
  float cur[CH];
#pragma unroll
  for (int i = 0; i < CH; ++i) cur[i] = lane + 32 * i < (int)d ? a.proj[(size_t)m0 * a.ld_proj + c0 + 32 * i] : 0.f;
  for (uint32_t m = m0; m < m1; ++m) {
    float v[8], q = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = 0.f;
#pragma unroll
    for (int i = 0; i < CH; ++i) {
      win[i][W - 1] = cur[i];
      cur[i] = m + 1 < m1 && lane + 32 * i < (int)d ? a.proj[(size_t)(m + 1) * a.ld_proj + c0 + 32 * i] : 0.f;  // the next row travels meanwhile
      float y = 0.f;
#pragma unroll
      for (int j = 0; j < W; ++j) y = fmaf(cw[i][j], win[i][j], y);
#pragma unroll
      for (int j = 0; j + 1 < W; ++j) win[i][j] = win[i][j + 1];
      v[i] = lane + 32 * i < (int)d ? y : 0.f;
      q = fmaf(v[i], v[i], q);
    }
    if (!is_v) {
      const float inv = 1.f / sqrtf(warp_sum(q) / (float)d + a.eps);
#pragma unroll
      for (int i = 0; i < CH; ++i) v[i] *= inv;
    }
    if (u < a.heads) {
      float *dst = q_out + ((size_t)m * a.heads + u) * d8;
#pragma unroll
      for (int i = 0; i < CH; ++i)
        if (lane + 32 * i < (int)d8) dst[lane + 32 * i] = v[i];
    } else {
      store_cache<CT>(a, slot, w.rows.pos0 + m, is_v ? u - HK : u - a.heads, is_v, lane, v);
    }
  }
}
// Any number of taps: one warp per (row, head unit).
template <typename CT>
__global__ void __launch_bounds__(256) conv_norm_any_kernel(const __grid_constant__ WinArgs w, float *__restrict__ q_out) {
  pdl_launch_dependents();
  pdl_wait();
  const greta_window_attn &a = w.a;
  const uint32_t u = blockIdx.x * 8 + (threadIdx.x >> 5), m = blockIdx.y, p = w.rows.pos0 + m;
  const int lane = threadIdx.x & 31;
  const uint32_t HK = a.heads + a.kv_heads;
  if (u >= HK + a.kv_heads) return;
  float v[8];
  conv_head(a, m, w.rows.slot0, p, w.rows.pos0, unit_col(a, u), u < HK ? a.dim : a.vdim, u < HK, lane, v);
  if (u < a.heads) {
    const uint32_t d8 = up8(a.dim);
    float *q = q_out + ((size_t)m * a.heads + u) * d8;
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (lane + 32 * i < d8) q[lane + 32 * i] = v[i];
  } else {
    const bool is_v = u >= HK;
    store_cache<CT>(a, w.rows.slot0, p, is_v ? u - HK : u - a.heads, is_v, lane, v);
  }
}
__global__ void conv_history_kernel(const __grid_constant__ WinArgs w) {
  pdl_launch_dependents();
  pdl_wait();
  const greta_window_attn &a = w.a;
  const uint32_t C = (a.heads + a.kv_heads) * a.dim + a.kv_heads * a.vdim, c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= C) return;
  const uint32_t m = w.rows.M - 1 - blockIdx.y, p = w.rows.pos0 + m;  // grid.y <= min(M, taps): distinct history rows
  a.history[((size_t)w.rows.slot0 * a.taps + p % a.taps) * C + c] = a.proj[(size_t)m * a.ld_proj + c];
}

__device__ __forceinline__ float score(const greta_window_attn &a, uint32_t h, float dot, uint32_t dist) {
  float s = dot * a.scale;
  if (a.temp) s *= a.temp[h];
  if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
  if (a.r1) s -= a.r1[h] * log1pf(a.r2[h] * (float)dist);
  return s;
}

constexpr int WR_KEYS = 256, WR_THREADS = 256, KPG = 4;  // keys of a pass; keys that a group of eight lanes has in flight

// grid (splits, kv heads * head passes, rows), cluster (splits, 1, 1); HN query heads of one key/value head per CTA.
template <typename CT, int HN, bool FUSED>
__global__ void __launch_bounds__(WR_THREADS) window_rows_kernel(const __grid_constant__ WinArgs w, const float *__restrict__ q_in, void *out, int out_fmt,
                                                                 uint32_t ld_out) {
  const greta_window_attn &a = w.a;
  extern __shared__ __align__(16) float smem[];
  const uint32_t d8 = up8(a.dim), v8 = up8(a.vdim), HG = a.heads / a.kv_heads, passes = (HG + HN - 1) / HN;
  const uint32_t quads = v8 / 4, tpp = (quads + 31) / 32 * 32, KG = WR_THREADS / tpp;
  float *sq = smem;                          // [HN][d8]
  float *sp = sq + HN * d8;                  // [HN][WR_KEYS] scores, then weights
  float *so = sp + HN * WR_KEYS;             // [HN][v8] this CTA's unnormalised output
  float *sx = so + HN * v8;                  // [KG][HN][v8] reduction over key groups
  float *sm = sx + (size_t)KG * HN * v8;     // [HN] running maximum
  float *sl = sm + HN, *sf = sl + HN;        // [HN] running sum, rescale factor
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t g = blockIdx.y / passes, h0 = g * HG + (blockIdx.y % passes) * HN, hn = min((uint32_t)HN, (g + 1) * HG - h0);
  const uint32_t m = blockIdx.z, split = blockIdx.x, S = gridDim.x;
  pdl_launch_dependents();
  pdl_wait();
  const uint32_t slot = w.rows.d_pos ? w.rows.slot0 + m : w.rows.slot0, i = w.rows.d_pos ? w.rows.d_pos[m] : w.rows.pos0 + m;
  const KeyList keys(a, i, i);
  const uint32_t total = keys.total, per = (total + S - 1) / S, t_begin = min(total, split * per), t_end = min(total, t_begin + per);
  const uint32_t rows = a.keep_first + a.ring;
  const CT *kc = static_cast<const CT *>(a.k_cache) + ((size_t)slot * a.kv_heads + g) * rows * d8;
  const CT *vc = static_cast<const CT *>(a.v_cache) + ((size_t)slot * a.kv_heads + g) * rows * v8;
  {  // this CTA's keys and values start their way to L2
    const uint32_t kl = (d8 * (uint32_t)sizeof(CT) + 127) / 128, vl = (v8 * (uint32_t)sizeof(CT) + 127) / 128;
    for (uint32_t e = threadIdx.x; e < (t_end - t_begin) * (kl + vl); e += WR_THREADS) {
      const uint32_t r = keys.row(t_begin + e / (kl + vl)), l = e % (kl + vl);
      const char *p = l < kl ? reinterpret_cast<const char *>(kc + (size_t)r * d8) + l * 128 : reinterpret_cast<const char *>(vc + (size_t)r * v8) + (l - kl) * 128;
      asm volatile("prefetch.global.L2 [%0];" ::"l"(p));
    }
  }
  if (FUSED) {
    const uint32_t C = (a.heads + a.kv_heads) * a.dim + a.kv_heads * a.vdim;
    float *hist = a.conv ? a.history + ((size_t)slot * a.taps + i % a.taps) * C : nullptr;
    const bool last = t_begin < t_end && t_end == total;
    for (uint32_t u = warp; u < HN + 2; u += WR_THREADS / 32) {
      float v[8];
      if (u < HN) {
        if (u >= hn) {
#pragma unroll
          for (int e = 0; e < 8; ++e)
            if (lane + 32 * e < d8) sq[u * d8 + lane + 32 * e] = 0.f;
          continue;
        }
        conv_head(a, m, slot, i, i, (h0 + u) * a.dim, a.dim, true, lane, v);
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const uint32_t c = lane + 32 * e;
          if (c < d8) sq[u * d8 + c] = v[e];
          if (hist && split == 0 && c < a.dim) hist[(h0 + u) * a.dim + c] = a.proj[(size_t)m * a.ld_proj + (h0 + u) * a.dim + c];
        }
      } else if (last) {
        const bool is_v = u == HN + 1;
        const uint32_t d = is_v ? a.vdim : a.dim, col = unit_col(a, a.heads + (is_v ? a.kv_heads : 0) + g);
        conv_head(a, m, slot, i, i, col, d, !is_v, lane, v);
        store_cache<CT>(a, slot, i, g, is_v, lane, v);
        if (hist)
          for (uint32_t c = lane; c < d; c += 32) hist[col + c] = a.proj[(size_t)m * a.ld_proj + col + c];
      }
    }
  } else {
    for (uint32_t e = threadIdx.x; e < HN * d8; e += WR_THREADS) {
      const uint32_t h = e / d8;
      sq[e] = h < hn ? q_in[((size_t)m * a.heads + h0 + h) * d8 + e % d8] : 0.f;
    }
  }
  if (threadIdx.x < HN) {
    sm[threadIdx.x] = -INFINITY;
    sl[threadIdx.x] = 0.f;
  }
  __syncthreads();  // also: this CTA's cache row is visible to it

  const uint32_t pr = threadIdx.x % tpp, kg = threadIdx.x / tpp;
  const bool pv = pr < quads && kg < KG;
  float acc[HN][4];
#pragma unroll
  for (int h = 0; h < HN; ++h) acc[h][0] = acc[h][1] = acc[h][2] = acc[h][3] = 0.f;
  for (uint32_t t0 = t_begin; t0 < t_end; t0 += WR_KEYS) {
    const uint32_t n = min((uint32_t)WR_KEYS, t_end - t0);
    const uint32_t l8 = threadIdx.x & 7, grp = threadIdx.x >> 3;  // 32 groups of 8 lanes, KPG keys each
    for (uint32_t part = 0; part < n; part += 32 * KPG) {
      uint32_t krow[KPG];
      float dot[KPG][HN];
#pragma unroll
      for (int e = 0; e < KPG; ++e) {
        const uint32_t t = part + grp + e * 32;
        krow[e] = keys.row(t0 + (t < n ? t : 0));
#pragma unroll
        for (int h = 0; h < HN; ++h) dot[e][h] = 0.f;
      }
      for (uint32_t c = l8 * 8; c < d8; c += 64) {
        float k[KPG][8];
#pragma unroll
        for (int e = 0; e < KPG; ++e) load8(kc + (size_t)krow[e] * d8 + c, k[e]);
#pragma unroll
        for (int h = 0; h < HN; ++h) {
          const float4 qa = *reinterpret_cast<const float4 *>(sq + h * d8 + c), qb = *reinterpret_cast<const float4 *>(sq + h * d8 + c + 4);
#pragma unroll
          for (int e = 0; e < KPG; ++e) {
            float x = dot[e][h];
            x = fmaf(k[e][0], qa.x, fmaf(k[e][1], qa.y, fmaf(k[e][2], qa.z, fmaf(k[e][3], qa.w, x))));
            dot[e][h] = fmaf(k[e][4], qb.x, fmaf(k[e][5], qb.y, fmaf(k[e][6], qb.z, fmaf(k[e][7], qb.w, x))));
          }
        }
      }
#pragma unroll
      for (int e = 0; e < KPG; ++e)
#pragma unroll
        for (int h = 0; h < HN; ++h) {
          float x = dot[e][h];
          x += __shfl_xor_sync(0xffffffffu, x, 1);
          x += __shfl_xor_sync(0xffffffffu, x, 2);
          dot[e][h] = x + __shfl_xor_sync(0xffffffffu, x, 4);
        }
      // the group's KPG * HN scores are finished by its eight lanes
#pragma unroll
      for (int r = 0; r < (KPG * HN + 7) / 8; ++r) {
        const uint32_t id = l8 + 8 * r, e = id / HN, h = id % HN;
        float mine = 0.f;
#pragma unroll
        for (int x = 0; x < KPG * HN; ++x)
          if (id == (uint32_t)x) mine = dot[x / HN][x % HN];
        const uint32_t t = part + grp + e * 32;
        if (id < (uint32_t)(KPG * HN) && h < hn) sp[h * WR_KEYS + t] = t < n ? score(a, h0 + h, mine, i - keys.position(t0 + t)) : -INFINITY;
      }
    }
    __syncthreads();
    if (warp < (int)hn) {
      float *s = sp + warp * WR_KEYS;
      const float old = sm[warp];
      float x[WR_KEYS / 32], mx = old, sum = 0.f;
#pragma unroll
      for (int e = 0; e < WR_KEYS / 32; ++e) {
        x[e] = lane + 32 * e < (int)n ? s[lane + 32 * e] : -INFINITY;
        mx = fmaxf(mx, x[e]);
      }
      mx = warp_max(mx);
      const float f = expf(old - mx);
#pragma unroll
      for (int e = 0; e < WR_KEYS / 32; ++e) {
        x[e] = expf(x[e] - mx);
        s[lane + 32 * e] = x[e];
        sum += x[e];
      }
      sum = warp_sum(sum);
      __syncwarp();
      if (lane == 0) {
        sm[warp] = mx;
        sl[warp] = sl[warp] * f + sum;
        sf[warp] = f;
      }
    }
    __syncthreads();
    if (pv) {
#pragma unroll
      for (int h = 0; h < HN; ++h)
        if (h < (int)hn)
#pragma unroll
          for (int x = 0; x < 4; ++x) acc[h][x] *= sf[h];
#pragma unroll 8
      for (uint32_t e = kg; e < n; e += KG) {
        const float4 v = load4(vc + (size_t)keys.row(t0 + e) * v8 + pr * 4);
#pragma unroll
        for (int h = 0; h < HN; ++h) {
          const float p = sp[h * WR_KEYS + e];
          if (h < (int)hn) {
            acc[h][0] = fmaf(p, v.x, acc[h][0]);
            acc[h][1] = fmaf(p, v.y, acc[h][1]);
            acc[h][2] = fmaf(p, v.z, acc[h][2]);
            acc[h][3] = fmaf(p, v.w, acc[h][3]);
          }
        }
      }
    }
    __syncthreads();
  }
  if (pv)
#pragma unroll
    for (int h = 0; h < HN; ++h)
#pragma unroll
      for (int x = 0; x < 4; ++x) sx[((size_t)kg * HN + h) * v8 + pr * 4 + x] = acc[h][x];
  __syncthreads();
  for (uint32_t e = threadIdx.x; e < hn * v8; e += WR_THREADS) {
    float t = 0.f;
    for (uint32_t k = 0; k < KG; ++k) t += sx[(size_t)k * HN * v8 + e];
    so[e] = t;
  }
  cg::cluster_group cl = cg::this_cluster();
  cl.sync();
  // the CTAs of the cluster share the merge: element e of the HN * v8 outputs goes to CTA (e / 256) % S
  for (uint32_t e = split * WR_THREADS + threadIdx.x; e < hn * v8; e += S * WR_THREADS) {
    const uint32_t h = e / v8, c = e % v8;
    if (c >= a.vdim) continue;
    float mx = a.sink ? a.sink[h0 + h] : -INFINITY;
    for (uint32_t s = 0; s < S; ++s) mx = fmaxf(mx, *cl.map_shared_rank(sm + h, s));
    float num = 0.f, den = a.sink ? expf(a.sink[h0 + h] - mx) : 0.f;
    for (uint32_t s = 0; s < S; ++s) {
      const float f = expf(*cl.map_shared_rank(sm + h, s) - mx);
      num = fmaf(f, *cl.map_shared_rank(so + e, s), num);
      den = fmaf(f, *cl.map_shared_rank(sl + h, s), den);
    }
    store_out(out, out_fmt, (size_t)m * ld_out + (size_t)(h0 + h) * a.vdim + c, num / den);
  }
  cl.sync();  // no CTA leaves while another reads its shared memory
}

// ---- prompts on the tensor cores -------------------------------------------------------------
constexpr int WM_Q = 64, WM_K = 64, WM_THREADS = 128;
template <int DB>
struct MmaCfg {
  static constexpr int ROWP = DB * 2 + 16;  // padded row: ldmatrix rows fall into different banks
  static constexpr size_t SMEM = (size_t)(WM_Q + 4 * WM_K) * ROWP;
};

// grid (query tiles, heads); DB: head size bucket (64, 128 or 256) for both dim and vdim, unused columns zero.
template <int DB>
__global__ void __launch_bounds__(WM_THREADS) window_mma_kernel(const __grid_constant__ WinArgs w, const float *__restrict__ q_in, void *out, int out_fmt,
                                                                uint32_t ld_out) {
  constexpr int ROWP = MmaCfg<DB>::ROWP;
  constexpr float LOG2E = 1.4426950408889634f;
  extern __shared__ __align__(16) uint8_t smb[];
  uint8_t *qs = smb, *kt = qs + WM_Q * ROWP, *vt = kt + 2 * WM_K * ROWP;  // two K tiles, two V tiles
  const greta_window_attn &a = w.a;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, tq = lane & 3, mat = lane >> 3, r8 = lane & 7;
  const uint32_t tile = gridDim.x - 1 - blockIdx.x, h = blockIdx.y, g = h / (a.heads / a.kv_heads);  // the longest rows first
  const uint32_t m0 = tile * WM_Q, nq = min((uint32_t)WM_Q, w.rows.M - m0), i0 = w.rows.pos0 + m0, i1 = i0 + nq - 1;
  const uint32_t d8 = up8(a.dim), v8 = up8(a.vdim), rows = a.keep_first + a.ring;
  for (uint32_t e = threadIdx.x; e < MmaCfg<DB>::SMEM / 16; e += WM_THREADS) reinterpret_cast<uint4 *>(smb)[e] = make_uint4(0, 0, 0, 0);
  pdl_launch_dependents();
  pdl_wait();
  __syncthreads();
  const __half *kc = static_cast<const __half *>(a.k_cache) + ((size_t)w.rows.slot0 * a.kv_heads + g) * rows * d8;
  const __half *vc = static_cast<const __half *>(a.v_cache) + ((size_t)w.rows.slot0 * a.kv_heads + g) * rows * v8;
  for (uint32_t e = threadIdx.x; e < nq * (d8 / 2); e += WM_THREADS) {
    const uint32_t r = e / (d8 / 2), c = e % (d8 / 2);
    const float2 q = *reinterpret_cast<const float2 *>(q_in + ((size_t)(m0 + r) * a.heads + h) * d8 + 2 * c);
    *reinterpret_cast<uint32_t *>(qs + (size_t)r * ROWP + c * 4) = half2_bits(q.x, q.y);
  }
  const KeyList keys(a, i0, i1);
  const uint32_t total = keys.total, ntiles = (total + WM_K - 1) / WM_K;
  auto stage = [&](uint32_t t, int buf) {
    if (t < ntiles) {
      const uint32_t kchunks = d8 / 8, per = kchunks + v8 / 8;
      for (uint32_t e = threadIdx.x; e < WM_K * per; e += WM_THREADS) {
        const uint32_t r = e / per, c = e % per, idx = t * WM_K + r;
        const bool on = idx < total;
        const uint32_t cr = keys.row(on ? idx : 0);
        if (c < kchunks)
          cp16z(kt + (size_t)(buf * WM_K + r) * ROWP + c * 16, kc + (size_t)cr * d8 + c * 8, on);
        else
          cp16z(vt + (size_t)(buf * WM_K + r) * ROWP + (c - kchunks) * 16, vc + (size_t)cr * v8 + (c - kchunks) * 8, on);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const float temp = a.temp ? a.temp[h] : 1.f, zs = a.scale * temp;
  const bool cap = a.softcap > 0.f;
  const float c1 = cap ? 2.f * LOG2E * zs / a.softcap : zs * LOG2E, cap2 = a.softcap * LOG2E;
  const float r1 = a.r1 ? a.r1[h] : 0.f, r2 = a.r1 ? a.r2[h] : 0.f;
  const bool bias = a.r1 != nullptr;
  const uint32_t qi[2] = {i0 + warp * 16 + gq, i0 + warp * 16 + gq + 8};
  float o[DB / 8][4], mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int n = 0; n < DB / 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[n][e] = 0.f;
  stage(0, 0);
  for (uint32_t t = 0; t < ntiles; ++t) {
    const int buf = t & 1;
    stage(t + 1, buf ^ 1);
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    float s[WM_K / 8][4];
#pragma unroll
    for (int n = 0; n < WM_K / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[n][e] = 0.f;
#pragma unroll
    for (int ks = 0; ks < DB / 16; ++ks) {
      if (ks * 16 >= (int)d8) break;
      uint32_t qa[4];
      ldsm_x4(qa, qs + (size_t)(warp * 16 + (mat & 1) * 8 + r8) * ROWP + ks * 32 + (mat >> 1) * 16);
#pragma unroll
      for (int n = 0; n < WM_K / 16; ++n) {
        uint32_t kb[4];
        ldsm_x4(kb, kt + (size_t)(buf * WM_K + n * 16 + (mat >> 1) * 8 + r8) * ROWP + ks * 32 + (mat & 1) * 16);
        mma16816(s[2 * n], qa, kb[0], kb[1]);
        mma16816(s[2 * n + 1], qa, kb[2], kb[3]);
      }
    }
    // scores in units of log2: cap tanh(z / cap) = cap - 2 cap / (1 + exp(2 z / cap))
    float tm[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int n = 0; n < WM_K / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const uint32_t idx = t * WM_K + n * 8 + 2 * tq + (e & 1), j = keys.position(idx), i = qi[e >> 1];
        float z = s[n][e] * c1;
        if (cap) z = cap2 - 2.f * cap2 * rcp(1.f + ex2(z));
        if (bias) z -= r1 * lg2(1.f + r2 * (float)(int)(i - j));
        const bool see = idx < total && j <= i && (!a.window || i - j < a.window || j < a.keep_first);
        z = see ? z : -INFINITY;
        s[n][e] = z;
        tm[e >> 1] = fmaxf(tm[e >> 1], z);
      }
    float f[2], base[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      tm[r] = fmaxf(tm[r], __shfl_xor_sync(0xffffffffu, tm[r], 1));
      tm[r] = fmaxf(tm[r], __shfl_xor_sync(0xffffffffu, tm[r], 2));
      const float nm = fmaxf(mx[r], tm[r]);
      base[r] = nm == -INFINITY ? 0.f : nm;  // a row that has seen no key yet
      f[r] = ex2(mx[r] - base[r]);
      mx[r] = nm;
      l[r] *= f[r];
    }
#pragma unroll
    for (int n = 0; n < WM_K / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s[n][e] = ex2(s[n][e] - base[e >> 1]);
        l[e >> 1] += s[n][e];
      }
#pragma unroll
    for (int n = 0; n < DB / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[n][e] *= f[e >> 1];
#pragma unroll
    for (int ks = 0; ks < WM_K / 16; ++ks) {
      const uint32_t pa[4] = {half2_bits(s[2 * ks][0], s[2 * ks][1]), half2_bits(s[2 * ks][2], s[2 * ks][3]), half2_bits(s[2 * ks + 1][0], s[2 * ks + 1][1]),
                              half2_bits(s[2 * ks + 1][2], s[2 * ks + 1][3])};
#pragma unroll
      for (int n = 0; n < DB / 16; ++n) {
        if (n * 16 >= (int)v8) break;
        uint32_t vb[4];
        ldsm_x4_trans(vb, vt + (size_t)(buf * WM_K + ks * 16 + (mat & 1) * 8 + r8) * ROWP + n * 32 + (mat >> 1) * 16);
        mma16816(o[2 * n], pa, vb[0], vb[1]);
        mma16816(o[2 * n + 1], pa, vb[2], vb[3]);
      }
    }
    __syncthreads();  // the tile may be overwritten
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  const float sink2 = a.sink ? a.sink[h] * LOG2E : -INFINITY;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    const float nm = fmaxf(mx[r], sink2), f = ex2(mx[r] - nm), inv = f / (l[r] * f + ex2(sink2 - nm));
    const uint32_t row = warp * 16 + gq + 8 * r;
    if (row < nq) {
#pragma unroll
      for (int n = 0; n < DB / 8; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const uint32_t c = n * 8 + 2 * tq + e;
          if (c < a.vdim) store_out(out, out_fmt, (size_t)(m0 + row) * ld_out + (size_t)h * a.vdim + c, o[n][2 * r + e] * inv);
        }
    }
  }
}

int check_win(const char *what, const greta_window_attn *a, const greta_rows *r) {
  GRETA_REQUIRE(a && r && r->M, "%s: null or empty argument", what);
  GRETA_REQUIRE(a->heads && a->kv_heads && a->heads % a->kv_heads == 0, "%s: %u query heads over %u key/value heads", what, a->heads, a->kv_heads);
  GRETA_REQUIRE(a->dim && a->dim <= 256 && a->vdim && a->vdim <= 256, "%s: head sizes %u / %u (1..256)", what, a->dim, a->vdim);
  GRETA_REQUIRE(a->ring && a->k_cache && a->v_cache && aligned16(a->k_cache) && aligned16(a->v_cache), "%s: no cache", what);
  GRETA_REQUIRE(a->cache_fmt == GRETA_FMT_F16 || a->cache_fmt == GRETA_FMT_F32, "%s: cache format %d", what, a->cache_fmt);
  GRETA_REQUIRE(!a->conv || (a->taps && a->history), "%s: a convolution without taps or history", what);
  GRETA_REQUIRE(!a->r1 == !a->r2, "%s: r1 and r2 come together", what);
  return GRETA_OK;
}

template <typename CT, int TAPS>
int launch_conv_taps(cudaStream_t s, const WinArgs &w, float *q) {
  const uint32_t d = std::max(w.a.dim, w.a.vdim);
  const dim3 grid((w.a.heads + 2 * w.a.kv_heads + 7) / 8, (w.rows.M + CV_ROWS - 1) / CV_ROWS);
  if (d <= 64)
    GRETA_CUDA_TRY(launch_pdl(conv_norm_kernel<CT, TAPS, 2>, grid, dim3(256), 0, s, w, q));
  else if (d <= 128)
    GRETA_CUDA_TRY(launch_pdl(conv_norm_kernel<CT, TAPS, 4>, grid, dim3(256), 0, s, w, q));
  else
    GRETA_CUDA_TRY(launch_pdl(conv_norm_kernel<CT, TAPS, 8>, grid, dim3(256), 0, s, w, q));
  return launched("conv_norm_kernel");
}
template <typename CT>
int launch_conv(cudaStream_t s, const WinArgs &w, float *q) {
  switch (w.a.conv ? w.a.taps : 0) {
    case 0: return launch_conv_taps<CT, 0>(s, w, q);
    case 1: return launch_conv_taps<CT, 1>(s, w, q);
    case 2: return launch_conv_taps<CT, 2>(s, w, q);
    case 3: return launch_conv_taps<CT, 3>(s, w, q);
    case 4: return launch_conv_taps<CT, 4>(s, w, q);
    default: break;
  }
  GRETA_CUDA_TRY(launch_pdl(conv_norm_any_kernel<CT>, dim3((w.a.heads + 2 * w.a.kv_heads + 7) / 8, w.rows.M), dim3(256), 0, s, w, q));
  return launched("conv_norm_any_kernel");
}

template <typename CT, int HN, bool FUSED>
int launch_rows(cudaStream_t s, const WinArgs &w, const float *q, void *out, int out_fmt, uint32_t ld_out, uint32_t splits) {
  const greta_window_attn &a = w.a;
  const uint32_t d8 = up8(a.dim), v8 = up8(a.vdim), tpp = (v8 / 4 + 31) / 32 * 32, KG = WR_THREADS / tpp;
  const size_t smem = ((size_t)HN * (d8 + WR_KEYS + v8 + (size_t)KG * v8) + 3 * HN) * 4;
  static bool attr_set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !attr_set[dev]) {
    GRETA_CUDA_TRY(cudaFuncSetAttribute(window_rows_kernel<CT, HN, FUSED>, cudaFuncAttributeMaxDynamicSharedMemorySize, 65536));
    attr_set[dev] = true;
  }
  const uint32_t HG = a.heads / a.kv_heads, passes = (HG + HN - 1) / HN;
  GRETA_REQUIRE(a.kv_heads * passes <= 65535 && w.rows.M <= 65535, "window_attn: grid too large");
  GRETA_CUDA_TRY(launch_pdl_cluster(window_rows_kernel<CT, HN, FUSED>, dim3(splits, a.kv_heads * passes, w.rows.M), dim3(WR_THREADS), splits, smem, s, w, q,
                                    out, out_fmt, ld_out));
  return launched("window_rows_kernel");
}
template <typename CT, bool FUSED>
int pick_heads(cudaStream_t s, const WinArgs &w, const float *q, void *out, int out_fmt, uint32_t ld_out, uint32_t splits) {
  // heads per CTA: all that share a key/value head, fewer where the grid would leave SMs idle
  uint32_t HG = w.a.heads / w.a.kv_heads;
  while (HG > 1 && (uint64_t)w.rows.M * w.a.kv_heads * splits * ((w.a.heads / w.a.kv_heads + HG / 2 - 1) / (HG / 2)) <= 160) HG /= 2;
  if (HG == 1) return launch_rows<CT, 1, FUSED>(s, w, q, out, out_fmt, ld_out, splits);
  if (HG == 2) return launch_rows<CT, 2, FUSED>(s, w, q, out, out_fmt, ld_out, splits);
  if (HG <= 4) return launch_rows<CT, 4, FUSED>(s, w, q, out, out_fmt, ld_out, splits);
  return launch_rows<CT, 8, FUSED>(s, w, q, out, out_fmt, ld_out, splits);
}
template <int DB>
int launch_mma(cudaStream_t s, const WinArgs &w, const float *q, void *out, int out_fmt, uint32_t ld_out) {
  static bool attr_set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !attr_set[dev]) {
    GRETA_CUDA_TRY(cudaFuncSetAttribute(window_mma_kernel<DB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MmaCfg<DB>::SMEM));
    attr_set[dev] = true;
  }
  GRETA_CUDA_TRY(launch_pdl(window_mma_kernel<DB>, dim3((w.rows.M + WM_Q - 1) / WM_Q, w.a.heads), dim3(WM_THREADS), MmaCfg<DB>::SMEM, s, w, q, out, out_fmt,
                            ld_out));
  return launched("window_mma_kernel");
}

}  // namespace

extern "C" {

int greta_cuda_window_attn_prepare(greta_stream_t stream, const greta_window_attn *a, const greta_rows *rows, float *q_out) {
  if (int rc = check_win("window_attn_prepare", a, rows)) return rc;
  GRETA_REQUIRE(!rows->d_pos && q_out && a->proj && rows->M <= 65535, "window_attn_prepare: null pointer, or rows of a batch");
  GRETA_REQUIRE(!a->window || a->ring >= a->window - 1 + rows->M || rows->pos0 + rows->M <= a->keep_first + a->ring,
                "window_attn_prepare: a portion of %u rows does not fit a ring of %u rows behind a window of %u", rows->M, a->ring, a->window);
  const WinArgs w{*a, *rows};
  cudaStream_t s = (cudaStream_t)stream;
  if (int rc = a->cache_fmt == GRETA_FMT_F16 ? launch_conv<__half>(s, w, q_out) : launch_conv<float>(s, w, q_out)) return rc;
  if (!a->conv) return GRETA_OK;
  const uint32_t C = (a->heads + a->kv_heads) * a->dim + a->kv_heads * a->vdim;
  GRETA_CUDA_TRY(launch_pdl(conv_history_kernel, dim3((C + 255) / 256, std::min(rows->M, a->taps)), dim3(256), 0, s, w));
  return launched("conv_history_kernel");
}

int greta_cuda_window_attn(greta_stream_t stream, const greta_window_attn *a, const greta_rows *rows, const float *q, void *out, int out_fmt,
                           uint32_t ld_out, uint32_t max_len) {
  if (int rc = check_win("window_attn", a, rows)) return rc;
  GRETA_REQUIRE(out && max_len && (q || (rows->d_pos && a->proj)), "window_attn: null pointer");
  const WinArgs w{*a, *rows};
  cudaStream_t s = (cudaStream_t)stream;
  // CTAs per row: enough to fill the GPU, at least 64 keys each, at most a portable cluster
  const uint32_t keys = a->window ? std::min(max_len, a->keep_first + a->window) : max_len;
  uint32_t splits = 1;
  while (splits < 8 && (uint64_t)rows->M * a->kv_heads * splits < 148 && keys > splits * 64) splits *= 2;
  if (a->cache_fmt == GRETA_FMT_F16)
    return q ? pick_heads<__half, false>(s, w, q, out, out_fmt, ld_out, splits) : pick_heads<__half, true>(s, w, q, out, out_fmt, ld_out, splits);
  return q ? pick_heads<float, false>(s, w, q, out, out_fmt, ld_out, splits) : pick_heads<float, true>(s, w, q, out, out_fmt, ld_out, splits);
}

int greta_cuda_window_attn_prefill(greta_stream_t stream, const greta_window_attn *a, const greta_rows *rows, const float *q, void *out, int out_fmt,
                                   uint32_t ld_out) {
  if (int rc = check_win("window_attn_prefill", a, rows)) return rc;
  GRETA_REQUIRE(!rows->d_pos && q && out && a->heads <= 65535, "window_attn_prefill: null pointer, or rows of a batch");
  GRETA_REQUIRE(a->cache_fmt == GRETA_FMT_F16, "window_attn_prefill: the cache must be F16");
  const WinArgs w{*a, *rows};
  cudaStream_t s = (cudaStream_t)stream;
  const uint32_t d = std::max(a->dim, a->vdim);
  if (d <= 64) return launch_mma<64>(s, w, q, out, out_fmt, ld_out);
  if (d <= 128) return launch_mma<128>(s, w, q, out, out_fmt, ld_out);
  return launch_mma<256>(s, w, q, out, out_fmt, ld_out);
}

}  // extern "C"
