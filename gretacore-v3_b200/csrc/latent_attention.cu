// Latent attention: every head's keys and values are linear images of one cached latent per token, plus one rotated key part
// that all heads share.
//   latent_prepare_kernel   portions: norm of the latent, rotation of the shared key part, cache row; for the expanded form also the
//                           rotated and scaled queries in fp16
//   absorbed form (decode, short portions; 32-bit models always)
//     latent_query_kernel   q W_uk per head and the rotated q, so that a score is one dot product with a cache row; the new
//                           tokens' cache rows are written beside it
//     latent_mma_kernel     one row's heads as the 16-row operand of mma.sync (fp16), the cached latents as keys and as values,
//                           the keys split over CTAs; partial sums, maxima and normalisers to scratch
//     latent_rows_kernel    the same in 32-bit on the CUDA cores
//     latent_value_kernel   merges the splits (with the sink), applies W_uv per head and the output gate
//   expanded form (prompts)
//     latent_prefill_kernel keys and values of all heads lie in a workspace (a dense product of the cached latents), the rotated key
//                           part is read from the cache; 128 query positions of a head per CTA on tcgen05: scores and outputs in
//                           TMEM, the softmax weights go back to TMEM as the second product's operand
// Scores, weights, sums and angles are fp32 throughout.
#include <algorithm>

#include "dense_device.cuh"
#include "mma_device.cuh"
#include "tc_device.cuh"

using namespace greta;

namespace {

__host__ __device__ constexpr uint32_t up8(uint32_t d) { return (d + 7u) & ~7u; }
__host__ __device__ constexpr uint32_t up16(uint32_t d) { return (d + 15u) & ~15u; }
constexpr float LOG2E = 1.4426950408889634f;
constexpr uint32_t MAX_RANK = 1024, MAX_ROT = 128, MAX_DIM = 256, MAX_SPLITS = 64;

struct LatArgs {
  greta_latent_attn a;
  greta_rows rows;
};
struct Where {
  uint32_t slot, pos;
};
__device__ __forceinline__ Where where(const greta_rows &r, uint32_t m) {
  return r.d_pos ? Where{r.slot0 + m, r.d_pos[m]} : Where{r.slot0, r.pos0 + m};
}
template <typename CT>
__device__ __forceinline__ CT to_cache(float v);
template <>
__device__ __forceinline__ float to_cache<float>(float v) { return v; }
template <>
__device__ __forceinline__ __half to_cache<__half>(float v) { return __float2half_rn(v); }

// Channel c of the rotated vector x at a position.
__device__ __forceinline__ float rotated(const greta_latent_attn &a, const float *x, uint32_t pos, uint32_t c) {
  const float own = x[c];
  if (c >= a.rot_dims) return own;
  const uint32_t half = a.rot_dims / 2;
  const uint32_t i = a.interleaved ? c >> 1 : c % half;
  const bool second = a.interleaved ? c & 1 : c >= half;
  const float other = x[a.interleaved ? c ^ 1 : second ? c - half : c + half];
  const float2 cs = __ldg(reinterpret_cast<const float2 *>(a.rotation) + (size_t)min(pos, a.positions - 1) * half + i);
  return second ? fmaf(own, cs.x, other * cs.y) : fmaf(own, cs.x, -other * cs.y);
}

// One warp: the cache row of activation row m.
template <typename CT>
__device__ __forceinline__ void write_cache_row(const greta_latent_attn &a, const greta_rows &rows, uint32_t m, int lane) {
  const Where at = where(rows, m);
  const float *x = a.down + (size_t)m * a.ld_down;
  const uint32_t R16 = up16(a.rank), P16 = up16(a.rot_dim);
  if (at.pos >= a.cap) return;
  CT *row = static_cast<CT *>(a.cache) + ((size_t)at.slot * a.cap + at.pos) * (R16 + P16);
  float q = 0.f;
  for (uint32_t c = lane; c < a.rank; c += 32) q = fmaf(x[c], x[c], q);
  const float inv = 1.f / sqrtf(warp_sum(q) / (float)a.rank + a.eps);
  for (uint32_t c = lane; c < R16; c += 32) row[c] = to_cache<CT>(c < a.rank ? x[c] * inv * __ldg(a.latent_norm + c) : 0.f);
  for (uint32_t c = lane; c < P16; c += 32) row[R16 + c] = to_cache<CT>(c < a.rot_dim ? rotated(a, x + a.rank, at.pos, c) : 0.f);
}
__host__ __device__ constexpr uint32_t slabs(uint32_t cols) { return (cols + 63) / 64; }  // column groups of a 128-byte swizzled tile
// One CTA per row: the last warp writes the cache row, the others the queries (q_out NULL: none) as [head][dim64 | rot64], in powers of
// two and zero past the head's channels.
template <typename CT>
__global__ void __launch_bounds__(256) latent_prepare_kernel(const __grid_constant__ LatArgs w, __half *__restrict__ q_out) {
  pdl_launch_dependents();
  pdl_wait();
  const greta_latent_attn &a = w.a;
  const uint32_t m = blockIdx.x;
  if (threadIdx.x >= 224) {
    write_cache_row<CT>(a, w.rows, m, threadIdx.x & 31);
    return;
  }
  if (!q_out) return;
  const uint32_t d64 = slabs(a.dim) * 64, width = d64 + slabs(a.rot_dim) * 64, pos = where(w.rows, m).pos;
  const float scale = a.scale * LOG2E;
  const float *q = a.q + (size_t)m * a.ld_q;
  for (uint32_t e = threadIdx.x; e < a.heads * width / 2; e += 224) {
    const uint32_t h = e / (width / 2), c = (e % (width / 2)) * 2;
    const float *x = q + (size_t)h * (a.dim + a.rot_dim);
    float v[2];
#pragma unroll
    for (int y = 0; y < 2; ++y) {
      const uint32_t col = c + y;
      v[y] = col < d64 ? (col < a.dim ? x[col] : 0.f) : (col - d64 < a.rot_dim ? rotated(a, x + a.dim, pos, col - d64) : 0.f);
    }
    *reinterpret_cast<uint32_t *>(q_out + (size_t)m * a.heads * width + 2 * (size_t)e) = half2_bits(v[0] * scale, v[1] * scale);
  }
}

// Eight consecutive weights as floats.
__device__ __forceinline__ void weights8(const __half *p, float (&f)[8]) {
  const uint4 u = ld_stream(p);
  const float2 a = h2_to_f2(u.x), b = h2_to_f2(u.y), c = h2_to_f2(u.z), d = h2_to_f2(u.w);
  f[0] = a.x, f[1] = a.y, f[2] = b.x, f[3] = b.y, f[4] = c.x, f[5] = c.y, f[6] = d.x, f[7] = d.y;
}
__device__ __forceinline__ void weights8(const float *p, float (&f)[8]) {
  const uint4 u = ld_stream(p), v = ld_stream(p + 4);
  f[0] = __uint_as_float(u.x), f[1] = __uint_as_float(u.y), f[2] = __uint_as_float(u.z), f[3] = __uint_as_float(u.w);
  f[4] = __uint_as_float(v.x), f[5] = __uint_as_float(v.y), f[6] = __uint_as_float(v.z), f[7] = __uint_as_float(v.w);
}

// grid (column tiles + 1, heads, row tiles): 128 latent columns of q W_uk for MT rows of one head.  Sixteen groups of sixteen threads
// share the head's channels; a thread holds eight columns.  The extra column tile of head 0 writes the rows' cache entries.
// q_out [M][heads][rank16 | rot16], times scale (and log2 e in the fp16 form, whose softmax works in powers of two).
constexpr uint32_t LQ_COLS = 128;
template <typename CT, int MT>
__global__ void __launch_bounds__(256) latent_query_kernel(const __grid_constant__ LatArgs w, CT *__restrict__ q_out) {
  const greta_latent_attn &a = w.a;
  __shared__ float qs[MT][MAX_DIM];
  __shared__ float red[16][MT][LQ_COLS];
  const uint32_t h = blockIdx.y, m0 = blockIdx.z * MT, R16 = up16(a.rank), P16 = up16(a.rot_dim), tiles = gridDim.x - 1;
  const uint32_t cg = threadIdx.x & 15, dg = threadIdx.x >> 4, col = blockIdx.x * LQ_COLS + cg * 8;
  const CT *wk = static_cast<const CT *>(a.w_kv) + (size_t)h * up8(a.dim) * a.ld_w;
  if (blockIdx.x < tiles && col < a.ld_w)
    for (uint32_t d = dg; d < a.dim; d += 16) asm volatile("prefetch.global.L2 [%0];" ::"l"(wk + (size_t)d * a.ld_w + col));
  pdl_launch_dependents();
  pdl_wait();
  if (blockIdx.x == tiles) {
    const uint32_t m = m0 + (threadIdx.x >> 5);
    if (h == 0 && (threadIdx.x >> 5) < MT && m < w.rows.M) write_cache_row<CT>(a, w.rows, m, threadIdx.x & 31);
    return;
  }
  const float scale = a.scale * (sizeof(CT) == 2 ? LOG2E : 1.f);
  for (uint32_t e = threadIdx.x; e < MT * a.dim; e += 256) {
    const uint32_t t = e / a.dim, d = e % a.dim;
    qs[t][d] = m0 + t < w.rows.M ? a.q[(size_t)(m0 + t) * a.ld_q + (size_t)h * (a.dim + a.rot_dim) + d] * scale : 0.f;
  }
  if (blockIdx.x == 0)
    for (uint32_t e = threadIdx.x; e < MT * P16; e += 256) {
      const uint32_t t = e / P16, c = e % P16, m = m0 + t;
      if (m >= w.rows.M) continue;
      const float *x = a.q + (size_t)m * a.ld_q + (size_t)h * (a.dim + a.rot_dim) + a.dim;
      q_out[((size_t)m * a.heads + h) * (R16 + P16) + R16 + c] = to_cache<CT>(c < a.rot_dim ? rotated(a, x, where(w.rows, m).pos, c) * scale : 0.f);
    }
  __syncthreads();
  float acc[MT][8];
#pragma unroll
  for (int t = 0; t < MT; ++t)
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[t][e] = 0.f;
  if (col < a.ld_w) {
#pragma unroll 4
    for (uint32_t d = dg; d < a.dim; d += 16) {
      float f[8];
      weights8(wk + (size_t)d * a.ld_w + col, f);
#pragma unroll
      for (int t = 0; t < MT; ++t)
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[t][e] = fmaf(qs[t][d], f[e], acc[t][e]);
    }
  }
#pragma unroll
  for (int t = 0; t < MT; ++t)
#pragma unroll
    for (int e = 0; e < 8; ++e) red[dg][t][cg * 8 + e] = acc[t][e];
  __syncthreads();
  for (uint32_t e = threadIdx.x; e < MT * LQ_COLS; e += 256) {
    const uint32_t t = e / LQ_COLS, c = e % LQ_COLS, r = blockIdx.x * LQ_COLS + c, m = m0 + t;
    if (m >= w.rows.M || r >= R16) continue;
    float s = 0.f;
#pragma unroll
    for (int g = 0; g < 16; ++g) s += red[g][t][c];
    q_out[((size_t)m * a.heads + h) * (R16 + P16) + r] = to_cache<CT>(r < a.rank ? s : 0.f);
  }
}

// Keys [begin, end) of a split: whole tiles of 64 where there is a choice.
__device__ __forceinline__ void split_keys(uint32_t total, uint32_t split, uint32_t S, uint32_t *begin, uint32_t *end) {
  const uint32_t per = ((total + S - 1) / S + 63) / 64 * 64;
  *begin = min(total, split * per);
  *end = min(total, *begin + per);
}
// Scratch of the absorbed form behind q: partial sums [M][heads][S][rank16], then {maximum, normaliser} [M][heads][S][2].
struct Parts {
  float *o, *ml;
};

constexpr int LM_K = 64, LM_THREADS = 256;
// grid (splits, groups of 16 HT heads, rows); NT: 16-column tiles of the latent per warp (8 warps).
template <int HT, int NT>
__global__ void __launch_bounds__(LM_THREADS) latent_mma_kernel(const __grid_constant__ LatArgs w, const __half *__restrict__ q_in, Parts parts, int buffers) {
  constexpr int HR = 16 * HT, PB = LM_K * 2 + 16;
  const greta_latent_attn &a = w.a;
  extern __shared__ __align__(16) uint8_t smb[];
  const uint32_t R16 = up16(a.rank), LD = R16 + up16(a.rot_dim), ROWB = LD * 2 + 16, S = gridDim.x, split = blockIdx.x;
  uint8_t *qs = smb, *ps = qs + HR * ROWB, *kt = ps + HR * PB;
  float *wmax = reinterpret_cast<float *>(kt + (size_t)buffers * LM_K * ROWB);  // [8][HR]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, tq = lane & 3, mat = lane >> 3, r8 = lane & 7;
  const uint32_t h0 = blockIdx.y * HR, hn = min((uint32_t)HR, a.heads - h0), m = blockIdx.z;
  pdl_launch_dependents();
  pdl_wait();
  const Where at = where(w.rows, m);
  uint32_t t_begin, t_end;
  split_keys(min(at.pos + 1, a.cap), split, S, &t_begin, &t_end);
  if (t_begin >= t_end) {
    for (uint32_t h = threadIdx.x; h < hn; h += LM_THREADS) {
      float *ml = parts.ml + (((size_t)m * a.heads + h0 + h) * S + split) * 2;
      ml[0] = -INFINITY, ml[1] = 0.f;
    }
    return;
  }
  const __half *cache = static_cast<const __half *>(a.cache) + (size_t)at.slot * a.cap * LD;
  const uint32_t chunks = LD / 8, ntiles = (t_end - t_begin + LM_K - 1) / LM_K;
  auto stage = [&](uint32_t t) {
    if (t < ntiles) {
      uint8_t *dst = kt + (size_t)(buffers == 2 ? t & 1 : 0) * LM_K * ROWB;
      for (uint32_t e = threadIdx.x; e < LM_K * chunks; e += LM_THREADS) {
        const uint32_t r = e / chunks, c = e % chunks, key = t_begin + t * LM_K + r;
        const bool on = key < t_end;
        cp16z(dst + (size_t)r * ROWB + c * 16, cache + (size_t)(on ? key : t_begin) * LD + c * 8, on);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  for (uint32_t e = threadIdx.x; e < HR * chunks; e += LM_THREADS) {
    const uint32_t r = e / chunks, c = e % chunks;
    cp16z(qs + (size_t)r * ROWB + c * 16, q_in + ((size_t)m * a.heads + h0 + (r < hn ? r : 0)) * LD + c * 8, r < hn);
  }
  stage(0);
  float o[HT][NT][2][4], mx[HT][2], l[HT][2];
#pragma unroll
  for (int x = 0; x < HT; ++x) {
    mx[x][0] = mx[x][1] = -INFINITY, l[x][0] = l[x][1] = 0.f;
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[x][j][n][e] = 0.f;
  }
  for (uint32_t t = 0; t < ntiles; ++t) {
    if (buffers == 2) {
      stage(t + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      if (t) stage(t);
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const uint8_t *kb = kt + (size_t)(buffers == 2 ? t & 1 : 0) * LM_K * ROWB;
    // scores of this warp's eight keys; two accumulators halve the chain of dependent products
    float s[HT][2][4];
#pragma unroll
    for (int x = 0; x < HT; ++x)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[x][n][e] = 0.f;
    auto dot = [&](uint32_t ks, int n) {
      uint32_t b[2];
      ldsm_x2(b, kb + (size_t)(warp * 8 + r8) * ROWB + ks * 32 + (mat & 1) * 16);
#pragma unroll
      for (int x = 0; x < HT; ++x) {
        uint32_t qa[4];
        ldsm_x4(qa, qs + (size_t)(x * 16 + (mat & 1) * 8 + r8) * ROWB + ks * 32 + (mat >> 1) * 16);
        mma16816(s[x][n], qa, b[0], b[1]);
      }
    };
    uint32_t ks = 0;
#pragma unroll 2
    for (; ks + 2 <= LD / 16; ks += 2) {
      dot(ks, 0);
      dot(ks + 1, 1);
    }
    if (ks < LD / 16) dot(ks, 0);
    const uint32_t key = t_begin + t * LM_K + warp * 8 + 2 * tq;
#pragma unroll
    for (int x = 0; x < HT; ++x) {
      float tm[2];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s[x][0][e] += s[x][1][e];
        if (key + (e & 1) >= t_end) s[x][0][e] = -INFINITY;
      }
      tm[0] = fmaxf(s[x][0][0], s[x][0][1]), tm[1] = fmaxf(s[x][0][2], s[x][0][3]);
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        tm[r] = fmaxf(tm[r], __shfl_xor_sync(0xffffffffu, tm[r], 1));
        tm[r] = fmaxf(tm[r], __shfl_xor_sync(0xffffffffu, tm[r], 2));
        if (tq == 0) wmax[warp * HR + x * 16 + gq + 8 * r] = tm[r];
      }
    }
    __syncthreads();
#pragma unroll
    for (int x = 0; x < HT; ++x)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const uint32_t row = x * 16 + gq + 8 * r;
        float nm = mx[x][r];
#pragma unroll
        for (int v = 0; v < 8; ++v) nm = fmaxf(nm, wmax[v * HR + row]);  // finite: a tile holds at least one key
        const float f = ex2(mx[x][r] - nm), p0 = ex2(s[x][0][2 * r] - nm), p1 = ex2(s[x][0][2 * r + 1] - nm);
        mx[x][r] = nm;
        l[x][r] = fmaf(l[x][r], f, p0 + p1);
        *reinterpret_cast<uint32_t *>(ps + (size_t)row * PB + (warp * 8 + 2 * tq) * 2) = half2_bits(p0, p1);
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            o[x][j][n][2 * r] *= f;
            o[x][j][n][2 * r + 1] *= f;
          }
      }
    __syncthreads();
#pragma unroll
    for (int k16 = 0; k16 < LM_K / 16; ++k16) {
      uint32_t pa[HT][4];
#pragma unroll
      for (int x = 0; x < HT; ++x) ldsm_x4(pa[x], ps + (size_t)(x * 16 + (mat & 1) * 8 + r8) * PB + k16 * 32 + (mat >> 1) * 16);
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        const uint32_t tile = warp + 8 * j;
        if (tile * 16 >= R16) break;
        uint32_t vb[4];
        ldsm_x4_trans(vb, kb + (size_t)(k16 * 16 + (mat & 1) * 8 + r8) * ROWB + tile * 32 + (mat >> 1) * 16);
#pragma unroll
        for (int x = 0; x < HT; ++x) {
          mma16816(o[x][j][0], pa[x], vb[0], vb[1]);
          mma16816(o[x][j][1], pa[x], vb[2], vb[3]);
        }
      }
    }
    __syncthreads();  // the tile, the weights and the maxima may be overwritten
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int x = 0; x < HT; ++x)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float t = l[x][r];
      t += __shfl_xor_sync(0xffffffffu, t, 1);
      t += __shfl_xor_sync(0xffffffffu, t, 2);
      const uint32_t row = x * 16 + gq + 8 * r;
      if (tq == 0) wmax[warp * HR + row] = t;
      if (row >= hn) continue;
      float *dst = parts.o + (((size_t)m * a.heads + h0 + row) * S + split) * R16;
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        const uint32_t tile = warp + 8 * j;
        if (tile * 16 >= R16) break;
#pragma unroll
        for (int n = 0; n < 2; ++n)
          *reinterpret_cast<float2 *>(dst + tile * 16 + n * 8 + 2 * tq) = make_float2(o[x][j][n][2 * r], o[x][j][n][2 * r + 1]);
      }
    }
  __syncthreads();
  if (warp == 0 && tq == 0) {
#pragma unroll
    for (int x = 0; x < HT; ++x)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const uint32_t row = x * 16 + gq + 8 * r;
        if (row >= hn) continue;
        float t = 0.f;
        for (int v = 0; v < 8; ++v) t += wmax[v * HR + row];
        float *ml = parts.ml + (((size_t)m * a.heads + h0 + row) * S + split) * 2;
        ml[0] = mx[x][r], ml[1] = t;
      }
  }
}

// 32-bit form: grid (splits, groups of HN heads, rows).  Eight lanes per key for the scores, four columns per thread for the sums.
constexpr int LR_KEYS = 128, LR_THREADS = 256;
template <int HN>
__global__ void __launch_bounds__(LR_THREADS) latent_rows_kernel(const __grid_constant__ LatArgs w, const float *__restrict__ q_in, Parts parts) {
  const greta_latent_attn &a = w.a;
  extern __shared__ __align__(16) float smf[];
  __shared__ float sm[HN], sl[HN], sf[HN];
  const uint32_t R16 = up16(a.rank), LD = R16 + up16(a.rot_dim), S = gridDim.x, split = blockIdx.x, h0 = blockIdx.y * HN, m = blockIdx.z;
  const uint32_t hn = min((uint32_t)HN, a.heads - h0), quads = R16 / 4, tpp = (quads + 31) / 32 * 32, KG = LR_THREADS / tpp;
  float *sq = smf, *sp = sq + HN * LD, *sx = sp + HN * LR_KEYS;  // [HN][LD] [HN][LR_KEYS] [KG][HN][R16]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_launch_dependents();
  pdl_wait();
  const Where at = where(w.rows, m);
  uint32_t t_begin, t_end;
  split_keys(min(at.pos + 1, a.cap), split, S, &t_begin, &t_end);
  const float *cache = static_cast<const float *>(a.cache) + (size_t)at.slot * a.cap * LD;
  for (uint32_t e = threadIdx.x; e < HN * LD; e += LR_THREADS) sq[e] = e / LD < hn ? q_in[((size_t)m * a.heads + h0) * LD + e] : 0.f;
  if (threadIdx.x < HN) sm[threadIdx.x] = -INFINITY, sl[threadIdx.x] = 0.f;
  __syncthreads();
  const uint32_t quad = threadIdx.x % tpp, kg = threadIdx.x / tpp;
  const bool pv = quad < quads && kg < KG;
  float acc[HN][4];
#pragma unroll
  for (int h = 0; h < HN; ++h) acc[h][0] = acc[h][1] = acc[h][2] = acc[h][3] = 0.f;
  for (uint32_t t0 = t_begin; t0 < t_end; t0 += LR_KEYS) {
    const uint32_t n = min((uint32_t)LR_KEYS, t_end - t0), l8 = threadIdx.x & 7, grp = threadIdx.x >> 3;
    for (uint32_t t = grp; t < (n + 31) / 32 * 32; t += 32) {
      float dot[HN];
#pragma unroll
      for (int h = 0; h < HN; ++h) dot[h] = 0.f;
      const float *k = cache + (size_t)(t0 + (t < n ? t : 0)) * LD;
      for (uint32_t c = l8 * 4; c < LD; c += 32) {
        const float4 kv = *reinterpret_cast<const float4 *>(k + c);
#pragma unroll
        for (int h = 0; h < HN; ++h) {
          const float4 qv = *reinterpret_cast<const float4 *>(sq + h * LD + c);
          dot[h] = fmaf(kv.x, qv.x, fmaf(kv.y, qv.y, fmaf(kv.z, qv.z, fmaf(kv.w, qv.w, dot[h]))));
        }
      }
#pragma unroll
      for (int h = 0; h < HN; ++h) {
        float x = dot[h];
        x += __shfl_xor_sync(0xffffffffu, x, 1);
        x += __shfl_xor_sync(0xffffffffu, x, 2);
        x += __shfl_xor_sync(0xffffffffu, x, 4);
        if (l8 == (uint32_t)h && t < n) sp[h * LR_KEYS + t] = x;
      }
    }
    __syncthreads();
    if (warp < HN) {
      float *s = sp + warp * LR_KEYS;
      const float old = sm[warp];
      float x[LR_KEYS / 32], mx = old, sum = 0.f;
#pragma unroll
      for (int e = 0; e < LR_KEYS / 32; ++e) {
        x[e] = lane + 32 * e < (int)n ? s[lane + 32 * e] : -INFINITY;
        mx = fmaxf(mx, x[e]);
      }
      mx = warp_max(mx);
      const float f = expf(old - mx);
#pragma unroll
      for (int e = 0; e < LR_KEYS / 32; ++e) {
        x[e] = expf(x[e] - mx);
        s[lane + 32 * e] = x[e];
        sum += x[e];
      }
      sum = warp_sum(sum);
      __syncwarp();
      if (lane == 0) sm[warp] = mx, sl[warp] = sl[warp] * f + sum, sf[warp] = f;
    }
    __syncthreads();
    if (pv) {
#pragma unroll
      for (int h = 0; h < HN; ++h)
#pragma unroll
        for (int x = 0; x < 4; ++x) acc[h][x] *= sf[h];
#pragma unroll 4
      for (uint32_t e = kg; e < n; e += KG) {
        const float4 v = *reinterpret_cast<const float4 *>(cache + (size_t)(t0 + e) * LD + quad * 4);
#pragma unroll
        for (int h = 0; h < HN; ++h) {
          const float p = sp[h * LR_KEYS + e];
          acc[h][0] = fmaf(p, v.x, acc[h][0]);
          acc[h][1] = fmaf(p, v.y, acc[h][1]);
          acc[h][2] = fmaf(p, v.z, acc[h][2]);
          acc[h][3] = fmaf(p, v.w, acc[h][3]);
        }
      }
    }
    __syncthreads();
  }
  if (pv)
#pragma unroll
    for (int h = 0; h < HN; ++h) *reinterpret_cast<float4 *>(sx + ((size_t)kg * HN + h) * R16 + quad * 4) = make_float4(acc[h][0], acc[h][1], acc[h][2], acc[h][3]);
  __syncthreads();
  for (uint32_t e = threadIdx.x; e < hn * R16; e += LR_THREADS) {
    float t = 0.f;
    for (uint32_t k = 0; k < KG; ++k) t += sx[(size_t)k * HN * R16 + e];
    parts.o[(((size_t)m * a.heads + h0 + e / R16) * S + split) * R16 + e % R16] = t;
  }
  if (threadIdx.x < hn) {
    float *ml = parts.ml + (((size_t)m * a.heads + h0 + threadIdx.x) * S + split) * 2;
    ml[0] = sm[threadIdx.x], ml[1] = sl[threadIdx.x];
  }
}

// grid (tiles of 32 value channels, heads, tiles of MT rows): the merged latent of every row, then W_uv and the gate.
constexpr uint32_t LV_ROWS = 32;
template <typename CT, int MT>
__global__ void __launch_bounds__(256) latent_value_kernel(const __grid_constant__ LatArgs w, Parts parts, uint32_t S, void *out, int out_fmt, uint32_t ld_out) {
  const greta_latent_attn &a = w.a;
  __shared__ __align__(16) float lat[MT][MAX_RANK];
  __shared__ float ws[MT][MAX_SPLITS];
  __shared__ uint32_t active[MT];
  const uint32_t h = blockIdx.y, m0 = blockIdx.z * MT, R16 = up16(a.rank), j0 = blockIdx.x * LV_ROWS;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const CT *wv = static_cast<const CT *>(a.w_kv) + ((size_t)a.heads * up8(a.dim) + (size_t)h * up8(a.vdim)) * a.ld_w;
  for (uint32_t j = j0 + warp * 4; j < min(j0 + warp * 4 + 4, a.vdim); ++j)
    for (uint32_t b = lane * 128; b < a.rank * (uint32_t)sizeof(CT); b += 32 * 128)
      asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const char *>(wv + (size_t)j * a.ld_w) + b));
  pdl_launch_dependents();
  pdl_wait();
  if (warp < MT) {  // weight of every split: exp(max - common max) / denominator; splits with keys come first
    uint32_t n = 0;
    if (m0 + warp < w.rows.M) {
      const float2 *ml = reinterpret_cast<const float2 *>(parts.ml) + ((size_t)(m0 + warp) * a.heads + h) * S;
      const float2 none = make_float2(-INFINITY, 0.f), x = lane < (int)S ? ml[lane] : none, y = lane + 32 < (int)S ? ml[lane + 32] : none;
      const bool p2 = sizeof(CT) == 2;
      const float sink = a.sink ? a.sink[h] * (p2 ? LOG2E : 1.f) : -INFINITY, mx = fmaxf(warp_max(fmaxf(x.x, y.x)), sink);
      const float fx = p2 ? exp2f(x.x - mx) : expf(x.x - mx), fy = p2 ? exp2f(y.x - mx) : expf(y.x - mx);
      const float den = warp_sum(fmaf(x.y, fx, y.y * fy)) + (a.sink ? (p2 ? exp2f(sink - mx) : expf(sink - mx)) : 0.f);
      ws[warp][lane] = fx / den;
      ws[warp][lane + 32] = fy / den;
      n = __popc(__ballot_sync(0xffffffffu, x.y > 0.f)) + __popc(__ballot_sync(0xffffffffu, y.y > 0.f));
    }
    if (lane == 0) active[warp] = n;
  }
  __syncthreads();
  for (uint32_t e = threadIdx.x * 4; e < MT * R16; e += 256 * 4) {
    const uint32_t t = e / R16, r = e % R16, m = m0 + t, n = active[t];
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    const float *o = parts.o + ((size_t)m * a.heads + h) * S * R16 + r;
#pragma unroll 8
    for (uint32_t s = 0; s < n; ++s) {
      const float4 v = *reinterpret_cast<const float4 *>(o + (size_t)s * R16);
      const float f = ws[t][s];
      x.x = fmaf(f, v.x, x.x), x.y = fmaf(f, v.y, x.y), x.z = fmaf(f, v.z, x.z), x.w = fmaf(f, v.w, x.w);
    }
    *reinterpret_cast<float4 *>(&lat[t][r]) = x;
  }
  __syncthreads();
  float acc[4][MT];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int t = 0; t < MT; ++t) acc[i][t] = 0.f;
  for (uint32_t r = lane * 8; r < R16; r += 256) {
    float f[4][8];
#pragma unroll
    for (int i = 0; i < 4; ++i) weights8(wv + (size_t)min(j0 + warp * 4 + i, a.vdim - 1) * a.ld_w + r, f[i]);
#pragma unroll
    for (int t = 0; t < MT; ++t) {
      const float4 u = *reinterpret_cast<const float4 *>(&lat[t][r]), v = *reinterpret_cast<const float4 *>(&lat[t][r + 4]);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        float y = acc[i][t];
        y = fmaf(f[i][0], u.x, fmaf(f[i][1], u.y, fmaf(f[i][2], u.z, fmaf(f[i][3], u.w, y))));
        acc[i][t] = fmaf(f[i][4], v.x, fmaf(f[i][5], v.y, fmaf(f[i][6], v.z, fmaf(f[i][7], v.w, y))));
      }
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const uint32_t j = j0 + warp * 4 + i;
    if (j >= a.vdim) break;
#pragma unroll
    for (int t = 0; t < MT; ++t) {
      const float y = warp_sum(acc[i][t]);
      const uint32_t m = m0 + t;
      if (lane == 0 && m < w.rows.M) {
        const uint32_t c = h * a.vdim + j;
        store_out(out, out_fmt, (size_t)m * ld_out + c, a.gate ? y * a.gate[(size_t)m * a.ld_gate + c] : y);
      }
    }
  }
}

// ---- prompts: tcgen05
__device__ __forceinline__ void tmem_st32(uint32_t taddr, const uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31,%32};" ::"r"(taddr),
      "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]),
      "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]), "r"(r[24]),
      "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
      : "memory");
}
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
// D[tmem] (+)= A[tmem, fp16 pairs] * B[smem desc], fp32 accumulate.
__device__ __forceinline__ void umma_f16_ts(uint32_t tmem_d, uint32_t tmem_a, uint32_t desc_b_lo, uint32_t desc_hi, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t.reg .b64 db;\n\t"
      "mov.b64 db, {%2, %3};\n\t"
      "setp.ne.b32 p, %5, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], db, %4, p;\n\t}" ::"r"(tmem_d),
      "r"(tmem_a), "r"(desc_b_lo), "r"(desc_hi), "r"(idesc), "r"(accumulate)
      : "memory");
}
constexpr uint32_t LP_Q = 128, LP_THREADS = 192, LP_TMEM = 512;
constexpr uint32_t LP_SLAB_Q = LP_Q * 128;          // bytes of 64 columns of the query tile
constexpr float LP_LAZY = 8.f;                      // a row's maximum may grow by this factor's exponent before its sums are rescaled

// grid (query tiles, heads).  Warp 0: TMA of the queries, keys (per-head part from the workspace, rotated part from the cache) and
// values; warp 1: MMA issuer; warps 2-5: softmax (one query row per thread) and outputs.  KT: keys per tile.
// A key tile's column slabs of 64 may reach into the next head's columns: the queries are zero there; surplus output columns are not read.
// TMEM columns: scores of even and odd tiles at 0 and 128, each overwritten by its weights (fp16 pairs); outputs from 256 on.
template <int KT>
__global__ void __launch_bounds__(LP_THREADS, 1)
latent_prefill_kernel(const __grid_constant__ LatArgs w, const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k, const __grid_constant__ CUtensorMap tmap_r, const __grid_constant__ CUtensorMap tmap_v,
                      void *out, int out_fmt, uint32_t ld_out, uint32_t stages) {
  const greta_latent_attn &a = w.a;
  extern __shared__ uint8_t smem_raw[];
  uint8_t *smem = reinterpret_cast<uint8_t *>(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  constexpr uint32_t SLAB = KT * 128;  // bytes of 64 columns of a key tile
  const uint32_t sd = slabs(a.dim), sr = slabs(a.rot_dim), sv = slabs(a.vdim), d8 = up8(a.dim), v8 = up8(a.vdim);
  uint8_t *qs = smem, *ks = qs + (sd + sr) * LP_SLAB_Q, *vs = ks + stages * (sd + sr) * SLAB;
  uint64_t *bars = reinterpret_cast<uint64_t *>(vs + stages * sv * SLAB);
  uint64_t *kf = bars, *ke = bars + 2, *vf = bars + 4, *ve = bars + 6, *sf = bars + 8, *pf = bars + 10, *od = bars + 12, *qf = bars + 13;
  uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(bars + 14);
  volatile int *abort_flag = reinterpret_cast<volatile int *>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t tile = gridDim.x - 1 - blockIdx.x, h = blockIdx.y;  // the longest rows first
  const uint32_t m0 = tile * LP_Q, nq = min(LP_Q, w.rows.M - m0), i0 = w.rows.pos0 + m0, total = i0 + nq, ntiles = (total + KT - 1) / KT;

  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; ++i) {
      mbar_init(&kf[i], 1);
      mbar_init(&ke[i], 1);
      mbar_init(&vf[i], 1);
      mbar_init(&ve[i], 1);
      mbar_init(&sf[i], 1);
      mbar_init(&pf[i], 4);
    }
    mbar_init(od, 1);
    mbar_init(qf, 1);
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tmap_q) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tmap_k) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tmap_r) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tmap_v) : "memory");
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, LP_TMEM);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  pdl_launch_dependents();
  pdl_wait();

  if (warp == 0) {
    if (lane == 0) {
      uint32_t issued = 0;
      bool ok = true;
      mbar_arrive_expect_tx(qf, (sd + sr) * LP_SLAB_Q);
      for (uint32_t c = 0; c < sd + sr; ++c) tma_load_2d(qs + c * LP_SLAB_Q, &tmap_q, (int)((h * (sd + sr) + c) * 64), (int)m0, qf);
      for (uint32_t t = 0; t < ntiles && ok; ++t) {
        const uint32_t st = t % stages, ph = ((t / stages) & 1) ^ 1;
        ok = mbar_wait(&ke[st], ph, abort_flag, 100 + st);
        if (!ok) break;
        uint8_t *kd = ks + st * (sd + sr) * SLAB, *vd = vs + st * sv * SLAB;
        mbar_arrive_expect_tx(&kf[st], (sd + sr) * SLAB);
        for (uint32_t c = 0; c < sd; ++c) tma_load_2d(kd + c * SLAB, &tmap_k, (int)(h * d8 + c * 64), (int)(t * KT), &kf[st]);
        for (uint32_t c = 0; c < sr; ++c) tma_load_2d(kd + (sd + c) * SLAB, &tmap_r, (int)(up16(a.rank) + c * 64), (int)(t * KT), &kf[st]);
        ok = mbar_wait(&ve[st], ph, abort_flag, 110 + st);
        issued = t + 1;
        if (!ok) break;
        mbar_arrive_expect_tx(&vf[st], sv * SLAB);
        for (uint32_t c = 0; c < sv; ++c) tma_load_2d(vd + c * SLAB, &tmap_v, (int)(h * v8 + c * 64), (int)(t * KT), &vf[st]);
      }
      if (*abort_flag) {  // give copies in flight a bounded chance to land before the CTA leaves
        const long long q0 = clock64();
        while (!mbar_try_wait(qf, 0) && clock64() - q0 < 20000000ll) {
        }
        for (uint32_t t = issued > stages ? issued - stages : 0; t < issued; ++t) {
          const long long c0 = clock64();
          while (!mbar_try_wait(&kf[t % stages], (t / stages) & 1) && clock64() - c0 < 20000000ll) {
          }
          while (!mbar_try_wait(&vf[t % stages], (t / stages) & 1) && clock64() - c0 < 40000000ll) {
          }
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc_s = instr_desc_f16(LP_Q, KT);
      const uint32_t idesc_o = instr_desc_f16(LP_Q, up16(a.vdim)) | (1u << 16);  // values: keys are the rows of memory (N-major operand)
      const uint32_t q_lo = smem_desc_lo(smem_u32(qs)), k_lo = smem_desc_lo(smem_u32(ks));
      const uint32_t v_lo = ((smem_u32(vs) >> 4) & 0x3FFFu) | ((SLAB >> 4) << 16);  // 64-column groups are a slab apart
      auto scores = [&](uint32_t t) {
        const uint32_t st = t % stages;
        if (!mbar_wait_now(&kf[st], (t / stages) & 1, abort_flag, 200 + st)) return false;
        tc_fence_after();
        uint32_t acc = 0;
        auto part = [&](uint32_t slab0, uint32_t cols) {
          for (uint32_t k16 = 0; k16 < (cols + 15) / 16; ++k16, acc = 1) {
            const uint32_t s = slab0 + k16 / 4, in = (k16 & 3) * 2;
            umma_f16(tmem + (t & 1) * 128, q_lo + s * (LP_SLAB_Q >> 4) + in, k_lo + (st * (sd + sr) + s) * (SLAB >> 4) + in, SMEM_DESC_HI_SW128, idesc_s, acc);
          }
        };
        part(0, a.dim);
        part(sd, a.rot_dim);
        umma_commit(&ke[st]);
        umma_commit(&sf[t & 1]);
        return true;
      };
      bool ok = mbar_wait_now(qf, 0, abort_flag, 210);
      tc_fence_after();
      ok = ok && scores(0) && (ntiles < 2 || scores(1));
      for (uint32_t t = 0; t < ntiles && ok; ++t) {
        const uint32_t st = t % stages;
        ok = mbar_wait_now(&pf[t & 1], (t >> 1) & 1, abort_flag, 220 + (t & 1)) && mbar_wait_now(&vf[st], (t / stages) & 1, abort_flag, 230 + st);
        if (!ok) break;
        tc_fence_after();
        for (uint32_t k16 = 0; k16 < KT / 16; ++k16)
          umma_f16_ts(tmem + 256, tmem + (t & 1) * 128 + k16 * 8, v_lo + st * sv * (SLAB >> 4) + k16 * (2048 >> 4), SMEM_DESC_HI_SW128, idesc_o, (t | k16) ? 1u : 0u);
        umma_commit(&ve[st]);
        umma_commit(od);
        if (t + 2 < ntiles) ok = mbar_wait_now(od, t & 1, abort_flag, 240) && scores(t + 2);  // the weights of tile t are read: its columns are free
      }
    }
  } else {
    const uint32_t quad = warp & 3, row = quad * 32 + lane, i = i0 + row;
    if (a.gate && row < nq)  // the gates travel to L2 meanwhile
      for (uint32_t c = 0; c < a.vdim; c += 32)
        asm volatile("prefetch.global.L2 [%0];" ::"l"(a.gate + (size_t)(m0 + row) * a.ld_gate + (size_t)h * a.vdim + c));
    const uint32_t lanes = tmem + (quad * 32 << 16), o_cols = up16(a.vdim);
    float mx = -INFINITY, l = 0.f;
    bool ok = true;
    for (uint32_t t = 0; t < ntiles && ok; ++t) {
      const uint32_t sb = lanes + (t & 1) * 128;
      ok = mbar_wait_now(&sf[t & 1], (t >> 1) & 1, abort_flag, 300 + (t & 1));
      if (!ok) break;
      tc_fence_after();
      __syncwarp();
      uint32_t v[KT / 32][32];
#pragma unroll
      for (int c = 0; c < KT / 32; ++c) tmem_ld32(sb + c * 32, v[c]);
      tmem_ld_wait();
      if (t * KT + KT - 1 > i0) {  // the diagonal (or the end) runs through the tile
#pragma unroll
        for (int c = 0; c < KT / 32; ++c)
#pragma unroll
          for (int j = 0; j < 32; ++j)
            if (t * KT + c * 32 + j > i) v[c][j] = 0xFF800000u;
      }
      float tm[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int c = 0; c < KT / 32; ++c)
#pragma unroll
        for (int j = 0; j < 32; ++j) tm[j & 3] = fmaxf(tm[j & 3], __uint_as_float(v[c][j]));
      const float nm = fmaxf(mx, fmaxf(fmaxf(tm[0], tm[1]), fmaxf(tm[2], tm[3])));  // finite from the first tile on: key 0
      if (t == 0) {
        mx = nm;
      } else if (__any_sync(0xffffffffu, nm > mx + LP_LAZY)) {
        const float f = nm > mx + LP_LAZY ? ex2(mx - nm) : 1.f;
        if (nm > mx + LP_LAZY) mx = nm;
        l *= f;
        ok = mbar_wait_now(od, (t - 1) & 1, abort_flag, 310);  // every product so far is in
        if (!ok) break;
        tc_fence_after();
        __syncwarp();
        for (uint32_t c = 0; c < o_cols; c += 32) {  // the last columns of a group of 32 may be surplus
          uint32_t o[32];
          tmem_ld32(lanes + 256 + c, o);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 32; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * f);
          tmem_st32(lanes + 256 + c, o);
        }
      }
      float sum[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int c = 0; c < KT / 64; ++c) {
        uint32_t p[32];
#pragma unroll
        for (int j = 0; j < 32; ++j) {
          const float p0 = ex2(__uint_as_float(v[2 * c + j / 16][(2 * j) & 31]) - mx), p1 = ex2(__uint_as_float(v[2 * c + j / 16][(2 * j + 1) & 31]) - mx);
          sum[(2 * j) & 3] += p0;
          sum[(2 * j + 1) & 3] += p1;
          p[j] = half2_bits(p0, p1);
        }
        tmem_st32(sb + c * 32, p);
      }
      l += (sum[0] + sum[1]) + (sum[2] + sum[3]);
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&pf[t & 1]);
    }
    // the last two products one after the other: a wait may be one phase behind its barrier, not two
    ok = ok && (ntiles < 2 || mbar_wait_now(od, (ntiles - 2) & 1, abort_flag, 320)) && mbar_wait_now(od, (ntiles - 1) & 1, abort_flag, 321);
    if (ok) {
      tc_fence_after();
      const float sink2 = a.sink ? a.sink[h] * LOG2E : -INFINITY, nm = fmaxf(mx, sink2), f = ex2(mx - nm), inv = f / (l * f + ex2(sink2 - nm));
      const size_t m = m0 + row, at = m * ld_out + (size_t)h * a.vdim;
      const float *gate = a.gate ? a.gate + m * a.ld_gate + (size_t)h * a.vdim : nullptr;
      const bool vec = a.vdim % 8 == 0 && ld_out % 8 == 0 && ((uintptr_t)out & 15) == 0 && (!gate || (a.ld_gate % 4 == 0 && ((uintptr_t)a.gate & 15) == 0));
      for (uint32_t c = 0; c < a.vdim; c += 32) {
        uint32_t o[32];
        __syncwarp();
        tmem_ld32(lanes + 256 + c, o);
        tmem_ld_wait();
        if (row >= nq) continue;
#pragma unroll
        for (int j = 0; j < 32; j += 8) {
          if (c + j >= a.vdim) break;
          float y[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) y[e] = __uint_as_float(o[j + e]) * inv;
          if (vec) {
            if (gate) {
              const float4 g0 = *reinterpret_cast<const float4 *>(gate + c + j), g1 = *reinterpret_cast<const float4 *>(gate + c + j + 4);
              y[0] *= g0.x, y[1] *= g0.y, y[2] *= g0.z, y[3] *= g0.w, y[4] *= g1.x, y[5] *= g1.y, y[6] *= g1.z, y[7] *= g1.w;
            }
            if (out_fmt == GRETA_OUT_BF16) {
              uint4 u;
              __nv_bfloat162 b0 = __floats2bfloat162_rn(y[0], y[1]), b1 = __floats2bfloat162_rn(y[2], y[3]);
              __nv_bfloat162 b2 = __floats2bfloat162_rn(y[4], y[5]), b3 = __floats2bfloat162_rn(y[6], y[7]);
              u.x = *reinterpret_cast<uint32_t *>(&b0), u.y = *reinterpret_cast<uint32_t *>(&b1);
              u.z = *reinterpret_cast<uint32_t *>(&b2), u.w = *reinterpret_cast<uint32_t *>(&b3);
              *reinterpret_cast<uint4 *>(static_cast<__nv_bfloat16 *>(out) + at + c + j) = u;
              continue;
            }
          }
#pragma unroll
          for (int e = 0; e < 8; ++e)
            if (c + j + e < a.vdim) store_out(out, out_fmt, at + c + j + e, gate && !vec ? y[e] * gate[c + j + e] : y[e]);
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, LP_TMEM);
  }
}

int check_latent(const char *what, const greta_latent_attn *a, const greta_rows *r) {
  GRETA_REQUIRE(a && r && r->M, "%s: null or empty argument", what);
  GRETA_REQUIRE(a->heads && a->dim && a->dim <= MAX_DIM && a->vdim && a->vdim <= MAX_DIM, "%s: head sizes %u / %u (1..%u)", what, a->dim, a->vdim, MAX_DIM);
  GRETA_REQUIRE(a->rank && a->rank <= MAX_RANK && a->rot_dim && a->rot_dim <= MAX_ROT, "%s: latent of %u (1..%u), rotated part of %u (1..%u)", what, a->rank,
                MAX_RANK, a->rot_dim, MAX_ROT);
  GRETA_REQUIRE(a->rot_dims % 2 == 0 && a->rot_dims <= a->rot_dim && (!a->rot_dims || (a->rotation && a->positions)), "%s: %u rotated channels of %u", what,
                a->rot_dims, a->rot_dim);
  GRETA_REQUIRE(a->fmt == GRETA_FMT_F16 || a->fmt == GRETA_FMT_F32, "%s: cache format %d", what, a->fmt);
  GRETA_REQUIRE(a->cache && aligned16(a->cache) && a->cap && a->down && a->latent_norm, "%s: no cache or no latent", what);
  GRETA_REQUIRE(r->d_pos || r->pos0 + r->M <= a->cap, "%s: positions past the cache's %u rows", what, a->cap);
  return GRETA_OK;
}

// Heads a CTA of the fp16 form takes (16 or 32), splits of the keys: enough CTAs to fill the GPU, at least a tile of keys each.
uint32_t head_group(const greta_latent_attn &a, uint32_t M) {
  return a.fmt == GRETA_FMT_F32 ? 8 : a.heads > 16 && a.rank <= 512 && (uint64_t)M * ((a.heads + 31) / 32) * 8 >= 148 ? 32 : 16;
}
uint32_t split_count(const greta_latent_attn &a, uint32_t M, uint32_t max_len) {
  const uint64_t ctas = (uint64_t)M * ((a.heads + head_group(a, M) - 1) / head_group(a, M));
  uint32_t s = 1;
  while (s < MAX_SPLITS && ctas * s * 2 <= 296 && max_len > s * 64) s *= 2;
  return s;
}

template <int HT, int NT>
int launch_mma(cudaStream_t s, const LatArgs &w, const __half *q, const Parts &parts, uint32_t splits) {
  constexpr size_t LIMIT = 227 * 1024;
  const uint32_t row = (up16(w.a.rank) + up16(w.a.rot_dim)) * 2 + 16;
  auto bytes = [&](int buffers) { return (size_t)16 * HT * (row + LM_K * 2 + 16) + (size_t)buffers * LM_K * row + 8 * 16 * HT * 4; };
  // Two tiles in flight, unless two CTAs with one each fit an SM and there are enough of them.
  const uint64_t ctas = (uint64_t)splits * ((w.a.heads + 16 * HT - 1) / (16 * HT)) * w.rows.M;
  const int buffers = bytes(2) <= LIMIT && !(ctas > (uint32_t)sm_count() && bytes(1) <= LIMIT / 2) ? 2 : 1;
  static bool attr_set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !attr_set[dev]) {
    GRETA_CUDA_TRY(cudaFuncSetAttribute(latent_mma_kernel<HT, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)LIMIT));
    attr_set[dev] = true;
  }
  GRETA_CUDA_TRY(launch_pdl(latent_mma_kernel<HT, NT>, dim3(splits, (w.a.heads + 16 * HT - 1) / (16 * HT), w.rows.M), dim3(LM_THREADS), bytes(buffers), s, w, q,
                            parts, buffers));
  return launched("latent_mma_kernel");
}
template <int HT>
int pick_mma(cudaStream_t s, const LatArgs &w, const __half *q, const Parts &parts, uint32_t splits) {
  const uint32_t tiles = (up16(w.a.rank) / 16 + 7) / 8;
  if (tiles <= 1) return launch_mma<HT, 1>(s, w, q, parts, splits);
  if (tiles <= 2) return launch_mma<HT, 2>(s, w, q, parts, splits);
  if (tiles <= 4) return launch_mma<HT, 4>(s, w, q, parts, splits);
  return launch_mma<1, 8>(s, w, q, parts, splits);
}
int launch_rows(cudaStream_t s, const LatArgs &w, const float *q, const Parts &parts, uint32_t splits) {
  constexpr int HN = 8;
  const uint32_t R16 = up16(w.a.rank), LD = R16 + up16(w.a.rot_dim), KG = LR_THREADS / ((R16 / 4 + 31) / 32 * 32);
  const size_t smem = (size_t)HN * (LD + LR_KEYS + (size_t)KG * R16) * 4;
  static bool attr_set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !attr_set[dev]) {
    GRETA_CUDA_TRY(cudaFuncSetAttribute(latent_rows_kernel<HN>, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024));
    attr_set[dev] = true;
  }
  GRETA_CUDA_TRY(launch_pdl(latent_rows_kernel<HN>, dim3(splits, (w.a.heads + HN - 1) / HN, w.rows.M), dim3(LR_THREADS), smem, s, w, q, parts));
  return launched("latent_rows_kernel");
}
template <typename CT, int MT>
int launch_query(cudaStream_t s, const LatArgs &w, CT *q) {
  const uint32_t tiles = (up16(w.a.rank) + LQ_COLS - 1) / LQ_COLS;
  GRETA_CUDA_TRY(launch_pdl(latent_query_kernel<CT, MT>, dim3(tiles + 1, w.a.heads, (w.rows.M + MT - 1) / MT), dim3(256), 0, s, w, q));
  return launched("latent_query_kernel");
}
template <typename CT, int MT>
int launch_value(cudaStream_t s, const LatArgs &w, const Parts &parts, uint32_t splits, void *out, int out_fmt, uint32_t ld_out) {
  GRETA_CUDA_TRY(launch_pdl(latent_value_kernel<CT, MT>, dim3((w.a.vdim + LV_ROWS - 1) / LV_ROWS, w.a.heads, (w.rows.M + MT - 1) / MT), dim3(256), 0, s, w,
                            parts, splits, out, out_fmt, ld_out));
  return launched("latent_value_kernel");
}
// 64-column boxes of a row-major fp16 matrix, 128-byte swizzle; columns and rows outside read as zero.
int make_map(CUtensorMap *map, const void *base, uint32_t cols, uint32_t rows, uint32_t box_rows) {
  EncodeTiledFn enc = encode_tiled();
  if (!enc) {
    set_error("latent_prefill: cuTensorMapEncodeTiled is not available from this driver");
    return GRETA_ERR_NOT_IMPLEMENTED;
  }
  const cuuint64_t dims[2] = {cols, rows}, strides[1] = {(cuuint64_t)cols * 2};
  const cuuint32_t box[2] = {64, box_rows}, estr[2] = {1, 1};
  const CUresult r = enc(map, CU_TENSOR_MAP_DATA_TYPE_FLOAT16, 2, const_cast<void *>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                         CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) {
    set_error("latent_prefill: cuTensorMapEncodeTiled failed with code %d", (int)r);
    return GRETA_ERR_INVALID_ARGS;
  }
  return GRETA_OK;
}
constexpr size_t LP_SMEM_LIMIT = 227 * 1024;
size_t prefill_smem(const greta_latent_attn &a, uint32_t kt, uint32_t stages) {
  const uint32_t q = slabs(a.dim) + slabs(a.rot_dim);
  return (size_t)q * LP_SLAB_Q + (size_t)stages * (q + slabs(a.vdim)) * kt * 128 + 1024 + 256;
}
template <int KT>
int launch_prefill(cudaStream_t s, const LatArgs &w, const void *q, const void *k, const void *v, void *out, int out_fmt, uint32_t ld_out, uint32_t stages) {
  const greta_latent_attn &a = w.a;
  const uint32_t total = w.rows.pos0 + w.rows.M, LD = up16(a.rank) + up16(a.rot_dim);
  CUtensorMap mq, mk, mr, mv;
  if (int rc = make_map(&mq, q, a.heads * (slabs(a.dim) + slabs(a.rot_dim)) * 64, w.rows.M, LP_Q)) return rc;
  if (int rc = make_map(&mk, k, a.heads * up8(a.dim), total, KT)) return rc;
  if (int rc = make_map(&mr, static_cast<const __half *>(a.cache) + (size_t)w.rows.slot0 * a.cap * LD, LD, total, KT)) return rc;
  if (int rc = make_map(&mv, v, a.heads * up8(a.vdim), total, KT)) return rc;
  static bool attr_set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !attr_set[dev]) {
    GRETA_CUDA_TRY(cudaFuncSetAttribute(latent_prefill_kernel<KT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)LP_SMEM_LIMIT));
    attr_set[dev] = true;
  }
  GRETA_CUDA_TRY(launch_pdl(latent_prefill_kernel<KT>, dim3((w.rows.M + LP_Q - 1) / LP_Q, a.heads), dim3(LP_THREADS), prefill_smem(a, KT, stages), s, w, mq, mk, mr, mv,
                            out, out_fmt, ld_out, stages));
  return launched("latent_prefill_kernel");
}
size_t q_bytes(const greta_latent_attn &a, uint32_t M) {
  return ((size_t)M * a.heads * (up16(a.rank) + up16(a.rot_dim)) * (a.fmt == GRETA_FMT_F32 ? 4 : 2) + 15) / 16 * 16;
}

}  // namespace

namespace greta {
cudaError_t latent_wait_status(int *code) { return cudaMemcpyFromSymbol(code, g_gemm_error, sizeof(int)); }
}  // namespace greta

extern "C" {

uint32_t greta_cuda_latent_row(uint32_t rank, uint32_t rot_dim) { return up16(rank) + up16(rot_dim); }

uint32_t greta_cuda_latent_query_row(uint32_t heads, uint32_t dim, uint32_t rot_dim) { return heads * (slabs(dim) + slabs(rot_dim)) * 64; }

int greta_cuda_latent_prepare(greta_stream_t stream, const greta_latent_attn *a, const greta_rows *rows, void *q_out) {
  if (int rc = check_latent("latent_prepare", a, rows)) return rc;
  GRETA_REQUIRE(!q_out || (a->q && aligned16(q_out)), "latent_prepare: no queries, or a misaligned output");
  const LatArgs w{*a, *rows};
  __half *q = static_cast<__half *>(q_out);
  if (a->fmt == GRETA_FMT_F16)
    GRETA_CUDA_TRY(launch_pdl(latent_prepare_kernel<__half>, dim3(rows->M), dim3(256), 0, (cudaStream_t)stream, w, q));
  else
    GRETA_CUDA_TRY(launch_pdl(latent_prepare_kernel<float>, dim3(rows->M), dim3(256), 0, (cudaStream_t)stream, w, q));
  return launched("latent_prepare_kernel");
}

size_t greta_cuda_latent_scratch_bytes(const greta_latent_attn *a, uint32_t M, uint32_t max_len) {
  size_t most = 0;
  for (uint32_t m = 1; m <= M; ++m)  // fewer rows are split further
    most = std::max(most, q_bytes(*a, m) + (size_t)m * a->heads * split_count(*a, m, max_len) * (up16(a->rank) + 2) * 4);
  return most;
}

int greta_cuda_latent_absorbed(greta_stream_t stream, const greta_latent_attn *a, const greta_rows *rows, void *scratch, void *out, int out_fmt,
                               uint32_t ld_out, uint32_t max_len) {
  if (int rc = check_latent("latent_absorbed", a, rows)) return rc;
  GRETA_REQUIRE(scratch && aligned16(scratch) && out && max_len && a->q && a->w_kv && aligned16(a->w_kv), "latent_absorbed: null or misaligned pointer");
  GRETA_REQUIRE(a->ld_w % 64 == 0 && a->ld_w >= a->rank && a->heads <= 65535 && rows->M <= 65535, "latent_absorbed: ld_w=%u", a->ld_w);
  const LatArgs w{*a, *rows};
  cudaStream_t s = (cudaStream_t)stream;
  const uint32_t S = split_count(*a, rows->M, max_len), R16 = up16(a->rank), M = rows->M;
  Parts parts;
  parts.o = reinterpret_cast<float *>(static_cast<uint8_t *>(scratch) + q_bytes(*a, M));
  parts.ml = parts.o + (size_t)M * a->heads * S * R16;
  if (a->fmt == GRETA_FMT_F16) {
    __half *q = static_cast<__half *>(scratch);
    if (int rc = M == 1 ? launch_query<__half, 1>(s, w, q) : launch_query<__half, 4>(s, w, q)) return rc;
    if (int rc = head_group(*a, M) == 32 ? pick_mma<2>(s, w, q, parts, S) : pick_mma<1>(s, w, q, parts, S)) return rc;
    return M == 1 ? launch_value<__half, 1>(s, w, parts, S, out, out_fmt, ld_out) : launch_value<__half, 4>(s, w, parts, S, out, out_fmt, ld_out);
  }
  float *q = static_cast<float *>(scratch);
  if (int rc = M == 1 ? launch_query<float, 1>(s, w, q) : launch_query<float, 4>(s, w, q)) return rc;
  if (int rc = launch_rows(s, w, q, parts, S)) return rc;
  return M == 1 ? launch_value<float, 1>(s, w, parts, S, out, out_fmt, ld_out) : launch_value<float, 4>(s, w, parts, S, out, out_fmt, ld_out);
}

int greta_cuda_latent_prefill(greta_stream_t stream, const greta_latent_attn *a, const greta_rows *rows, const void *q, const void *k, const void *v,
                              void *out, int out_fmt, uint32_t ld_out) {
  if (int rc = check_latent("latent_prefill", a, rows)) return rc;
  GRETA_REQUIRE(!rows->d_pos && q && k && v && aligned16(q) && aligned16(k) && aligned16(v) && out && a->heads <= 65535, "latent_prefill: null pointer, or rows of a batch");
  GRETA_REQUIRE(a->fmt == GRETA_FMT_F16, "latent_prefill: the cache must be F16");
  const LatArgs w{*a, *rows};
  cudaStream_t s = (cudaStream_t)stream;
  for (uint32_t stages = 2; stages >= 1; --stages) {  // wide heads: shorter key tiles, then a single stage
    if (prefill_smem(*a, 128, stages) <= LP_SMEM_LIMIT) return launch_prefill<128>(s, w, q, k, v, out, out_fmt, ld_out, stages);
    if (prefill_smem(*a, 64, stages) <= LP_SMEM_LIMIT) return launch_prefill<64>(s, w, q, k, v, out, out_fmt, ld_out, stages);
  }
  set_error("latent_prefill: head sizes %u + %u / %u do not fit shared memory", a->dim, a->rot_dim, a->vdim);
  return GRETA_ERR_INVALID_ARGS;
}

}  // extern "C"
