// Latent attention: every head's keys and values are linear images of one cached latent per token, plus one rotated key part
// that all heads share.
//   latent_cache_kernel     norm of the latent, rotation of the shared key part, cache row
//   absorbed form (decode, short portions; 32-bit models always)
//     latent_query_kernel   q W_uk per head and the rotated q, so that a score is one dot product with a cache row; the new
//                           tokens' cache rows are written beside it
//     latent_mma_kernel     one row's heads as the 16-row operand of mma.sync (fp16), the cached latents as keys and as values,
//                           the keys split over CTAs; partial sums, maxima and normalisers to scratch
//     latent_rows_kernel    the same in 32-bit on the CUDA cores
//     latent_value_kernel   merges the splits (with the sink), applies W_uv per head and the output gate
//   expanded form (prompts)
//     latent_prefill_kernel keys and values of all heads lie in a workspace (a dense product of the cached latents); tiles of
//                           query positions x 64 keys on the tensor cores, the rotated key part read from the cache
// Scores, weights, sums and angles are fp32 throughout.
#include <algorithm>

#include "dense_device.cuh"
#include "mma_device.cuh"

using namespace greta;

namespace {

__host__ __device__ constexpr uint32_t up8(uint32_t d) { return (d + 7u) & ~7u; }
__host__ __device__ constexpr uint32_t up16(uint32_t d) { return (d + 15u) & ~15u; }
constexpr float LOG2E = 1.4426950408889634f;
constexpr uint32_t MAX_RANK = 1024, MAX_ROT = 128, MAX_DIM = 256, MAX_SPLITS = 32;

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
template <typename CT>
__global__ void __launch_bounds__(256) latent_cache_kernel(const __grid_constant__ LatArgs w) {
  pdl_launch_dependents();
  pdl_wait();
  const uint32_t m = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (m < w.rows.M) write_cache_row<CT>(w.a, w.rows, m, threadIdx.x & 31);
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
  __shared__ float lat[MT][MAX_RANK];
  __shared__ float ws[MT][MAX_SPLITS];
  const uint32_t h = blockIdx.y, m0 = blockIdx.z * MT, R16 = up16(a.rank), j0 = blockIdx.x * LV_ROWS;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const CT *wv = static_cast<const CT *>(a.w_kv) + ((size_t)a.heads * up8(a.dim) + (size_t)h * up8(a.vdim)) * a.ld_w;
  for (uint32_t j = j0 + warp * 4; j < min(j0 + warp * 4 + 4, a.vdim); ++j)
    for (uint32_t b = lane * 128; b < a.rank * (uint32_t)sizeof(CT); b += 32 * 128)
      asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const char *>(wv + (size_t)j * a.ld_w) + b));
  pdl_launch_dependents();
  pdl_wait();
  if (warp < MT && m0 + warp < w.rows.M) {  // weight of every split: exp(max - common max) / denominator
    const float *ml = parts.ml + ((size_t)(m0 + warp) * a.heads + h) * S * 2;
    const float mine = lane < (int)S ? ml[lane * 2] : -INFINITY, sum = lane < (int)S ? ml[lane * 2 + 1] : 0.f;
    const bool p2 = sizeof(CT) == 2;
    const float sink = a.sink ? a.sink[h] * (p2 ? LOG2E : 1.f) : -INFINITY;
    const float mx = fmaxf(warp_max(mine), sink), f = p2 ? exp2f(mine - mx) : expf(mine - mx);
    const float den = warp_sum(sum * f) + (a.sink ? (p2 ? exp2f(sink - mx) : expf(sink - mx)) : 0.f);
    if (lane < (int)S) ws[warp][lane] = f / den;
  }
  __syncthreads();
  for (uint32_t e = threadIdx.x; e < MT * R16; e += 256) {
    const uint32_t t = e / R16, r = e % R16, m = m0 + t;
    float x = 0.f;
    if (m < w.rows.M) {
      const float *o = parts.o + ((size_t)m * a.heads + h) * S * R16 + r;
      for (uint32_t s = 0; s < S; ++s)
        if (ws[t][s] != 0.f) x = fmaf(ws[t][s], o[(size_t)s * R16], x);  // a split without keys has left nothing
    }
    lat[t][r] = x;
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const uint32_t j = j0 + warp * 4 + i;
    if (j >= a.vdim) break;
    float acc[MT];
#pragma unroll
    for (int t = 0; t < MT; ++t) acc[t] = 0.f;
    for (uint32_t r = lane * 8; r < R16; r += 256) {
      float f[8];
      weights8(wv + (size_t)j * a.ld_w + r, f);
#pragma unroll
      for (int t = 0; t < MT; ++t)
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[t] = fmaf(f[e], lat[t][r + e], acc[t]);
    }
#pragma unroll
    for (int t = 0; t < MT; ++t) {
      const float y = warp_sum(acc[t]);
      const uint32_t m = m0 + t;
      if (lane == 0 && m < w.rows.M) {
        const uint32_t c = h * a.vdim + j;
        store_out(out, out_fmt, (size_t)m * ld_out + c, a.gate ? y * a.gate[(size_t)m * a.ld_gate + c] : y);
      }
    }
  }
}

// Prompts: blockDim / 32 warps x 16 query positions of one head per CTA, 64 keys per step, two steps in flight.
// DV: value size bucket (64, 128 or 256).
constexpr uint32_t LP_K = 64;
template <int DV>
__global__ void __launch_bounds__(256) latent_prefill_kernel(const __grid_constant__ LatArgs w, const __half *__restrict__ kx, const __half *__restrict__ vx,
                                                             void *out, int out_fmt, uint32_t ld_out) {
  const greta_latent_attn &a = w.a;
  extern __shared__ __align__(16) uint8_t smb[];
  const uint32_t D16 = up16(a.dim), P16 = up16(a.rot_dim), KD = D16 + P16, V16 = up16(a.vdim), KB = KD * 2 + 16, VB = V16 * 2 + 16;
  const uint32_t nq_max = blockDim.x / 2, threads = blockDim.x;
  uint8_t *qs = smb, *kt = qs + (size_t)nq_max * KB, *vt = kt + 2 * LP_K * KB;
  const uint32_t smem = nq_max * KB + 2 * LP_K * (KB + VB);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, tq = lane & 3, mat = lane >> 3, r8 = lane & 7;
  const uint32_t tile = gridDim.x - 1 - blockIdx.x, h = blockIdx.y;  // the longest rows first
  const uint32_t m0 = tile * nq_max, nq = min(nq_max, w.rows.M - m0), i0 = w.rows.pos0 + m0, total = i0 + nq;
  const uint32_t R16 = up16(a.rank), LD = R16 + P16, d8 = up8(a.dim), v8 = up8(a.vdim);
  for (uint32_t e = threadIdx.x; e < smem / 16; e += threads) reinterpret_cast<uint4 *>(smb)[e] = make_uint4(0, 0, 0, 0);
  pdl_launch_dependents();
  pdl_wait();
  __syncthreads();
  const __half *cache = static_cast<const __half *>(a.cache) + (size_t)w.rows.slot0 * a.cap * LD + R16;
  const __half *kh = kx + (size_t)h * d8, *vh = vx + (size_t)h * v8;
  const uint32_t ntiles = (total + LP_K - 1) / LP_K, kc = d8 / 8, rc = P16 / 8, per = kc + rc + v8 / 8;
  auto stage = [&](uint32_t t, int buf) {
    if (t < ntiles) {
      for (uint32_t e = threadIdx.x; e < LP_K * per; e += threads) {
        const uint32_t r = e / per, c = e % per, key = t * LP_K + r;
        const bool on = key < total;
        const size_t j = on ? key : 0;
        uint8_t *krow = kt + (size_t)(buf * LP_K + r) * KB;
        if (c < kc)
          cp16z(krow + c * 16, kh + j * a.heads * d8 + c * 8, on);
        else if (c < kc + rc)
          cp16z(krow + (D16 / 8 + c - kc) * 16, cache + j * LD + (c - kc) * 8, on);
        else
          cp16z(vt + (size_t)(buf * LP_K + r) * VB + (c - kc - rc) * 16, vh + j * a.heads * v8 + (c - kc - rc) * 8, on);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  stage(0, 0);
  const float scale = a.scale * LOG2E;
  for (uint32_t e = threadIdx.x; e < nq * KD; e += threads) {
    const uint32_t r = e / KD, c = e % KD;
    const float *x = a.q + (size_t)(m0 + r) * a.ld_q + (size_t)h * (a.dim + a.rot_dim);
    float v = 0.f;
    if (c < a.dim) v = x[c];
    else if (c >= D16 && c - D16 < a.rot_dim) v = rotated(a, x + a.dim, i0 + r, c - D16);
    *reinterpret_cast<__half *>(qs + (size_t)r * KB + c * 2) = __float2half_rn(v * scale);
  }
  const uint32_t qi[2] = {i0 + warp * 16 + gq, i0 + warp * 16 + gq + 8};
  float o[DV / 8][4], mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int n = 0; n < DV / 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[n][e] = 0.f;
  for (uint32_t t = 0; t < ntiles; ++t) {
    const int buf = t & 1;
    stage(t + 1, buf ^ 1);
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    if (t * LP_K <= i0 + warp * 16 + 15) {  // some key of the tile is visible to some row of this warp
      float s[LP_K / 8][4];
#pragma unroll
      for (int n = 0; n < (int)LP_K / 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[n][e] = 0.f;
#pragma unroll 2
      for (uint32_t ks = 0; ks < KD / 16; ++ks) {
        uint32_t qa[4];
        ldsm_x4(qa, qs + (size_t)(warp * 16 + (mat & 1) * 8 + r8) * KB + ks * 32 + (mat >> 1) * 16);
#pragma unroll
        for (int n = 0; n < (int)LP_K / 16; ++n) {
          uint32_t kb[4];
          ldsm_x4(kb, kt + (size_t)(buf * LP_K + n * 16 + (mat >> 1) * 8 + r8) * KB + ks * 32 + (mat & 1) * 16);
          mma16816(s[2 * n], qa, kb[0], kb[1]);
          mma16816(s[2 * n + 1], qa, kb[2], kb[3]);
        }
      }
      if (t * LP_K + LP_K - 1 > i0 + warp * 16) {  // the diagonal runs through the tile
#pragma unroll
        for (int n = 0; n < (int)LP_K / 8; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (t * LP_K + n * 8 + 2 * tq + (e & 1) > qi[e >> 1]) s[n][e] = -INFINITY;
      }
      float f[2], base[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        float tm = -INFINITY;
#pragma unroll
        for (int n = 0; n < (int)LP_K / 8; ++n) tm = fmaxf(tm, fmaxf(s[n][2 * r], s[n][2 * r + 1]));
        tm = fmaxf(tm, __shfl_xor_sync(0xffffffffu, tm, 1));
        tm = fmaxf(tm, __shfl_xor_sync(0xffffffffu, tm, 2));
        const float nm = fmaxf(mx[r], tm);
        base[r] = nm == -INFINITY ? 0.f : nm;
        f[r] = ex2(mx[r] - base[r]);
        mx[r] = nm;
        l[r] *= f[r];
      }
#pragma unroll
      for (int n = 0; n < (int)LP_K / 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          s[n][e] = ex2(s[n][e] - base[e >> 1]);
          l[e >> 1] += s[n][e];
        }
#pragma unroll
      for (int n = 0; n < DV / 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[n][e] *= f[e >> 1];
#pragma unroll
      for (int ks = 0; ks < (int)LP_K / 16; ++ks) {
        const uint32_t pa[4] = {half2_bits(s[2 * ks][0], s[2 * ks][1]), half2_bits(s[2 * ks][2], s[2 * ks][3]),
                                half2_bits(s[2 * ks + 1][0], s[2 * ks + 1][1]), half2_bits(s[2 * ks + 1][2], s[2 * ks + 1][3])};
#pragma unroll
        for (int n = 0; n < DV / 16; ++n) {
          if (n * 16 >= (int)V16) break;
          uint32_t vb[4];
          ldsm_x4_trans(vb, vt + (size_t)(buf * LP_K + ks * 16 + (mat & 1) * 8 + r8) * VB + n * 32 + (mat >> 1) * 16);
          mma16816(o[2 * n], pa, vb[0], vb[1]);
          mma16816(o[2 * n + 1], pa, vb[2], vb[3]);
        }
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
    const uint32_t row = warp * 16 + gq + 8 * r, m = m0 + row;
    if (row >= nq) continue;
#pragma unroll
    for (int n = 0; n < DV / 8; ++n)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const uint32_t c = n * 8 + 2 * tq + e, col = h * a.vdim + c;
        if (c >= a.vdim) continue;
        const float y = o[n][2 * r + e] * inv;
        store_out(out, out_fmt, (size_t)m * ld_out + col, a.gate ? y * a.gate[(size_t)m * a.ld_gate + col] : y);
      }
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
  const int buffers = bytes(2) <= LIMIT ? 2 : 1;
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
template <int DV>
int launch_prefill(cudaStream_t s, const LatArgs &w, const __half *k, const __half *v, void *out, int out_fmt, uint32_t ld_out) {
  constexpr size_t LIMIT = 227 * 1024;
  const uint32_t KB = (up16(w.a.dim) + up16(w.a.rot_dim)) * 2 + 16, VB = up16(w.a.vdim) * 2 + 16;
  auto bytes = [&](uint32_t warps) { return (size_t)warps * 16 * KB + 2 * LP_K * (KB + VB); };
  const uint32_t warps = w.rows.M > 64 && bytes(8) <= LIMIT ? 8 : 4;
  GRETA_REQUIRE(bytes(warps) <= LIMIT, "latent_prefill: head sizes %u + %u / %u need %zu bytes of shared memory", w.a.dim, w.a.rot_dim, w.a.vdim, bytes(warps));
  static bool attr_set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !attr_set[dev]) {
    GRETA_CUDA_TRY(cudaFuncSetAttribute(latent_prefill_kernel<DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)LIMIT));
    attr_set[dev] = true;
  }
  GRETA_CUDA_TRY(launch_pdl(latent_prefill_kernel<DV>, dim3((w.rows.M + warps * 16 - 1) / (warps * 16), w.a.heads), dim3(warps * 32), bytes(warps), s, w, k, v,
                            out, out_fmt, ld_out));
  return launched("latent_prefill_kernel");
}
size_t q_bytes(const greta_latent_attn &a, uint32_t M) {
  return ((size_t)M * a.heads * (up16(a.rank) + up16(a.rot_dim)) * (a.fmt == GRETA_FMT_F32 ? 4 : 2) + 15) / 16 * 16;
}

}  // namespace

extern "C" {

uint32_t greta_cuda_latent_row(uint32_t rank, uint32_t rot_dim) { return up16(rank) + up16(rot_dim); }

int greta_cuda_latent_cache(greta_stream_t stream, const greta_latent_attn *a, const greta_rows *rows) {
  if (int rc = check_latent("latent_cache", a, rows)) return rc;
  const LatArgs w{*a, *rows};
  const dim3 grid((rows->M + 7) / 8);
  if (a->fmt == GRETA_FMT_F16)
    GRETA_CUDA_TRY(launch_pdl(latent_cache_kernel<__half>, grid, dim3(256), 0, (cudaStream_t)stream, w));
  else
    GRETA_CUDA_TRY(launch_pdl(latent_cache_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, w));
  return launched("latent_cache_kernel");
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

int greta_cuda_latent_prefill(greta_stream_t stream, const greta_latent_attn *a, const greta_rows *rows, const void *k, const void *v, void *out,
                              int out_fmt, uint32_t ld_out) {
  if (int rc = check_latent("latent_prefill", a, rows)) return rc;
  GRETA_REQUIRE(!rows->d_pos && k && v && aligned16(k) && aligned16(v) && out && a->q && a->heads <= 65535, "latent_prefill: null pointer, or rows of a batch");
  GRETA_REQUIRE(a->fmt == GRETA_FMT_F16, "latent_prefill: the cache must be F16");
  const LatArgs w{*a, *rows};
  cudaStream_t s = (cudaStream_t)stream;
  const __half *kh = static_cast<const __half *>(k), *vh = static_cast<const __half *>(v);
  if (a->vdim <= 64) return launch_prefill<64>(s, w, kh, vh, out, out_fmt, ld_out);
  if (a->vdim <= 128) return launch_prefill<128>(s, w, kh, vh, out, out_fmt, ld_out);
  return launch_prefill<256>(s, w, kh, vh, out, out_fmt, ld_out);
}

}  // extern "C"
