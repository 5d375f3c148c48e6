// Dense linears on many activation rows (prompts and long portions).
//
// bf16 or fp16: tensor cores.  The weight rows are the 128-row operand of tcgen05.mma and TN tokens its N dimension, so a thread
// of the epilogue owns one weight row (one segment, one bias) and a warp stores 32 consecutive outputs of a token.
// Persistent CTAs, one per SM, walk the tiles with the token tiles innermost: the CTAs in flight share a few weight row
// tiles, which are read from HBM once.  Roles (320 threads): warp 0 TMA producer of both operands (128-byte swizzle, 64
// columns per stage), warp 1 MMA issuer (one lane), warps 2-9 epilogue, two per TMEM lane quadrant.  Two accumulators in
// TMEM: a tile's epilogue runs under the next tile's MMAs.  Every mbarrier wait is bounded (see
// greta_cuda_linear_gemm_status).
// Where there are fewer tiles than SMs, a cluster of 2, 4 or 8 CTAs shares a tile's K loop: every CTA leaves its partial
// tile in its shared memory and finishes a share of the tokens, adding the partial sums in rank order through distributed
// shared memory.
//
// fp32: plain 64 x 64 tiles of 32-bit FMAs, for models that run in 32-bit.
#include <cooperative_groups.h>

#include <algorithm>

#include "dense_device.cuh"
#include "tc_device.cuh"

using namespace greta;

namespace greta {
int check_linear(const char *what, const greta_linear *l, Segments *sg);
cudaError_t latent_wait_status(int *code);
}

namespace {

template <int TN>
struct DCfg {
  static constexpr int A_BYTES = TILE_N * BK * 2, B_BYTES = TN * BK * 2, STAGE = A_BYTES + B_BYTES;
  static constexpr int ST = TN == 256 ? 4 : TN == 128 ? 6 : 8;
  static constexpr int COLS = 2 * TN < 32 ? 32 : 2 * TN;  // two accumulators; a power of two
  static constexpr int EPI_WARPS = TN >= 64 ? 8 : 4;
  static constexpr int THREADS = 64 + EPI_WARPS * 32;
  static constexpr size_t SMEM = (size_t)ST * STAGE + 1024 + 256;
  static_assert(COLS <= 512 && SMEM <= 232448, "tile configuration");
};

// 32 consecutive tokens (from m on, cnt of them present) of one weight row per lane: bias, activation, store.  All lanes call; those
// past the last row are off.  PAIRED (16-bit outputs): neighbouring lanes hold neighbouring columns of one segment and exchange every
// other token, so that each stores two columns at a time.
template <int ACT>
__device__ __forceinline__ void finish_row_act(const greta_out_segment &g, uint32_t r, float bias, uint32_t m, uint32_t cnt, const uint32_t (&v)[32], bool on,
                                               bool paired) {
  const size_t base = (size_t)m * g.ld + g.col0 + r;
  const float rate = ACT == GRETA_ACT_SOFTPLUS_DECAY && on ? __ldg(g.rate + r) : 0.f;
  if (paired) {
    const uint32_t odd = threadIdx.x & 1;
    uint32_t *o = reinterpret_cast<uint32_t *>(static_cast<uint16_t *>(g.out) + base + (size_t)odd * g.ld - odd);
    const bool half = g.out_fmt == GRETA_OUT_F16;
#pragma unroll
    for (int j = 0; j < 32; j += 2) {
      const float x = apply_act(ACT, __uint_as_float(v[j]) + bias, rate), y = apply_act(ACT, __uint_as_float(v[j + 1]) + bias, rate);
      const float other = __shfl_xor_sync(0xffffffffu, odd ? x : y, 1);
      const float lo = odd ? other : x, hi = odd ? y : other;
      uint32_t bits;
      if (half) {
        const __half2 h = __floats2half2_rn(lo, hi);
        bits = *reinterpret_cast<const uint32_t *>(&h);
      } else {
        const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
        bits = *reinterpret_cast<const uint32_t *>(&h);
      }
      if (j + odd < cnt) o[(size_t)(j / 2) * g.ld] = bits;
    }
    return;
  }
  if (!on) return;
  if (g.accumulate) {
    float *o = static_cast<float *>(g.out) + base;
    float old[32];
#pragma unroll
    for (int j = 0; j < 32; ++j) old[j] = j < cnt ? o[(size_t)j * g.ld] : 0.f;
#pragma unroll
    for (int j = 0; j < 32; ++j)
      if (j < cnt) o[(size_t)j * g.ld] = old[j] + apply_act(ACT, __uint_as_float(v[j]) + bias, rate);
  } else if (g.out_fmt == GRETA_OUT_F32) {
    float *o = static_cast<float *>(g.out) + base;
#pragma unroll
    for (int j = 0; j < 32; ++j)
      if (j < cnt) o[(size_t)j * g.ld] = apply_act(ACT, __uint_as_float(v[j]) + bias, rate);
  } else {
#pragma unroll
    for (int j = 0; j < 32; ++j)
      if (j < cnt) store_out(g.out, g.out_fmt, base + (size_t)j * g.ld, apply_act(ACT, __uint_as_float(v[j]) + bias, rate), g.pair_offset);
  }
}
__device__ __forceinline__ void finish_row(const greta_out_segment &g, uint32_t r, float bias, uint32_t m, uint32_t cnt, const uint32_t (&v)[32], bool on,
                                           bool paired) {
  switch (g.act) {
    case GRETA_ACT_GELU_ERF: finish_row_act<GRETA_ACT_GELU_ERF>(g, r, bias, m, cnt, v, on, paired); break;
    case GRETA_ACT_SIGMOID: finish_row_act<GRETA_ACT_SIGMOID>(g, r, bias, m, cnt, v, on, paired); break;
    case GRETA_ACT_TANH: finish_row_act<GRETA_ACT_TANH>(g, r, bias, m, cnt, v, on, paired); break;
    case GRETA_ACT_DELTA_DECAY: finish_row_act<GRETA_ACT_DELTA_DECAY>(g, r, bias, m, cnt, v, on, paired); break;
    case GRETA_ACT_RELU2: finish_row_act<GRETA_ACT_RELU2>(g, r, bias, m, cnt, v, on, paired); break;
    case GRETA_ACT_SOFTPLUS_DECAY: finish_row_act<GRETA_ACT_SOFTPLUS_DECAY>(g, r, bias, m, cnt, v, on, paired); break;
    default: finish_row_act<GRETA_ACT_NONE>(g, r, bias, m, cnt, v, on, paired); break;
  }
}
// The whole warp's 32 rows can be stored in pairs: one segment with 16-bit outputs, even columns on even lanes.
__device__ __forceinline__ bool rows_paired(const greta_out_segment &g, uint32_t r, int segment, bool on) {
  const bool same = __shfl_sync(0xffffffffu, segment, 0) == segment;
  const bool fits = on && (g.out_fmt == GRETA_OUT_F16 || g.out_fmt == GRETA_OUT_BF16) && g.ld % 2 == 0 && ((g.col0 + r + threadIdx.x) & 1) == 0 &&
                    (reinterpret_cast<uintptr_t>(g.out) & 3) == 0;
  return __all_sync(0xffffffffu, same && fits);
}

// A copy still in flight must not outlive the CTA: after an abort the producer gives the last ones a bounded chance to land.
__device__ __forceinline__ void drain_copies(uint64_t *full, uint32_t issued, uint32_t stages) {
  for (uint32_t j = issued > stages ? issued - stages : 0; j < issued; ++j) {
    const long long t0 = clock64();
    while (!mbar_try_wait(&full[j % stages], (j / stages) & 1) && clock64() - t0 < 20000000ll) {
    }
  }
}

template <int TN>
__global__ void __launch_bounds__(DCfg<TN>::THREADS, 1)
linear_tc_kernel(const __grid_constant__ CUtensorMap tmap_w, const __grid_constant__ CUtensorMap tmap_x, const __grid_constant__ Segments sg, uint32_t M,
                 uint32_t N, uint32_t K, uint32_t idesc) {
  using C = DCfg<TN>;
  constexpr int ST = C::ST;
  extern __shared__ uint8_t smem_raw[];
  uint8_t *smem = reinterpret_cast<uint8_t *>(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  uint64_t *bars = reinterpret_cast<uint64_t *>(smem + (size_t)ST * C::STAGE);
  uint64_t *full = bars, *empty = bars + ST, *acc_full = bars + 2 * ST, *acc_empty = acc_full + 2;
  uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(acc_empty + 2);
  volatile int *abort_flag = reinterpret_cast<volatile int *>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t KT = (K + BK - 1) / BK, tok_tiles = (M + TN - 1) / TN, tiles = tok_tiles * ((N + TILE_N - 1) / TILE_N);

  if (threadIdx.x == 0) {
    for (int s = 0; s < ST; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    for (int b = 0; b < 2; ++b) {
      mbar_init(&acc_full[b], 1);
      mbar_init(&acc_empty[b], C::EPI_WARPS);
    }
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tmap_w) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tmap_x) : "memory");
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, C::COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  pdl_launch_dependents();
  pdl_wait();

  if (warp == 0) {
    if (lane == 0) {
      uint32_t issued = 0, s = 0, ph = 1;
      bool ok = true;
      for (uint32_t t = blockIdx.x; t < tiles && ok; t += gridDim.x) {
        const int n0 = (int)(t / tok_tiles) * TILE_N, m0 = (int)(t % tok_tiles) * TN;
        for (uint32_t kt = 0; kt < KT; ++kt) {
          ok = mbar_wait(&empty[s], ph, abort_flag, 100 + s);
          if (!ok) break;
          uint8_t *st = smem + (size_t)s * C::STAGE;
          mbar_arrive_expect_tx(&full[s], C::STAGE);
          tma_load_2d(st, &tmap_w, (int)(kt * BK), n0, &full[s]);
          tma_load_2d(st + C::A_BYTES, &tmap_x, (int)(kt * BK), m0, &full[s]);
          ++issued;
          if (++s == ST) {
            s = 0;
            ph ^= 1;
          }
        }
      }
      if (*abort_flag) drain_copies(full, issued, ST);
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t lo0 = smem_desc_lo(smem_u32(smem));
      uint32_t s = 0, ph = 0, it = 0;
      bool ok = true;
      for (uint32_t t = blockIdx.x; t < tiles && ok; t += gridDim.x, ++it) {
        const uint32_t b = it & 1;
        ok = mbar_wait(&acc_empty[b], ((it >> 1) & 1) ^ 1, abort_flag, 300 + b);
        if (!ok) break;
        tc_fence_after();
        for (uint32_t kt = 0; kt < KT; ++kt) {
          ok = mbar_wait(&full[s], ph, abort_flag, 200 + s);
          if (!ok) break;
          tc_fence_after();
          const uint32_t w_lo = lo0 + s * (C::STAGE >> 4), x_lo = w_lo + (C::A_BYTES >> 4);
#pragma unroll
          for (int k16 = 0; k16 < BK / 16; ++k16)
            umma_f16(tmem_base + b * TN, w_lo + k16 * 2, x_lo + k16 * 2, SMEM_DESC_HI_SW128, idesc, (kt | k16) ? 1u : 0u);
          umma_commit(&empty[s]);
          if (++s == ST) {
            s = 0;
            ph ^= 1;
          }
        }
        if (ok) umma_commit(&acc_full[b]);
      }
    }
  } else {
    constexpr int SHARE = TN / (C::EPI_WARPS / 4);  // tokens per warp
    const int quad = warp & 3, c_begin = ((warp - 2) >> 2) * SHARE;
    uint32_t it = 0;
    for (uint32_t t = blockIdx.x; t < tiles; t += gridDim.x, ++it) {
      const uint32_t b = it & 1, m0 = (t % tok_tiles) * TN, row = (t / tok_tiles) * TILE_N + quad * 32 + lane;
      greta_out_segment g{};
      uint32_t r = 0;
      float bias = 0.f;
      int which = -1;
      if (row < N) {
        which = segment_of(sg, row);
        g = sg.s[which];
        r = row - g.row0;
        if (g.bias) bias = __ldg(g.bias + r);
      }
      const bool paired = rows_paired(g, r, which, row < N);
      if (!mbar_wait(&acc_full[b], (it >> 1) & 1, abort_flag, 400 + b)) break;
      tc_fence_after();
#pragma unroll 1
      for (int c = c_begin; c < c_begin + SHARE; c += 32) {
        uint32_t v[32];
        __syncwarp();
        if (m0 + c < M) {
          tmem_ld32(tmem_base + ((uint32_t)(quad * 32) << 16) + b * TN + c, v);
          tmem_ld_wait();
        }
        if (c + 32 >= c_begin + SHARE) {  // this warp's share is read: the issuer may overwrite it
          tc_fence_before();
          __syncwarp();
          if (lane == 0) mbar_arrive(&acc_empty[b]);
        }
        if (m0 + c < M) finish_row(g, r, bias, m0 + c, min(32u, M - m0 - c), v, row < N, paired);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, C::COLS);
  }
}

// One tile per cluster, its K loop shared by the cluster's CTAs.  Same roles; warps 2-9 first leave the partial tile
// [token][128 rows] in the idle ring, then finish tokens rank * TN / S ...
template <int TN>
__global__ void __launch_bounds__(DCfg<TN>::THREADS, 1)
linear_tc_split_kernel(const __grid_constant__ CUtensorMap tmap_w, const __grid_constant__ CUtensorMap tmap_x, const __grid_constant__ Segments sg,
                       uint32_t M, uint32_t N, uint32_t K, uint32_t idesc) {
  namespace cg = cooperative_groups;
  using C = DCfg<TN>;
  constexpr int ST = C::ST, COLS = TN < 32 ? 32 : TN;
  static_assert((size_t)TN * TILE_N * 4 <= (size_t)ST * C::STAGE, "the partial tile reuses the ring");
  cg::cluster_group cl = cg::this_cluster();
  const uint32_t S = cl.num_blocks(), rank = cl.block_rank();
  extern __shared__ uint8_t smem_raw[];
  uint8_t *smem = reinterpret_cast<uint8_t *>(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  uint64_t *bars = reinterpret_cast<uint64_t *>(smem + (size_t)ST * C::STAGE);
  uint64_t *full = bars, *empty = bars + ST, *acc_full = bars + 2 * ST;
  uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(acc_full + 1);
  volatile int *abort_flag = reinterpret_cast<volatile int *>(tmem_slot + 1);
  float *part = reinterpret_cast<float *>(smem);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t KT = (K + BK - 1) / BK, tok_tiles = (M + TN - 1) / TN, tile = blockIdx.x / S;
  const uint32_t n0 = (tile / tok_tiles) * TILE_N, m0 = (tile % tok_tiles) * TN;
  const uint32_t kt0 = KT * rank / S, kt1 = KT * (rank + 1) / S;  // the plan leaves every CTA some stages

  if (threadIdx.x == 0) {
    for (int s = 0; s < ST; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    mbar_init(acc_full, 1);
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tmap_w) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(&tmap_x) : "memory");
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  pdl_launch_dependents();
  pdl_wait();

  if (warp == 0) {
    if (lane == 0) {
      uint32_t issued = 0, s = 0, ph = 1;
      for (uint32_t kt = kt0; kt < kt1; ++kt) {
        if (!mbar_wait(&empty[s], ph, abort_flag, 100 + s)) break;
        uint8_t *st = smem + (size_t)s * C::STAGE;
        mbar_arrive_expect_tx(&full[s], C::STAGE);
        tma_load_2d(st, &tmap_w, (int)(kt * BK), (int)n0, &full[s]);
        tma_load_2d(st + C::A_BYTES, &tmap_x, (int)(kt * BK), (int)m0, &full[s]);
        ++issued;
        if (++s == ST) {
          s = 0;
          ph ^= 1;
        }
      }
      if (*abort_flag) drain_copies(full, issued, ST);
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t lo0 = smem_desc_lo(smem_u32(smem));
      uint32_t s = 0, ph = 0;
      bool ok = true;
      for (uint32_t kt = kt0; kt < kt1; ++kt) {
        ok = mbar_wait(&full[s], ph, abort_flag, 200 + s);
        if (!ok) break;
        tc_fence_after();
        const uint32_t w_lo = lo0 + s * (C::STAGE >> 4), x_lo = w_lo + (C::A_BYTES >> 4);
#pragma unroll
        for (int k16 = 0; k16 < BK / 16; ++k16)
          umma_f16(tmem_base, w_lo + k16 * 2, x_lo + k16 * 2, SMEM_DESC_HI_SW128, idesc, (kt > kt0 || k16) ? 1u : 0u);
        umma_commit(&empty[s]);
        if (++s == ST) {
          s = 0;
          ph ^= 1;
        }
      }
      if (ok) umma_commit(acc_full);
    }
  } else {
    constexpr int SHARE = TN / (C::EPI_WARPS / 4);
    const int quad = warp & 3, c_begin = ((warp - 2) >> 2) * SHARE;
    if (mbar_wait(acc_full, 0, abort_flag, 400)) {  // every stage has been loaded and multiplied: the ring is idle
      tc_fence_after();
#pragma unroll 1
      for (int c = c_begin; c < c_begin + SHARE; c += 32) {
        uint32_t v[32];
        __syncwarp();
        tmem_ld32(tmem_base + ((uint32_t)(quad * 32) << 16) + c, v);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 32; ++j) part[(size_t)(c + j) * TILE_N + quad * 32 + lane] = __uint_as_float(v[j]);
      }
    }
  }
  tc_fence_before();
  __syncwarp();
  cl.sync();
  if (warp >= 2) {
    const uint32_t per = TN / S, wq = (warp - 2) & 3, half = (warp - 2) >> 2, halves = C::EPI_WARPS / 4;
    const uint32_t row_l = wq * 32 + lane, row = n0 + row_l;
    if (row < N) {
      const greta_out_segment g = sg.s[segment_of(sg, row)];
      constexpr int U = 8;  // tokens whose partial sums (and old values) are in flight together
      for (uint32_t j = half; j < per; j += halves * U) {
        const uint32_t c = rank * per + j, m = m0 + c;
        float z[U], old[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
          z[u] = old[u] = 0.f;
          if (g.accumulate && j + u * halves < per && m + u * halves < M) old[u] = static_cast<float *>(g.out)[(size_t)(m + u * halves) * g.ld + g.col0 + row - g.row0];
        }
        for (uint32_t q = 0; q < S; ++q) {
          const float *from = cl.map_shared_rank(part + (size_t)c * TILE_N + row_l, q);
#pragma unroll
          for (int u = 0; u < U; ++u)
            if (j + u * halves < per) z[u] += from[(size_t)u * halves * TILE_N];
        }
#pragma unroll
        for (int u = 0; u < U; ++u)
          if (j + u * halves < per && m + u * halves < M) store_segment(g, row, m + u * halves, z[u], old[u]);
      }
    }
  }
  __syncwarp();
  cl.sync();  // no CTA leaves while another reads its shared memory
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, COLS);
  }
}

// C tile 64 rows of x x 64 rows of W, 256 threads, 4 x 4 outputs each, 16 columns per step.
__global__ void __launch_bounds__(256) linear_f32_kernel(const float *__restrict__ W, uint32_t N, uint32_t ldw, const float *__restrict__ x, uint32_t ldx,
                                                         uint32_t M, const __grid_constant__ Segments sg) {
  __shared__ float ws[16][68], xs[16][68];
  pdl_launch_dependents();
  pdl_wait();
  const uint32_t n0 = blockIdx.x * 64, m0 = blockIdx.y * 64;
  const uint32_t lr = threadIdx.x >> 2, lc = (threadIdx.x & 3) * 4;  // loads: row, column group
  const uint32_t tn = (threadIdx.x & 15) * 4, tm = (threadIdx.x >> 4) * 4;
  const float *wp = W + (size_t)min(n0 + lr, N - 1) * ldw + lc, *xp = x + (size_t)min(m0 + lr, M - 1) * ldx + lc;
  float acc[4][4] = {};
  for (uint32_t k = 0; k < ldw; k += 16) {
    const float4 a = *reinterpret_cast<const float4 *>(wp + k), b = *reinterpret_cast<const float4 *>(xp + k);
    __syncthreads();
    ws[lc][lr] = a.x, ws[lc + 1][lr] = a.y, ws[lc + 2][lr] = a.z, ws[lc + 3][lr] = a.w;
    xs[lc][lr] = b.x, xs[lc + 1][lr] = b.y, xs[lc + 2][lr] = b.z, xs[lc + 3][lr] = b.w;
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < 16; ++kk) {
      const float4 p = *reinterpret_cast<const float4 *>(&ws[kk][tn]), q = *reinterpret_cast<const float4 *>(&xs[kk][tm]);
      const float pn[4] = {p.x, p.y, p.z, p.w}, qm[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(qm[i], pn[j], acc[i][j]);
    }
  }
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const uint32_t row = n0 + tn + j;
    if (row >= N) continue;
    const greta_out_segment &g = sg.s[segment_of(sg, row)];
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (m0 + tm + i < M) store_segment(g, row, m0 + tm + i, acc[i][j]);
  }
}

int make_map(CUtensorMap *map, int fmt, const void *base, uint32_t cols, uint32_t rows, uint32_t ld, uint32_t box_rows) {
  EncodeTiledFn enc = encode_tiled();
  if (!enc) {
    set_error("linear_gemm: cuTensorMapEncodeTiled is not available from this driver");
    return GRETA_ERR_NOT_IMPLEMENTED;
  }
  const cuuint64_t dims[2] = {cols, rows}, strides[1] = {(cuuint64_t)ld * 2};
  const cuuint32_t box[2] = {BK, box_rows}, estr[2] = {1, 1};
  const CUresult r = enc(map, fmt == GRETA_FMT_F16 ? CU_TENSOR_MAP_DATA_TYPE_FLOAT16 : CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                         CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) {
    set_error("linear_gemm: cuTensorMapEncodeTiled failed with code %d", (int)r);
    return GRETA_ERR_INVALID_ARGS;
  }
  return GRETA_OK;
}

template <int TN>
int launch_dense(cudaStream_t s, const greta_linear *l, const Segments &sg, const void *x, uint32_t ldx, uint32_t M, uint32_t split) {
  using C = DCfg<TN>;
  static bool attr_set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !attr_set[dev]) {
    GRETA_CUDA_TRY(cudaFuncSetAttribute(linear_tc_kernel<TN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)C::SMEM));
    GRETA_CUDA_TRY(cudaFuncSetAttribute(linear_tc_split_kernel<TN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)C::SMEM));
    attr_set[dev] = true;
  }
  CUtensorMap mw, mx;
  if (int rc = make_map(&mw, l->fmt, l->w, l->K, l->N, l->ldw, TILE_N)) return rc;  // columns past K read as zero in both operands
  if (int rc = make_map(&mx, l->fmt, x, l->K, M, ldx, TN)) return rc;
  const uint32_t tiles = ((l->N + TILE_N - 1) / TILE_N) * ((M + TN - 1) / TN);
  const uint32_t idesc = l->fmt == GRETA_FMT_F16 ? instr_desc_f16(TILE_N, TN) : instr_desc_bf16(TILE_N, TN);  // both operands are of one type
  if (split > 1) {
    GRETA_CUDA_TRY(launch_pdl_cluster(linear_tc_split_kernel<TN>, dim3(tiles * split), dim3(C::THREADS), split, C::SMEM, s, mw, mx, sg, M, l->N, l->K, idesc));
    return launched("linear_tc_split_kernel");
  }
  GRETA_CUDA_TRY(launch_pdl(linear_tc_kernel<TN>, dim3(std::min(tiles, (uint32_t)sm_count())), dim3(C::THREADS), C::SMEM, s, mw, mx, sg, M, l->N, l->K, idesc));
  return launched("linear_tc_kernel");
}

// Clusters of `split` CTAs (one per SM) that the device runs at the same time: a GPC's SMs may not divide by the cluster size.
uint32_t resident_clusters(uint32_t split) {
  static uint32_t known[64][4] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  uint32_t *n = &known[dev & 63][split == 2 ? 1 : split == 4 ? 2 : 3];
  if (*n == 0) {
    using C = DCfg<32>;
    cudaFuncSetAttribute(linear_tc_split_kernel<32>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)C::SMEM);
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3((uint32_t)sm_count() / split * split);
    cfg.blockDim = dim3(C::THREADS);
    cfg.dynamicSmemBytes = C::SMEM;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = split;
    attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    int got = 0;
    if (cudaOccupancyMaxActiveClusters(&got, linear_tc_split_kernel<32>, &cfg) != cudaSuccess || got < 1) {
      cudaGetLastError();
      got = sm_count() / (int)split;
    }
    *n = (uint32_t)got;
  }
  return *n;
}

// Token tile and K split for a product: the pair with the smallest estimate of its time.  Of one SM, in ns: a stage's bytes from L2 (all
// SMs share about 13.5 TB/s, one takes up to 170 GB/s) or its products, whichever takes longer; the last tile's epilogue; and, for a split,
// the exchange of the partial tiles.
void plan_dense(uint32_t M, uint32_t N, uint32_t K, uint32_t *tn, uint32_t *split) {
  const uint32_t row_tiles = (N + TILE_N - 1) / TILE_N, KT = (K + BK - 1) / BK, sms = (uint32_t)sm_count();
  float best = 0.f;
  for (uint32_t t : {256u, 128u, 64u, 32u}) {
    if (t > 32 && M <= t / 2) continue;  // mostly padding
    const uint32_t tiles = row_tiles * ((M + t - 1) / t);
    for (uint32_t s = 1; s <= 8; s *= 2) {
      if (s > 1 && (tiles * s > sms || KT < s * 3)) break;
      const uint32_t at_once = s == 1 ? sms : resident_clusters(s), ctas = std::min(tiles, at_once) * s, rounds = (tiles + at_once - 1) / at_once;
      const float bytes = TILE_N * BK * 2 + (float)t * BK * 2, rate = std::min(170.f, 13500.f / ctas);
      const float stage = std::max(bytes / rate, t * 1.5f);
      const float ns = rounds * (float)((KT + s - 1) / s) * stage + (s == 1 ? t * (t >= 64 ? 11.f : 20.f) : 1500.f + t * 20.f / s);
      if (best == 0.f || ns < best) best = ns, *tn = t, *split = s;
    }
  }
}

}  // namespace

extern "C" {

int greta_cuda_linear_gemm(greta_stream_t stream, const greta_linear *l, const void *x, uint32_t ldx, uint32_t M) {
  if (M == 0) return GRETA_OK;
  Segments sg{};
  if (int rc = check_linear("linear_gemm", l, &sg)) return rc;
  GRETA_REQUIRE(x && aligned16(x), "linear_gemm: null or misaligned activations");
  cudaStream_t s = (cudaStream_t)stream;
  if (l->fmt == GRETA_FMT_F32) {
    GRETA_REQUIRE(ldx >= l->ldw && ldx % 4 == 0, "linear_gemm: fp32 activations need rows of ldw=%u columns (ldx=%u)", l->ldw, ldx);
    GRETA_CUDA_TRY(launch_pdl(linear_f32_kernel, dim3((l->N + 63) / 64, (M + 63) / 64), dim3(256), 0, s, static_cast<const float *>(l->w), l->N, l->ldw,
                              static_cast<const float *>(x), ldx, M, sg));
    return launched("linear_f32_kernel");
  }
  GRETA_REQUIRE(ldx >= l->K && ldx % 8 == 0, "linear_gemm: ldx=%u K=%u", ldx, l->K);
  uint32_t tn = 32, split = 1;
  plan_dense(M, l->N, l->K, &tn, &split);
  if (tn == 256) return launch_dense<256>(s, l, sg, x, ldx, M, split);
  if (tn == 128) return launch_dense<128>(s, l, sg, x, ldx, M, split);
  if (tn == 64) return launch_dense<64>(s, l, sg, x, ldx, M, split);
  return launch_dense<32>(s, l, sg, x, ldx, M, split);
}

int greta_cuda_linear_gemm_status(int *code) {
  GRETA_REQUIRE(code, "linear_gemm_status: null out pointer");
  GRETA_CUDA_TRY(cudaMemcpyFromSymbol(code, g_gemm_error, sizeof(int)));
  if (*code == 0) GRETA_CUDA_TRY(latent_wait_status(code));
  return GRETA_OK;
}

}  // extern "C"
