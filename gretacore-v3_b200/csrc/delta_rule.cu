// Generalised delta rule (recurrent mixer with a matrix state per head), fp32 throughout:
//   S <- diag(w) S - (a * u)(u^T S) + k v^T,  u = k / sqrt(k.k + 1e-6),  o = S^T r.
// The columns of S (one per value channel) do not mix: column j only needs the scalar c_j = k^T S_j of the old state,
//   S_j <- w * S_j + k v_j - ak c_j,   ak = a * k / (k.k + 1e-6),   o_j = r^T S_j,
// so eight lanes hold one column in registers (row i * 32 + lane8 * 4 + e in register 4 i + e) and a step is two dot
// products over eight lanes and one update.  Rows past dim are padding: every vector is zero there, so they stay zero.
//
// The scan takes four tokens at a time, so that one reduction serves four tokens.  With W(a..b) the product of the decays of
// tokens a..b of such a block (0..3) and S the state before it,
//   c_i = (k_i W(0..i-1))^T S_j + sum_{j<i} P_ij v_j - Q_ij c_j          P, Q: (k_i W(j+1..i-1)) . k_j, ... . ak_j
//   o_i = (r_i W(0..i))^T S_j   + sum_{j<=i} R_ij v_j - T_ij c_j         R, T: (r_i W(j+1..i)) . k_j, ... . ak_j
//   S_j <- W(0..3) S_j + sum_i (k_i W(i+1..3)) v_i - (ak_i W(i+1..3)) c_i
// The 17 vectors and 32 scalars of a block are the same for every column; producer warps derive them from the staged
// tokens one chunk ahead of the warps that hold the state.  No decay is ever divided by.
//
// The gated form decays first and writes what the decayed state misses,
//   S <- diag(g) S;  S <- S + bk (v - S^T k)^T,  bk = beta k;  o = S^T q
// so a block needs one set of write vectors and one of pairs: with d_i the row that token i writes,
//   d_i = v_i - (k_i W(0..i))^T S_j - sum_{j<i} P_ij d_j                  P: (k_i W(j+1..i)) . bk_j
//   o_i = (q_i W(0..i))^T S_j + sum_{j<=i} R_ij d_j                       R: (q_i W(j+1..i)) . bk_j
//   S_j <- W(0..3) S_j + sum_i (bk_i W(i+1..3)) d_i
// Thirteen vectors and 16 scalars.  Its key and value sizes differ, value heads may share query / key heads, and q, k, v pass a
// short convolution first (gated_prepare_kernel; in decode inside gated_step_kernel).
#include <algorithm>

#include "dense_device.cuh"

using namespace greta;

namespace {

constexpr uint32_t DR_LANES = 8;
__host__ __device__ constexpr uint32_t dim32(uint32_t d) { return (d + 31u) & ~31u; }

__device__ __forceinline__ float sum8(float v) {  // over the eight lanes of a column
  v += __shfl_xor_sync(0xffffffffu, v, 1);
  v += __shfl_xor_sync(0xffffffffu, v, 2);
  return v + __shfl_xor_sync(0xffffffffu, v, 4);
}
__device__ __forceinline__ float4 lds4(const float *p) { return *reinterpret_cast<const float4 *>(p); }
__device__ __forceinline__ float dot4(const float4 &a, const float4 &b, float acc) {
  acc = fmaf(a.x, b.x, acc);
  acc = fmaf(a.y, b.y, acc);
  acc = fmaf(a.z, b.z, acc);
  return fmaf(a.w, b.w, acc);
}
// S = w S + k v - ak c
__device__ __forceinline__ void update4(float4 &s, const float4 &w, const float4 &k, const float4 &ak, float v, float nc) {
  s.x = fmaf(w.x, s.x, fmaf(k.x, v, ak.x * nc));
  s.y = fmaf(w.y, s.y, fmaf(k.y, v, ak.y * nc));
  s.z = fmaf(w.z, s.z, fmaf(k.z, v, ak.z * nc));
  s.w = fmaf(w.w, s.w, fmaf(k.w, v, ak.w * nc));
}

struct DeltaArgs {
  greta_delta_rule d;
  greta_rows rows;
};

// One token of every sequence: grid (heads, rows).
template <int RB>
__global__ void __launch_bounds__(512) delta_step_kernel(const __grid_constant__ DeltaArgs a, void *out, int out_fmt, uint32_t ld_out) {
  constexpr int DP = RB * 32;
  __shared__ __align__(16) float sk[DP], sw[DP], sak[DP], sr[DP];
  __shared__ float so[DP], red[32];
  extern __shared__ float st[];  // [rank]
  const greta_delta_rule &d = a.d;
  const uint32_t h = blockIdx.x, m = blockIdx.y, D = d.dim, slot = a.rows.slot0 + m;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, l8 = lane & 7;
  const uint32_t nw = blockDim.x >> 5, cols_per_pass = blockDim.x / DR_LANES;
  float *state = d.state + ((size_t)slot * d.heads + h) * D * DP;
  pdl_launch_dependents();
  pdl_wait();
  const bool fresh = a.rows.d_pos[m] == 0;
  for (uint32_t i = threadIdx.x; i < d.rank; i += blockDim.x) st[i] = d.t[(size_t)m * d.ld_t + i];
  const size_t at = (size_t)m * d.ld + (size_t)h * D;
  float kk = 0.f;
  for (uint32_t i = threadIdx.x; i < (uint32_t)DP; i += blockDim.x) {
    const float k = i < D ? d.k[at + i] : 0.f;
    sk[i] = k;
    sak[i] = i < D ? d.a[at + i] * k : 0.f;
    sr[i] = i < D ? d.r[at + i] : 0.f;
    if (i >= D) sw[i] = 0.f;
    kk = fmaf(k, k, kk);
  }
  const float inv2 = 1.f / (block_sum_all(kk, red) + 1e-6f);  // also orders the writes to st
  for (uint32_t c = warp; c < D; c += nw) {
    const float *w2 = d.w2 + ((size_t)h * D + c) * d.rank;
    float z = 0.f;
    for (uint32_t j = lane; j < d.rank; j += 32) z = fmaf(w2[j], st[j], z);
    z = warp_sum(z);
    if (lane == 0) sw[c] = apply_act(GRETA_ACT_DELTA_DECAY, z + d.w0[(size_t)h * D + c]);
  }
  __syncthreads();
  float oo = 0.f;
  for (uint32_t c0 = 0; c0 < D; c0 += cols_per_pass) {
    const uint32_t col = c0 + threadIdx.x / DR_LANES;
    const bool on = col < D;
    float4 s[RB];
    float c = 0.f;
#pragma unroll
    for (int i = 0; i < RB; ++i) {
      const int row = i * 32 + l8 * 4;
      s[i] = on && !fresh ? *reinterpret_cast<const float4 *>(state + (size_t)col * DP + row) : make_float4(0.f, 0.f, 0.f, 0.f);
      c = dot4(lds4(sk + row), s[i], c);
    }
    c = -sum8(c) * inv2;
    const float v = on ? d.v[at + col] : 0.f;
    float o = 0.f;
#pragma unroll
    for (int i = 0; i < RB; ++i) {
      const int row = i * 32 + l8 * 4;
      update4(s[i], lds4(sw + row), lds4(sk + row), lds4(sak + row), v, c);
      o = dot4(lds4(sr + row), s[i], o);
      if (on) *reinterpret_cast<float4 *>(state + (size_t)col * DP + row) = s[i];
    }
    o = sum8(o);
    if (on && l8 == 0) {
      so[col] = o;
      oo = fmaf(o, o, oo);
    }
  }
  const float inv = 1.f / sqrtf(block_sum_all(oo, red) / (float)D + d.eps);
  for (uint32_t i = threadIdx.x; i < D; i += blockDim.x)
    store_out(out, out_fmt, (size_t)m * ld_out + (size_t)h * D + i, so[i] * inv * d.norm[(size_t)h * D + i] * d.gate[at + i]);
}

__device__ __forceinline__ void cp16(void *dst, const void *src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp4(void *dst, const void *src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// What the scan reads, for either form: rows of consecutive tokens.
struct ScanArgs {
  const float *w, *k, *a, *r, *v;  // decay, key, removal rate (general) or write strength per head (gated), receptance / query, value
  uint32_t ld_w, ld_k, ld_a, ld_r, ld_v;
  uint32_t heads, per, dim, vdim;  // per: value heads that share a query / key head
  uint32_t T, pos0, slot;
  float *state;
};

// The recurrence over a portion: grid (heads, column groups).  A CTA keeps COLS columns of one head in the registers of its
// first warps, NC columns per group of eight lanes, and walks the tokens in chunks of TC = a block per producer warp.
template <int RB, int NC, int COLS_, bool GATED>
struct ScanCfg {
  static constexpr int DP = RB * 32, COLS = COLS_;
  static constexpr int TC = RB <= 2 ? 32 : RB <= 4 ? 16 : 8, NB = TC / 4;
  static constexpr int NV = GATED ? 3 : 4;                                      // staged vectors of a token: w, k, (a,) r
  static constexpr int RAW_ROW = NV * DP + COLS + (GATED ? 4 : 0), RAW = TC * RAW_ROW;  // then v (and the write strength)
  static constexpr int VEC = GATED ? 13 : 17, SCAL = VEC * DP, VT = SCAL + (GATED ? 32 : 48);  // {P, -Q | R | -T} or {P | R}, v [column][4]
  static constexpr int BLK = VT + 4 * COLS, DER = NB * BLK;
  static constexpr int CW = COLS / (4 * NC), PW = NB < 4 ? 4 : NB, THREADS = (CW + PW) * 32;
  static constexpr size_t SMEM = (size_t)(2 * RAW + 2 * DER + 2 * TC * COLS) * 4;
  static_assert(SMEM <= 232448, "chunk buffers exceed shared memory");
};
// Four values over the eight lanes of a group: lane l8 receives the total of value l8 >> 1.
__device__ __forceinline__ float sum8_of4(const float (&v)[4], int l8) {
  const bool b4 = l8 & 4, b2 = l8 & 2;
  const float p0 = (b4 ? v[2] : v[0]) + __shfl_xor_sync(0xffffffffu, b4 ? v[0] : v[2], 4);
  const float p1 = (b4 ? v[3] : v[1]) + __shfl_xor_sync(0xffffffffu, b4 ? v[1] : v[3], 4);
  const float q = (b2 ? p1 : p0) + __shfl_xor_sync(0xffffffffu, b2 ? p0 : p1, 2);
  return q + __shfl_xor_sync(0xffffffffu, q, 1);
}
// N = 32 or 16 values over the 32 lanes of a warp: lane l receives the total of value l % N.
template <int N>
__device__ __forceinline__ float sum32_of(float (&v)[N], int lane) {
  if (N == 16) {
#pragma unroll
    for (int j = 0; j < N; ++j) v[j] += __shfl_xor_sync(0xffffffffu, v[j], 16);
  }
#pragma unroll
  for (int n = N / 2; n >= 1; n >>= 1) {
    const bool up = lane & n;
#pragma unroll
    for (int j = 0; j < n; ++j) v[j] = (up ? v[j + n] : v[j]) + __shfl_xor_sync(0xffffffffu, up ? v[j] : v[j + n], n);
  }
  return v[0];
}

template <int RB, int NC, int COLS_, bool GATED>
__global__ void __launch_bounds__(ScanCfg<RB, NC, COLS_, GATED>::THREADS) delta_scan_kernel(const __grid_constant__ ScanArgs a, float *__restrict__ o_buf, int vec) {
  using C = ScanCfg<RB, NC, COLS_, GATED>;
  constexpr int DP = C::DP, TC = C::TC, COLS = C::COLS, NV = C::NV;
  extern __shared__ __align__(16) float sm[];
  float *derived = sm + 2 * C::RAW, *so = derived + 2 * C::DER;  // so: [2][TC][COLS]
  const uint32_t h = blockIdx.x, hk = h / a.per, c0 = blockIdx.y * COLS, D = a.dim, V = a.vdim, T = a.T;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, l8 = lane & 7;
  const bool producer = warp >= C::CW;
  const int pw = warp - C::CW;
  const uint32_t vcols = min((uint32_t)COLS, V - c0), chunks = (T + TC - 1) / TC;
  float *state = a.state + ((size_t)a.slot * a.heads + h) * V * DP;
  for (int i = threadIdx.x; i < 2 * C::RAW + 2 * C::DER; i += C::THREADS) sm[i] = 0.f;
  pdl_launch_dependents();
  pdl_wait();
  __syncthreads();

  auto stage = [&](uint32_t c) {  // producer warps
    if (c < chunks) {
      const uint32_t t0 = c * TC, n = min((uint32_t)TC, T - t0);
      float *b = sm + (c & 1) * C::RAW;
      for (uint32_t t = pw; t < n; t += C::PW) {
        const size_t m = t0 + t;
        float *dst = b + t * C::RAW_ROW;
        const float *k = a.k + m * a.ld_k + (size_t)hk * D, *r = a.r + m * a.ld_r + (size_t)hk * D;
        const float *src[4] = {a.w + m * a.ld_w + (size_t)h * D, k, GATED ? r : a.a + m * a.ld_a + (size_t)h * D, r};
        const float *v = a.v + m * a.ld_v + (size_t)h * V + c0;
        if (GATED && lane == 0) cp4(dst + NV * DP + COLS, a.a + m * a.ld_a + h);
        if (vec) {
#pragma unroll
          for (int i = 0; i < NV; ++i)
#pragma unroll
            for (int j = 0; j < (DP + 127) / 128; ++j)
              if (lane * 4 + j * 128 < (int)D) cp16(dst + i * DP + lane * 4 + j * 128, src[i] + lane * 4 + j * 128);
          if (lane * 4 < (int)vcols) cp16(dst + NV * DP + lane * 4, v + lane * 4);
        } else {
#pragma unroll
          for (int i = 0; i < NV; ++i)
            for (uint32_t e = lane; e < D; e += 32) cp4(dst + i * DP + e, src[i] + e);
          if (lane < (int)vcols) cp4(dst + NV * DP + lane, v + lane);
        }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto landed = [&]() {  // the chunk before the last one staged is complete for every producer
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    asm volatile("bar.sync 1, %0;" ::"n"(C::PW * 32) : "memory");
  };
  auto prepare = [&](uint32_t c) {  // producer warp pw: block pw of the chunk, once it has landed
    if (c >= chunks || pw >= C::NB) return;
    const int n = (int)min((uint32_t)TC, T - c * TC) - pw * 4;  // tokens of the block that exist; the others leave the state as it is
    const float *raw = sm + (c & 1) * C::RAW + pw * 4 * C::RAW_ROW;
    float *der = derived + (c & 1) * C::DER + pw * C::BLK;
    float inv2[4];  // general: 1 / (k.k + 1e-6); gated: the write strength
#pragma unroll
    for (int t = 0; t < 4; ++t) {
      if (GATED) {
        inv2[t] = raw[t * C::RAW_ROW + NV * DP + COLS];
        continue;
      }
      float kk = 0.f;
#pragma unroll
      for (int i = 0; i < RB; ++i) {
        const float k = raw[t * C::RAW_ROW + DP + i * 32 + lane];
        kk = fmaf(k, k, kk);
      }
      inv2[t] = kk;
    }
    if (!GATED)
#pragma unroll
      for (int t = 0; t < 4; ++t) inv2[t] = 1.f / (warp_sum(inv2[t]) + 1e-6f);
    constexpr int PAIRS = GATED ? 16 : 32;
    float acc[PAIRS];
#pragma unroll
    for (int j = 0; j < PAIRS; ++j) acc[j] = 0.f;
#pragma unroll
    for (int i = 0; i < RB; ++i) {
      const int e = i * 32 + lane;
      float w[4], k[4], ak[4], r[4];
#pragma unroll
      for (int t = 0; t < 4; ++t) {
        const float *row = raw + t * C::RAW_ROW + e;
        const bool on = t < n;
        w[t] = on ? row[0] : 1.f;
        k[t] = on ? row[DP] : 0.f;
        ak[t] = on ? (GATED ? 1.f : row[2 * DP]) * k[t] * inv2[t] : 0.f;
        r[t] = on ? row[(NV - 1) * DP] : 0.f;
      }
      const float w01 = w[0] * w[1], w12 = w[1] * w[2], w23 = w[2] * w[3], w02 = w01 * w[2], w13 = w12 * w[3];
      float *o = der + e;
      // left factors of the pairs (i, j): (1,0) (2,0) (2,1) (3,0) (3,1) (3,2); and with the diagonal (0,0) (1,0) (1,1) (2,0) .. (3,3)
      constexpr int pj[6] = {0, 0, 1, 0, 1, 2}, rj[10] = {0, 0, 1, 0, 1, 2, 0, 1, 2, 3};
      const float rl[10] = {r[0], r[1] * w[1], r[1], r[2] * w12, r[2] * w[2], r[2], r[3] * w13, r[3] * w23, r[3] * w[3], r[3]};
      o[4 * DP] = r[0] * w[0], o[5 * DP] = r[1] * w01, o[6 * DP] = r[2] * w02, o[7 * DP] = r[3] * (w02 * w[3]);
      o[8 * DP] = w[0] * w13;
      if constexpr (GATED) {
        o[0] = k[0] * w[0], o[DP] = k[1] * w01, o[2 * DP] = k[2] * w02, o[3 * DP] = k[3] * (w02 * w[3]);
        o[9 * DP] = ak[0] * w13, o[10 * DP] = ak[1] * w23, o[11 * DP] = ak[2] * w[3], o[12 * DP] = ak[3];
        const float pl[6] = {k[1] * w[1], k[2] * w12, k[2] * w[2], k[3] * w13, k[3] * w23, k[3] * w[3]};
#pragma unroll
        for (int x = 0; x < 6; ++x) acc[x] = fmaf(pl[x], ak[pj[x]], acc[x]);
#pragma unroll
        for (int x = 0; x < 10; ++x) acc[6 + x] = fmaf(rl[x], ak[rj[x]], acc[6 + x]);
      } else {
        o[0] = k[0], o[DP] = k[1] * w[0], o[2 * DP] = k[2] * w01, o[3 * DP] = k[3] * w02;
        o[9 * DP] = k[0] * w13, o[10 * DP] = k[1] * w23, o[11 * DP] = k[2] * w[3], o[12 * DP] = k[3];
        o[13 * DP] = -ak[0] * w13, o[14 * DP] = -ak[1] * w23, o[15 * DP] = -ak[2] * w[3], o[16 * DP] = -ak[3];
        const float pl[6] = {k[1], k[2] * w[1], k[2], k[3] * w12, k[3] * w[2], k[3]};
#pragma unroll
        for (int x = 0; x < 6; ++x) {
          acc[x] = fmaf(pl[x], k[pj[x]], acc[x]);
          acc[6 + x] = fmaf(-pl[x], ak[pj[x]], acc[6 + x]);
        }
#pragma unroll
        for (int x = 0; x < 10; ++x) {
          acc[12 + x] = fmaf(rl[x], k[rj[x]], acc[12 + x]);
          acc[22 + x] = fmaf(-rl[x], ak[rj[x]], acc[22 + x]);
        }
      }
    }
    const float total = sum32_of<PAIRS>(acc, lane);
    constexpr int FIRST = GATED ? 6 : 12;  // then the lower triangles; their upper halves stay zero
    const int x = lane < FIRST ? 0 : (lane - FIRST) % 10, ri = x < 1 ? 0 : x < 3 ? 1 : x < 6 ? 2 : 3;
    if (lane < PAIRS) der[C::SCAL + (lane < FIRST ? lane : (lane < FIRST + 10 ? 16 : 32) + ri * 4 + x - ri * (ri + 1) / 2)] = total;
    const float *v = raw + NV * DP + lane;
    if (lane < COLS) *reinterpret_cast<float4 *>(der + C::VT + lane * 4) = make_float4(v[0], v[C::RAW_ROW], v[2 * C::RAW_ROW], v[3 * C::RAW_ROW]);
  };
  auto write_back = [&](uint32_t c) {
    const uint32_t n = min((uint32_t)TC, T - c * TC);
    const float *src = so + (c & 1) * TC * COLS;
    for (uint32_t t = pw; t < n; t += C::PW)
      if (lane < (int)vcols) o_buf[((size_t)(c * TC + t) * a.heads + h) * V + c0 + lane] = src[t * COLS + lane];
  };

  const int grp = threadIdx.x >> 3;  // state warps: columns c0 + grp * NC ..
  float4 s[NC][RB];
  if (producer) {
    stage(0);
    stage(1);
    landed();
    prepare(0);
  } else {
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const uint32_t col = c0 + grp * NC + c;
#pragma unroll
      for (int i = 0; i < RB; ++i) {
        s[c][i] = col < V && a.pos0 ? *reinterpret_cast<const float4 *>(state + (size_t)col * DP + i * 32 + l8 * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
    }
  }
  __syncthreads();
  for (uint32_t ch = 0; ch < chunks; ++ch) {
    if (producer) {
      stage(ch + 2);
      landed();
      prepare(ch + 1);
      if (ch) write_back(ch - 1);
    } else {
      float *out = so + (ch & 1) * TC * COLS;
#pragma unroll 1
      for (int blk = 0; blk < C::NB; ++blk) {
        const float *b = derived + (ch & 1) * C::DER + blk * C::BLK;
        float x[NC][4], o[NC][4];
#pragma unroll
        for (int c = 0; c < NC; ++c)
#pragma unroll
          for (int t = 0; t < 4; ++t) x[c][t] = o[c][t] = 0.f;
#pragma unroll
        for (int i = 0; i < RB; ++i)
#pragma unroll
          for (int t = 0; t < 4; ++t) {
            const float4 k = lds4(b + t * DP + i * 32 + l8 * 4), r = lds4(b + (4 + t) * DP + i * 32 + l8 * 4);
#pragma unroll
            for (int c = 0; c < NC; ++c) {
              x[c][t] = dot4(k, s[c][i], x[c][t]);
              o[c][t] = dot4(r, s[c][i], o[c][t]);
            }
          }
        // P10 P20 P21 P30 | P31 P32 -Q10 -Q20 | -Q21 -Q30 -Q31 -Q32
        const float4 s0 = lds4(b + C::SCAL), s1 = lds4(b + C::SCAL + 4);
        const float4 R = lds4(b + C::SCAL + 16 + (l8 >> 1) * 4);  // of this lane's token
        float4 s2, Tn;
        if constexpr (!GATED) s2 = lds4(b + C::SCAL + 8), Tn = lds4(b + C::SCAL + 32 + (l8 >> 1) * 4);
        float4 v[NC], cc[NC];  // gated: cc are the written rows d
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          v[c] = lds4(b + C::VT + (grp * NC + c) * 4);
          const float q = sum8_of4(x[c], l8);
          const int base = lane & 24;
          const float q0 = __shfl_sync(0xffffffffu, q, base), q1 = __shfl_sync(0xffffffffu, q, base + 2);
          const float q2 = __shfl_sync(0xffffffffu, q, base + 4), q3 = __shfl_sync(0xffffffffu, q, base + 6);
          if constexpr (GATED) {
            cc[c].x = v[c].x - q0;
            cc[c].y = fmaf(-s0.x, cc[c].x, v[c].y - q1);
            cc[c].z = fmaf(-s0.z, cc[c].y, fmaf(-s0.y, cc[c].x, v[c].z - q2));
            cc[c].w = fmaf(-s1.y, cc[c].z, fmaf(-s1.x, cc[c].y, fmaf(-s0.w, cc[c].x, v[c].w - q3)));
          } else {
            cc[c].x = q0;
            cc[c].y = fmaf(s1.z, cc[c].x, fmaf(s0.x, v[c].x, q1));
            cc[c].z = fmaf(s2.x, cc[c].y, fmaf(s1.w, cc[c].x, fmaf(s0.z, v[c].y, fmaf(s0.y, v[c].x, q2))));
            const float p3 = fmaf(s1.y, v[c].z, fmaf(s1.x, v[c].y, fmaf(s0.w, v[c].x, q3)));
            cc[c].w = fmaf(s2.w, cc[c].z, fmaf(s2.z, cc[c].y, fmaf(s2.y, cc[c].x, p3)));
          }
        }
#pragma unroll
        for (int i = 0; i < RB; ++i) {
          const int at = i * 32 + l8 * 4;
          const float4 w = lds4(b + 8 * DP + at);
#pragma unroll
          for (int c = 0; c < NC; ++c) s[c][i] = make_float4(w.x * s[c][i].x, w.y * s[c][i].y, w.z * s[c][i].z, w.w * s[c][i].w);
#pragma unroll
          for (int t = 0; t < 4; ++t) {
            const float4 k = lds4(b + (9 + t) * DP + at);
            float4 ak;
            if constexpr (!GATED) ak = lds4(b + (13 + t) * DP + at);
#pragma unroll
            for (int c = 0; c < NC; ++c) {
              const float vt = t == 0 ? v[c].x : t == 1 ? v[c].y : t == 2 ? v[c].z : v[c].w;
              const float ct = t == 0 ? cc[c].x : t == 1 ? cc[c].y : t == 2 ? cc[c].z : cc[c].w;
              if constexpr (GATED) {
                s[c][i].x = fmaf(k.x, ct, s[c][i].x);
                s[c][i].y = fmaf(k.y, ct, s[c][i].y);
                s[c][i].z = fmaf(k.z, ct, s[c][i].z);
                s[c][i].w = fmaf(k.w, ct, s[c][i].w);
              } else {
                s[c][i].x = fmaf(ak.x, ct, fmaf(k.x, vt, s[c][i].x));
                s[c][i].y = fmaf(ak.y, ct, fmaf(k.y, vt, s[c][i].y));
                s[c][i].z = fmaf(ak.z, ct, fmaf(k.z, vt, s[c][i].z));
                s[c][i].w = fmaf(ak.w, ct, fmaf(k.w, vt, s[c][i].w));
              }
            }
          }
        }
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          float y = sum8_of4(o[c], l8);
          if constexpr (GATED) {
            y = fmaf(R.x, cc[c].x, fmaf(R.y, cc[c].y, fmaf(R.z, cc[c].z, fmaf(R.w, cc[c].w, y))));
          } else {
            y = fmaf(R.x, v[c].x, fmaf(R.y, v[c].y, fmaf(R.z, v[c].z, fmaf(R.w, v[c].w, y))));
            y = fmaf(Tn.x, cc[c].x, fmaf(Tn.y, cc[c].y, fmaf(Tn.z, cc[c].z, fmaf(Tn.w, cc[c].w, y))));
          }
          if (!(l8 & 1)) out[(blk * 4 + (l8 >> 1)) * COLS + grp * NC + c] = y;
        }
      }
    }
    __syncthreads();
  }
  if (producer) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    write_back(chunks - 1);
  } else {
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const uint32_t col = c0 + grp * NC + c;
#pragma unroll
      for (int i = 0; i < RB; ++i)
        if (col < V) *reinterpret_cast<float4 *>(state + (size_t)col * DP + i * 32 + l8 * 4) = s[c][i];
    }
  }
}

// Norm over every head's outputs, norm weight and gate: LPH lanes per (row, head), each with its channels in registers
// (four consecutive ones at a time where the sizes allow it).
struct OutArgs {
  const float *gate, *norm;  // [M][heads * dim] rows ld_gate apart; one weight per channel of every head, or (shared) of one head
  uint32_t ld_gate, heads, dim, M;
  int shared;
  float eps;
};
template <int LPH, bool VEC>
__global__ void __launch_bounds__(256) delta_output_kernel(const __grid_constant__ OutArgs d, const float *__restrict__ o_buf, void *out, int out_fmt,
                                                           uint32_t ld_out) {
  constexpr int PER = VEC ? 4 : 1, MAXU = VEC ? 2 : 8;  // units per lane: LPH * MAXU * PER >= 256 channels for the widest heads
  pdl_launch_dependents();
  pdl_wait();
  const uint32_t i = (blockIdx.x * 256 + threadIdx.x) / LPH, l = threadIdx.x % LPH, D = d.dim;
  const bool on = i < d.M * d.heads;
  const uint32_t m = on ? i / d.heads : 0, h = on ? i % d.heads : 0;
  const float *o = o_buf + (size_t)(on ? i : 0) * D;
  float v[MAXU][PER], q = 0.f;
#pragma unroll
  for (int u = 0; u < MAXU; ++u) {
    const uint32_t c = (u * LPH + l) * PER;
#pragma unroll
    for (int e = 0; e < PER; ++e) v[u][e] = 0.f;
    if (on && c < D) {
      if (VEC) {
        const float4 t = *reinterpret_cast<const float4 *>(o + c);
        v[u][0] = t.x, v[u][PER > 1 ? 1 : 0] = t.y, v[u][PER > 1 ? 2 : 0] = t.z, v[u][PER > 1 ? 3 : 0] = t.w;
      } else {
        v[u][0] = o[c];
      }
    }
#pragma unroll
    for (int e = 0; e < PER; ++e) q = fmaf(v[u][e], v[u][e], q);
  }
#pragma unroll
  for (int off = LPH / 2; off > 0; off >>= 1) q += __shfl_xor_sync(0xffffffffu, q, off);
  const float inv = 1.f / sqrtf(q / (float)D + d.eps);
#pragma unroll
  for (int u = 0; u < MAXU; ++u) {
    const uint32_t c = (u * LPH + l) * PER;
    if (!on || c >= D) continue;
    float y[PER];
    const float *g = d.gate + (size_t)m * d.ld_gate + h * D + c, *n = d.norm + (d.shared ? 0 : (size_t)h * D) + c;
#pragma unroll
    for (int e = 0; e < PER; ++e) y[e] = v[u][e] * inv * n[e] * g[e];
    const size_t at = (size_t)m * ld_out + h * D + c;
    if (VEC && out_fmt == GRETA_OUT_BF16) {
      const __nv_bfloat162 lo = __floats2bfloat162_rn(y[0], y[PER > 1 ? 1 : 0]), hi = __floats2bfloat162_rn(y[PER > 2 ? 2 : 0], y[PER > 3 ? 3 : 0]);
      uint2 w;
      w.x = *reinterpret_cast<const uint32_t *>(&lo);
      w.y = *reinterpret_cast<const uint32_t *>(&hi);
      *reinterpret_cast<uint2 *>(static_cast<__nv_bfloat16 *>(out) + at) = w;
    } else {
#pragma unroll
      for (int e = 0; e < PER; ++e) store_out(out, out_fmt, at + e, y[e]);
    }
  }
}

// ---- gated form: what enters the recurrence, and one token per sequence
struct GatedArgs {
  greta_gated_delta d;
  greta_rows rows;
};
__device__ __forceinline__ float silu(float z) { return __fdividef(z, 1.f + expf(-z)); }
// Projected channel c of sequence `slot` at position p - back: from the launch's rows (m is the row of position p, rows of this
// sequence start at position first) or from the history; zero in front of the sequence.
__device__ __forceinline__ float channel_at(const greta_gated_delta &d, uint32_t C, uint32_t slot, uint32_t m, uint32_t p, uint32_t first, uint32_t back,
                                            uint32_t c) {
  if (back > p) return 0.f;
  const uint32_t q = p - back;
  return q >= first ? d.proj[(size_t)(m - back) * d.ld_proj + c] : d.history[((size_t)slot * d.taps + q % d.taps) * C + c];
}

// A warp takes one head unit (query heads, key heads, value heads) through GP_ROWS consecutive rows.  TAPS > 0: the convolution's
// weights and its window stay in registers, every projected value is read once; TAPS 0: any number of taps, window re-read.
constexpr int GP_ROWS = 16;
template <int TAPS, int CH>
__global__ void __launch_bounds__(256) gated_prepare_kernel(const __grid_constant__ GatedArgs a) {
  constexpr int W = TAPS > 0 ? TAPS : 1;
  const greta_gated_delta &d = a.d;
  const uint32_t u = blockIdx.x * 8 + (threadIdx.x >> 5), m0 = blockIdx.y * GP_ROWS, m1 = min(m0 + GP_ROWS, a.rows.M), slot = a.rows.slot0;
  const int lane = threadIdx.x & 31;
  const uint32_t G = d.kv_heads, C = 2 * G * d.dim + d.heads * d.vdim;
  if (u >= 2 * G + d.heads) return;
  const bool is_v = u >= 2 * G;
  const uint32_t n = is_v ? d.vdim : d.dim, c0 = (is_v ? 2 * G * d.dim + (u - 2 * G) * d.vdim : u * d.dim) + lane;
  const float after = u < G ? 1.f / sqrtf((float)d.dim) : 1.f;
  float cw[CH][W], win[CH][W];  // win[.][j]: the projected value W - 1 - j rows back
  pdl_launch_dependents();
  pdl_wait();
  if (TAPS)
#pragma unroll
    for (int i = 0; i < CH; ++i)
#pragma unroll
      for (int j = 0; j < W; ++j) {
        const bool on = lane + 32 * i < (int)n;
        cw[i][j] = on ? d.conv[(size_t)(c0 + 32 * i) * W + j] : 0.f;
        win[i][j] = on && j < W - 1 ? channel_at(d, C, slot, m0, a.rows.pos0 + m0, a.rows.pos0, W - 1 - j, c0 + 32 * i) : 0.f;
      }
  constexpr int RG = 4;  // rows of a group; the next group's loads are in flight while one is computed
  float cur[RG][CH];
  auto load = [&](uint32_t m) {
#pragma unroll
    for (int r = 0; r < RG; ++r)
#pragma unroll
      for (int i = 0; i < CH; ++i) cur[r][i] = m + r < m1 && lane + 32 * i < (int)n ? d.proj[(size_t)(m + r) * d.ld_proj + c0 + 32 * i] : 0.f;
  };
  if (TAPS) load(m0);
  for (uint32_t m = m0; m < m1; m += RG) {
    float v[RG][CH], q[RG];
#pragma unroll
    for (int r = 0; r < RG; ++r) {
      q[r] = 0.f;
#pragma unroll
      for (int i = 0; i < CH; ++i) {
        float y = 0.f;
        if (TAPS) {
          win[i][W - 1] = cur[r][i];
#pragma unroll
          for (int j = 0; j < W; ++j) y = fmaf(cw[i][j], win[i][j], y);
#pragma unroll
          for (int j = 0; j + 1 < W; ++j) win[i][j] = win[i][j + 1];
        } else if (m + r < m1 && lane + 32 * i < (int)n) {
          for (uint32_t j = 0; j < d.taps; ++j)
            y = fmaf(d.conv[(size_t)(c0 + 32 * i) * d.taps + j], channel_at(d, C, slot, m + r, a.rows.pos0 + m + r, a.rows.pos0, d.taps - 1 - j, c0 + 32 * i), y);
        }
        v[r][i] = y;
      }
    }
    if (TAPS) load(m + RG);
#pragma unroll
    for (int r = 0; r < RG; ++r)
#pragma unroll
      for (int i = 0; i < CH; ++i) {
        v[r][i] = lane + 32 * i < (int)n ? silu(v[r][i]) : 0.f;
        q[r] = fmaf(v[r][i], v[r][i], q[r]);
      }
    if (!is_v) {
#pragma unroll
      for (int r = 0; r < RG; ++r) q[r] = after / sqrtf(warp_sum(q[r]) + 1e-6f);
    }
#pragma unroll
    for (int r = 0; r < RG; ++r)
#pragma unroll
      for (int i = 0; i < CH; ++i)
        if (m + r < m1 && lane + 32 * i < (int)n) d.u[(size_t)(m + r) * d.ld_u + c0 + 32 * i] = is_v ? v[r][i] : v[r][i] * q[r];
  }
}
__global__ void gated_history_kernel(const __grid_constant__ GatedArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const greta_gated_delta &d = a.d;
  const uint32_t C = 2 * d.kv_heads * d.dim + d.heads * d.vdim, c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= C) return;
  const uint32_t m = a.rows.M - 1 - blockIdx.y, p = a.rows.pos0 + m;  // grid.y <= min(M, taps): distinct history rows
  d.history[((size_t)a.rows.slot0 * d.taps + p % d.taps) * C + c] = d.proj[(size_t)m * d.ld_proj + c];
}

// Eight lanes: W[row] . t over n columns; every lane of the group receives the total.
__device__ __forceinline__ float row_dot8(const float *w, const float *t, uint32_t n, int l8) {
  float z = 0.f;
  if (n % 4 == 0) {
#pragma unroll 4
    for (uint32_t j = l8 * 4; j < n; j += 32) z = dot4(*reinterpret_cast<const float4 *>(w + j), make_float4(t[j], t[j + 1], t[j + 2], t[j + 3]), z);
  } else {
    for (uint32_t j = l8; j < n; j += 8) z = fmaf(w[j], t[j], z);
  }
  return sum8(z);
}
// One token of every sequence: grid (heads, rows).
template <int RB>
__global__ void __launch_bounds__(512) gated_step_kernel(const __grid_constant__ GatedArgs a, void *out, int out_fmt, uint32_t ld_out) {
  constexpr int DP = RB * 32;
  __shared__ __align__(16) float sq[DP], sk[DP], sw[DP];
  __shared__ float sv[256], so[256], sg[256], red[32];
  extern __shared__ float low[];  // [rank_a | rank_g]
  const greta_gated_delta &d = a.d;
  const uint32_t h = blockIdx.x, m = blockIdx.y, D = d.dim, V = d.vdim, G = d.kv_heads, per = d.heads / G, hk = h / per, slot = a.rows.slot0 + m;
  const int l8 = threadIdx.x & 7;
  const uint32_t C = 2 * G * D + d.heads * V, groups = blockDim.x / DR_LANES, grp = threadIdx.x / DR_LANES;
  float *state = d.state + ((size_t)slot * d.heads + h) * V * DP;
  const float *a2 = d.a2 + (size_t)h * D * d.rank_a, *g2 = d.g2 + (size_t)h * V * d.rank_g;
  for (uint32_t b = threadIdx.x * 32; b < D * d.rank_a; b += blockDim.x * 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(a2 + b));
  for (uint32_t b = threadIdx.x * 32; b < V * d.rank_g; b += blockDim.x * 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(g2 + b));
  for (uint32_t b = threadIdx.x * 32; b < V * DP; b += blockDim.x * 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(state + b));
  pdl_launch_dependents();
  pdl_wait();
  const uint32_t p = a.rows.d_pos[m];
  const bool fresh = p == 0;
  for (uint32_t i = threadIdx.x; i < d.rank_a + d.rank_g; i += blockDim.x)
    low[i] = d.low[(size_t)m * d.ld_low + (i < d.rank_a ? i : d.low_g + i - d.rank_a)];
  float qq = 0.f, kk = 0.f;
  for (uint32_t e = threadIdx.x; e < 2 * D + V; e += blockDim.x) {
    const uint32_t c = e < D ? hk * D + e : e < 2 * D ? (G + hk) * D + e - D : 2 * G * D + h * V + e - 2 * D;
    float y = 0.f, cur = 0.f;
#pragma unroll 4
    for (uint32_t j = 0; j < d.taps; ++j) {
      const float x = channel_at(d, C, slot, m, p, p, d.taps - 1 - j, c);
      y = fmaf(d.conv[(size_t)c * d.taps + j], x, y);
      cur = x;
    }
    y = silu(y);
    if (e < D) sq[e] = y, qq = fmaf(y, y, qq);
    else if (e < 2 * D) sk[e - D] = y, kk = fmaf(y, y, kk);
    else sv[e - 2 * D] = y;
    if (d.taps > 1 && (e >= 2 * D || h % per == 0)) d.history[((size_t)slot * d.taps + p % d.taps) * C + c] = cur;
  }
  for (uint32_t i = D + threadIdx.x; i < (uint32_t)DP; i += blockDim.x) sq[i] = sk[i] = sw[i] = 0.f;
  const float qi = 1.f / (sqrtf(block_sum_all(qq, red) + 1e-6f) * sqrtf((float)D)), ki = 1.f / sqrtf(block_sum_all(kk, red) + 1e-6f);
  for (uint32_t r0 = 0; r0 < D + V; r0 += groups) {  // decays and gates, eight lanes each; whole warps take part
    const uint32_t r = r0 + grp;
    const bool dec = r < D;
    const float *w = dec ? a2 + (size_t)r * d.rank_a : g2 + (size_t)min(r - D, V - 1) * d.rank_g;
    const float z = row_dot8(w, dec ? low : low + d.rank_a, dec ? d.rank_a : d.rank_g, l8);
    if (l8 == 0 && dec) sw[r] = apply_act(GRETA_ACT_SOFTPLUS_DECAY, z + d.dt_bias[(size_t)h * D + r], d.rate[(size_t)h * D + r]);
    else if (l8 == 0 && r < D + V) sg[r - D] = act_sigmoid(z);
  }
  const float beta = d.beta[(size_t)m * d.ld_beta + h];
  __syncthreads();
  float oo = 0.f;
  for (uint32_t c0 = 0; c0 < V; c0 += groups) {
    const uint32_t col = c0 + grp;
    const bool on = col < V;
    float4 s[RB];
    float c = 0.f;
#pragma unroll
    for (int i = 0; i < RB; ++i) {
      const int row = i * 32 + l8 * 4;
      s[i] = on && !fresh ? *reinterpret_cast<const float4 *>(state + (size_t)col * DP + row) : make_float4(0.f, 0.f, 0.f, 0.f);
      const float4 w = lds4(sw + row);
      s[i] = make_float4(w.x * s[i].x, w.y * s[i].y, w.z * s[i].z, w.w * s[i].w);
      c = dot4(lds4(sk + row), s[i], c);
    }
    c = sum8(c) * ki;
    const float u = on ? beta * (sv[col] - c) * ki : 0.f;
    float o = 0.f;
#pragma unroll
    for (int i = 0; i < RB; ++i) {
      const int row = i * 32 + l8 * 4;
      const float4 k = lds4(sk + row);
      s[i] = make_float4(fmaf(k.x, u, s[i].x), fmaf(k.y, u, s[i].y), fmaf(k.z, u, s[i].z), fmaf(k.w, u, s[i].w));
      o = dot4(lds4(sq + row), s[i], o);
      if (on) *reinterpret_cast<float4 *>(state + (size_t)col * DP + row) = s[i];
    }
    o = sum8(o) * qi;
    if (on && l8 == 0) {
      so[col] = o;
      oo = fmaf(o, o, oo);
    }
  }
  const float inv = 1.f / sqrtf(block_sum_all(oo, red) / (float)V + d.eps);
  for (uint32_t i = threadIdx.x; i < V; i += blockDim.x)
    store_out(out, out_fmt, (size_t)m * ld_out + (size_t)h * V + i, so[i] * inv * d.norm[i] * sg[i]);
}

int check_gated(const char *what, const greta_gated_delta *d, const greta_rows *r) {
  GRETA_REQUIRE(d && r && r->M, "%s: null or empty argument", what);
  GRETA_REQUIRE(d->heads && d->kv_heads && d->heads % d->kv_heads == 0, "%s: %u value heads over %u query / key heads", what, d->heads, d->kv_heads);
  GRETA_REQUIRE(d->dim && d->dim <= 256 && d->vdim && d->vdim <= 256, "%s: head sizes %u / %u (1..256)", what, d->dim, d->vdim);
  GRETA_REQUIRE(d->taps && (d->taps == 1 || d->history) && d->state && aligned16(d->state), "%s: no convolution, history or state", what);
  return GRETA_OK;
}
template <int RB>
int launch_gated_step(cudaStream_t s, const GatedArgs &a, void *out, int out_fmt, uint32_t ld_out) {
  const uint32_t threads = std::min(512u, (std::max(a.d.dim, a.d.vdim) * DR_LANES + 31) / 32 * 32);
  GRETA_CUDA_TRY(launch_pdl(gated_step_kernel<RB>, dim3(a.d.heads, a.rows.M), dim3(threads), (size_t)(a.d.rank_a + a.d.rank_g) * 4, s, a, out, out_fmt, ld_out));
  return launched("gated_step_kernel");
}
template <int TAPS, int CH>
int launch_prepare(cudaStream_t s, const GatedArgs &a) {
  const dim3 grid((2 * a.d.kv_heads + a.d.heads + 7) / 8, (a.rows.M + GP_ROWS - 1) / GP_ROWS);
  GRETA_CUDA_TRY(launch_pdl(gated_prepare_kernel<TAPS, CH>, grid, dim3(256), 0, s, a));
  return launched("gated_prepare_kernel");
}
template <int CH>
int pick_prepare(cudaStream_t s, const GatedArgs &a) {
  switch (a.d.taps) {
    case 2: return launch_prepare<2, CH>(s, a);
    case 3: return launch_prepare<3, CH>(s, a);
    case 4: return launch_prepare<4, CH>(s, a);
    default: return launch_prepare<0, CH>(s, a);
  }
}

int check_delta(const char *what, const greta_delta_rule *d, const greta_rows *r) {
  GRETA_REQUIRE(d && r && r->M, "%s: null or empty argument", what);
  GRETA_REQUIRE(d->heads && d->dim && d->dim <= 256, "%s: %u heads of %u channels (1..256)", what, d->heads, d->dim);
  return GRETA_OK;
}

template <int RB, int NC, int COLS, bool GATED>
int launch_scan(cudaStream_t s, const ScanArgs &a, float *o_buf, int vec) {
  using C = ScanCfg<RB, NC, COLS, GATED>;
  // A grid that fits the SMs asks for more than half of an SM's shared memory: CTAs that become resident while the previous
  // kernel drains would otherwise pair up on the SMs that fall idle first, and the pairs would set the pace.
  constexpr size_t ALONE = 118 * 1024;
  static bool attr_set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !attr_set[dev]) {
    GRETA_CUDA_TRY(cudaFuncSetAttribute(delta_scan_kernel<RB, NC, COLS, GATED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)std::max(C::SMEM, ALONE)));
    attr_set[dev] = true;
  }
  const dim3 grid(a.heads, (a.vdim + C::COLS - 1) / C::COLS);
  const size_t smem = grid.x * grid.y <= (uint32_t)sm_count() ? std::max(C::SMEM, ALONE) : C::SMEM;
  GRETA_CUDA_TRY(launch_pdl(delta_scan_kernel<RB, NC, COLS, GATED>, grid, dim3(C::THREADS), smem, s, a, o_buf, vec));
  return launched("delta_scan_kernel");
}
template <bool GATED>
int pick_scan(cudaStream_t s, const ScanArgs &a, float *o_buf) {
  const int vec = a.dim % 4 == 0 && a.vdim % 4 == 0 && a.ld_w % 4 == 0 && a.ld_k % 4 == 0 && a.ld_r % 4 == 0 && a.ld_v % 4 == 0 && aligned16(a.w) &&
                  aligned16(a.k) && aligned16(a.r) && aligned16(a.v) && (GATED || (a.ld_a % 4 == 0 && aligned16(a.a)));
  // Few heads: half the columns per CTA where the doubled grid still has an SM for every CTA (the usual head sizes).
  const bool narrow = a.heads * ((a.vdim + 15) / 16) <= (uint32_t)sm_count();
  switch (dim32(a.dim) / 32) {
    case 1: return launch_scan<1, 2, 32, GATED>(s, a, o_buf, vec);
    case 2: return narrow ? launch_scan<2, 1, 16, GATED>(s, a, o_buf, vec) : launch_scan<2, 2, 32, GATED>(s, a, o_buf, vec);
    case 3: return launch_scan<3, 2, 32, GATED>(s, a, o_buf, vec);
    case 4: return narrow ? launch_scan<4, 1, 16, GATED>(s, a, o_buf, vec) : launch_scan<4, 2, 32, GATED>(s, a, o_buf, vec);
    case 5: return launch_scan<5, 1, 32, GATED>(s, a, o_buf, vec);
    case 6: return launch_scan<6, 1, 32, GATED>(s, a, o_buf, vec);
    case 7: return launch_scan<7, 1, 32, GATED>(s, a, o_buf, vec);
    default: return launch_scan<8, 1, 32, GATED>(s, a, o_buf, vec);
  }
}
int launch_output(cudaStream_t s, const OutArgs &a, const float *o_buf, void *out, int out_fmt, uint32_t ld_out) {
  const uint32_t D = a.dim, pairs = a.M * a.heads;
  const bool vec = D % 4 == 0 && a.ld_gate % 4 == 0 && ld_out % 4 == 0 && aligned16(o_buf) && aligned16(a.gate) && aligned16(a.norm) && aligned16(out);
  auto grid = [&](uint32_t lanes) { return dim3((pairs + 256 / lanes - 1) / (256 / lanes)); };
  if (vec && D <= 64)
    GRETA_CUDA_TRY(launch_pdl(delta_output_kernel<16, true>, grid(16), dim3(256), 0, s, a, o_buf, out, out_fmt, ld_out));
  else if (vec)
    GRETA_CUDA_TRY(launch_pdl(delta_output_kernel<32, true>, grid(32), dim3(256), 0, s, a, o_buf, out, out_fmt, ld_out));
  else
    GRETA_CUDA_TRY(launch_pdl(delta_output_kernel<32, false>, grid(32), dim3(256), 0, s, a, o_buf, out, out_fmt, ld_out));
  return launched("delta_output_kernel");
}
template <int RB>
int launch_step(cudaStream_t s, const DeltaArgs &a, void *out, int out_fmt, uint32_t ld_out) {
  const uint32_t threads = std::min(512u, (a.d.dim * DR_LANES + 31) / 32 * 32);
  GRETA_CUDA_TRY(launch_pdl(delta_step_kernel<RB>, dim3(a.d.heads, a.rows.M), dim3(threads), (size_t)a.d.rank * 4, s, a, out, out_fmt, ld_out));
  return launched("delta_step_kernel");
}

}  // namespace

extern "C" {

size_t greta_cuda_delta_state_bytes(uint32_t heads, uint32_t dim) { return (size_t)heads * dim * dim32(dim) * 4; }

int greta_cuda_delta_step(greta_stream_t stream, const greta_delta_rule *d, const greta_rows *rows, void *out, int out_fmt, uint32_t ld_out) {
  if (int rc = check_delta("delta_step", d, rows)) return rc;
  GRETA_REQUIRE(rows->d_pos && out && d->r && d->k && d->v && d->a && d->gate && d->t && d->w2 && d->w0 && d->norm && d->state,
                "delta_step: null pointer");
  GRETA_REQUIRE(d->rank >= 1 && d->rank <= 8192 && rows->M <= 65535, "delta_step: rank %u", d->rank);
  GRETA_REQUIRE(aligned16(d->state), "delta_step: misaligned state");
  const DeltaArgs a{*d, *rows};
  cudaStream_t s = (cudaStream_t)stream;
  switch (dim32(d->dim) / 32) {
    case 1: return launch_step<1>(s, a, out, out_fmt, ld_out);
    case 2: return launch_step<2>(s, a, out, out_fmt, ld_out);
    case 3: return launch_step<3>(s, a, out, out_fmt, ld_out);
    case 4: return launch_step<4>(s, a, out, out_fmt, ld_out);
    case 5: return launch_step<5>(s, a, out, out_fmt, ld_out);
    case 6: return launch_step<6>(s, a, out, out_fmt, ld_out);
    case 7: return launch_step<7>(s, a, out, out_fmt, ld_out);
    default: return launch_step<8>(s, a, out, out_fmt, ld_out);
  }
}

int greta_cuda_delta_scan(greta_stream_t stream, const greta_delta_rule *d, const greta_rows *rows, float *o_buf) {
  if (int rc = check_delta("delta_scan", d, rows)) return rc;
  GRETA_REQUIRE(!rows->d_pos && o_buf && d->r && d->k && d->v && d->a && d->decay && d->state, "delta_scan: null pointer, or rows of a batch");
  GRETA_REQUIRE(aligned16(d->state), "delta_scan: misaligned state");
  return pick_scan<false>((cudaStream_t)stream, ScanArgs{d->decay, d->k, d->a, d->r, d->v, d->ld_decay, d->ld, d->ld, d->ld, d->ld, d->heads, 1, d->dim, d->dim,
                                                        rows->M, rows->pos0, rows->slot0, d->state}, o_buf);
}

int greta_cuda_delta_output(greta_stream_t stream, const greta_delta_rule *d, const float *o_buf, uint32_t M, void *out, int out_fmt, uint32_t ld_out) {
  const greta_rows rows{M, 0, 0, nullptr};
  if (int rc = check_delta("delta_output", d, &rows)) return rc;
  GRETA_REQUIRE(o_buf && out && d->norm && d->gate, "delta_output: null pointer");
  return launch_output((cudaStream_t)stream, OutArgs{d->gate, d->norm, d->ld, d->heads, d->dim, M, 0, d->eps}, o_buf, out, out_fmt, ld_out);
}

size_t greta_cuda_gated_delta_state_bytes(uint32_t heads, uint32_t dim, uint32_t vdim) { return (size_t)heads * vdim * dim32(dim) * 4; }

int greta_cuda_gated_delta_step(greta_stream_t stream, const greta_gated_delta *d, const greta_rows *rows, void *out, int out_fmt, uint32_t ld_out) {
  if (int rc = check_gated("gated_delta_step", d, rows)) return rc;
  GRETA_REQUIRE(rows->d_pos && rows->M <= 65535 && out && d->proj && d->conv && d->beta && d->low && d->a2 && d->g2 && d->rate && d->dt_bias && d->norm,
                "gated_delta_step: null pointer");
  GRETA_REQUIRE(d->rank_a && d->rank_g && d->rank_a + d->rank_g <= 8192, "gated_delta_step: low-rank widths %u and %u", d->rank_a, d->rank_g);
  const GatedArgs a{*d, *rows};
  cudaStream_t s = (cudaStream_t)stream;
  switch (dim32(d->dim) / 32) {
    case 1: return launch_gated_step<1>(s, a, out, out_fmt, ld_out);
    case 2: return launch_gated_step<2>(s, a, out, out_fmt, ld_out);
    case 3: return launch_gated_step<3>(s, a, out, out_fmt, ld_out);
    case 4: return launch_gated_step<4>(s, a, out, out_fmt, ld_out);
    case 5: return launch_gated_step<5>(s, a, out, out_fmt, ld_out);
    case 6: return launch_gated_step<6>(s, a, out, out_fmt, ld_out);
    case 7: return launch_gated_step<7>(s, a, out, out_fmt, ld_out);
    default: return launch_gated_step<8>(s, a, out, out_fmt, ld_out);
  }
}

int greta_cuda_gated_delta_prepare(greta_stream_t stream, const greta_gated_delta *d, const greta_rows *rows) {
  if (int rc = check_gated("gated_delta_prepare", d, rows)) return rc;
  GRETA_REQUIRE(!rows->d_pos && d->proj && d->conv && d->u && rows->M <= 16u * 65535u, "gated_delta_prepare: null pointer, or rows of a batch");
  const GatedArgs a{*d, *rows};
  cudaStream_t s = (cudaStream_t)stream;
  const uint32_t wide = std::max(d->dim, d->vdim);
  if (int rc = wide <= 64 ? pick_prepare<2>(s, a) : wide <= 128 ? pick_prepare<4>(s, a) : pick_prepare<8>(s, a)) return rc;
  if (d->taps == 1) return GRETA_OK;
  const uint32_t C = 2 * d->kv_heads * d->dim + d->heads * d->vdim;
  GRETA_CUDA_TRY(launch_pdl(gated_history_kernel, dim3((C + 255) / 256, std::min(rows->M, d->taps)), dim3(256), 0, s, a));
  return launched("gated_history_kernel");
}

int greta_cuda_gated_delta_scan(greta_stream_t stream, const greta_gated_delta *d, const greta_rows *rows, float *o_buf) {
  if (int rc = check_gated("gated_delta_scan", d, rows)) return rc;
  GRETA_REQUIRE(!rows->d_pos && o_buf && d->u && d->beta && d->decay, "gated_delta_scan: null pointer, or rows of a batch");
  const uint32_t GD = d->kv_heads * d->dim;
  return pick_scan<true>((cudaStream_t)stream, ScanArgs{d->decay, d->u + GD, d->beta, d->u, d->u + 2 * GD, d->ld_decay, d->ld_u, d->ld_beta, d->ld_u, d->ld_u,
                                                       d->heads, d->heads / d->kv_heads, d->dim, d->vdim, rows->M, rows->pos0, rows->slot0, d->state}, o_buf);
}

int greta_cuda_gated_delta_output(greta_stream_t stream, const greta_gated_delta *d, const float *o_buf, uint32_t M, void *out, int out_fmt, uint32_t ld_out) {
  const greta_rows rows{M, 0, 0, nullptr};
  if (int rc = check_gated("gated_delta_output", d, &rows)) return rc;
  GRETA_REQUIRE(o_buf && out && d->norm && d->gate, "gated_delta_output: null pointer");
  return launch_output((cudaStream_t)stream, OutArgs{d->gate, d->norm, d->ld_gate, d->heads, d->vdim, M, 1, d->eps}, o_buf, out, out_fmt, ld_out);
}

}  // extern "C"
