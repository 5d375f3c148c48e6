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

// The recurrence over a portion: grid (heads, column groups).  A CTA keeps 32 columns of one head in the registers of its
// first warps, NC columns per group of eight lanes, and walks the tokens in chunks of TC = a block per producer warp.
template <int RB, int NC>
struct ScanCfg {
  static constexpr int DP = RB * 32, COLS = 32;
  static constexpr int TC = RB <= 2 ? 32 : RB <= 4 ? 16 : 8, NB = TC / 4;
  static constexpr int RAW_ROW = 4 * DP + COLS, RAW = TC * RAW_ROW;   // a staged token: w, k, a, r, v
  static constexpr int SCAL = 17 * DP, VT = SCAL + 48;                // of a block: 17 vectors, {P, -Q | R | -T}, v [column][4]
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
// 32 values over the 32 lanes of a warp: lane l receives the total of value l.
__device__ __forceinline__ float sum32_of32(float (&v)[32], int lane) {
#pragma unroll
  for (int n = 16; n >= 1; n >>= 1) {
    const bool up = lane & n;
#pragma unroll
    for (int j = 0; j < n; ++j) v[j] = (up ? v[j + n] : v[j]) + __shfl_xor_sync(0xffffffffu, up ? v[j] : v[j + n], n);
  }
  return v[0];
}

template <int RB, int NC>
__global__ void __launch_bounds__(ScanCfg<RB, NC>::THREADS) delta_scan_kernel(const __grid_constant__ DeltaArgs a, float *__restrict__ o_buf, int vec) {
  using C = ScanCfg<RB, NC>;
  constexpr int DP = C::DP, TC = C::TC, COLS = C::COLS;
  extern __shared__ __align__(16) float sm[];
  float *derived = sm + 2 * C::RAW, *so = derived + 2 * C::DER;  // so: [2][TC][COLS]
  const greta_delta_rule &d = a.d;
  const uint32_t h = blockIdx.x, c0 = blockIdx.y * COLS, D = d.dim, T = a.rows.M;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, l8 = lane & 7;
  const bool producer = warp >= C::CW;
  const int pw = warp - C::CW;
  const uint32_t vcols = min((uint32_t)COLS, D - c0), chunks = (T + TC - 1) / TC;
  float *state = d.state + ((size_t)a.rows.slot0 * d.heads + h) * D * DP;
  for (int i = threadIdx.x; i < 2 * C::RAW + 2 * C::DER; i += C::THREADS) sm[i] = 0.f;
  pdl_launch_dependents();
  pdl_wait();
  __syncthreads();

  auto stage = [&](uint32_t c) {  // producer warps
    if (c < chunks) {
      const uint32_t t0 = c * TC, n = min((uint32_t)TC, T - t0);
      float *b = sm + (c & 1) * C::RAW;
      for (uint32_t t = pw; t < n; t += C::PW) {
        const size_t m = t0 + t, at = m * d.ld + (size_t)h * D;
        float *dst = b + t * C::RAW_ROW;
        const float *src[4] = {d.decay + m * d.ld_decay + (size_t)h * D, d.k + at, d.a + at, d.r + at};
        if (vec) {
#pragma unroll
          for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < (DP + 127) / 128; ++j)
              if (lane * 4 + j * 128 < (int)D) cp16(dst + i * DP + lane * 4 + j * 128, src[i] + lane * 4 + j * 128);
          if (lane * 4 < (int)vcols) cp16(dst + 4 * DP + lane * 4, d.v + at + c0 + lane * 4);
        } else {
#pragma unroll
          for (int i = 0; i < 4; ++i)
            for (uint32_t e = lane; e < D; e += 32) cp4(dst + i * DP + e, src[i] + e);
          if (lane < (int)vcols) cp4(dst + 4 * DP + lane, d.v + at + c0 + lane);
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
    float inv2[4];
#pragma unroll
    for (int t = 0; t < 4; ++t) {
      float kk = 0.f;
#pragma unroll
      for (int i = 0; i < RB; ++i) {
        const float k = raw[t * C::RAW_ROW + DP + i * 32 + lane];
        kk = fmaf(k, k, kk);
      }
      inv2[t] = kk;
    }
#pragma unroll
    for (int t = 0; t < 4; ++t) inv2[t] = 1.f / (warp_sum(inv2[t]) + 1e-6f);
    float acc[32];
#pragma unroll
    for (int j = 0; j < 32; ++j) acc[j] = 0.f;
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
        ak[t] = on ? row[2 * DP] * k[t] * inv2[t] : 0.f;
        r[t] = on ? row[3 * DP] : 0.f;
      }
      const float w01 = w[0] * w[1], w12 = w[1] * w[2], w23 = w[2] * w[3], w02 = w01 * w[2], w13 = w12 * w[3];
      float *o = der + e;
      o[0] = k[0], o[DP] = k[1] * w[0], o[2 * DP] = k[2] * w01, o[3 * DP] = k[3] * w02;
      o[4 * DP] = r[0] * w[0], o[5 * DP] = r[1] * w01, o[6 * DP] = r[2] * w02, o[7 * DP] = r[3] * (w02 * w[3]);
      o[8 * DP] = w[0] * w13;
      o[9 * DP] = k[0] * w13, o[10 * DP] = k[1] * w23, o[11 * DP] = k[2] * w[3], o[12 * DP] = k[3];
      o[13 * DP] = -ak[0] * w13, o[14 * DP] = -ak[1] * w23, o[15 * DP] = -ak[2] * w[3], o[16 * DP] = -ak[3];
      // left factors of the pairs (i, j): P, Q (1,0) (2,0) (2,1) (3,0) (3,1) (3,2); R, T (0,0) (1,0) (1,1) (2,0) .. (3,3)
      const float pl[6] = {k[1], k[2] * w[1], k[2], k[3] * w12, k[3] * w[2], k[3]};
      const float rl[10] = {r[0], r[1] * w[1], r[1], r[2] * w12, r[2] * w[2], r[2], r[3] * w13, r[3] * w23, r[3] * w[3], r[3]};
      constexpr int pj[6] = {0, 0, 1, 0, 1, 2}, rj[10] = {0, 0, 1, 0, 1, 2, 0, 1, 2, 3};
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
    const float total = sum32_of32(acc, lane);
    const int x = lane < 12 ? 0 : (lane - 12) % 10, ri = x < 1 ? 0 : x < 3 ? 1 : x < 6 ? 2 : 3;  // upper triangles of R and T stay zero
    der[C::SCAL + (lane < 12 ? lane : (lane < 22 ? 16 : 32) + ri * 4 + x - ri * (ri + 1) / 2)] = total;
    const float *v = raw + 4 * DP + lane;
    *reinterpret_cast<float4 *>(der + C::VT + lane * 4) = make_float4(v[0], v[C::RAW_ROW], v[2 * C::RAW_ROW], v[3 * C::RAW_ROW]);
  };
  auto write_back = [&](uint32_t c) {
    const uint32_t n = min((uint32_t)TC, T - c * TC);
    const float *src = so + (c & 1) * TC * COLS;
    for (uint32_t t = pw; t < n; t += C::PW)
      if (lane < (int)vcols) o_buf[((size_t)(c * TC + t) * d.heads + h) * D + c0 + lane] = src[t * COLS + lane];
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
        s[c][i] = col < D && a.rows.pos0 ? *reinterpret_cast<const float4 *>(state + (size_t)col * DP + i * 32 + l8 * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
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
        const float4 s0 = lds4(b + C::SCAL), s1 = lds4(b + C::SCAL + 4), s2 = lds4(b + C::SCAL + 8);
        const float4 R = lds4(b + C::SCAL + 16 + (l8 >> 1) * 4), Tn = lds4(b + C::SCAL + 32 + (l8 >> 1) * 4);  // of this lane's token
        float4 v[NC], cc[NC];
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          v[c] = lds4(b + C::VT + (grp * NC + c) * 4);
          const float q = sum8_of4(x[c], l8);
          const int base = lane & 24;
          cc[c].x = __shfl_sync(0xffffffffu, q, base);
          cc[c].y = fmaf(s1.z, cc[c].x, fmaf(s0.x, v[c].x, __shfl_sync(0xffffffffu, q, base + 2)));
          cc[c].z = fmaf(s2.x, cc[c].y, fmaf(s1.w, cc[c].x, fmaf(s0.z, v[c].y, fmaf(s0.y, v[c].x, __shfl_sync(0xffffffffu, q, base + 4)))));
          const float p3 = fmaf(s1.y, v[c].z, fmaf(s1.x, v[c].y, fmaf(s0.w, v[c].x, __shfl_sync(0xffffffffu, q, base + 6))));
          cc[c].w = fmaf(s2.w, cc[c].z, fmaf(s2.z, cc[c].y, fmaf(s2.y, cc[c].x, p3)));
        }
#pragma unroll
        for (int i = 0; i < RB; ++i) {
          const int at = i * 32 + l8 * 4;
          const float4 w = lds4(b + 8 * DP + at);
#pragma unroll
          for (int c = 0; c < NC; ++c) s[c][i] = make_float4(w.x * s[c][i].x, w.y * s[c][i].y, w.z * s[c][i].z, w.w * s[c][i].w);
#pragma unroll
          for (int t = 0; t < 4; ++t) {
            const float4 k = lds4(b + (9 + t) * DP + at), ak = lds4(b + (13 + t) * DP + at);
#pragma unroll
            for (int c = 0; c < NC; ++c) {
              const float vt = t == 0 ? v[c].x : t == 1 ? v[c].y : t == 2 ? v[c].z : v[c].w;
              const float ct = t == 0 ? cc[c].x : t == 1 ? cc[c].y : t == 2 ? cc[c].z : cc[c].w;
              s[c][i].x = fmaf(ak.x, ct, fmaf(k.x, vt, s[c][i].x));
              s[c][i].y = fmaf(ak.y, ct, fmaf(k.y, vt, s[c][i].y));
              s[c][i].z = fmaf(ak.z, ct, fmaf(k.z, vt, s[c][i].z));
              s[c][i].w = fmaf(ak.w, ct, fmaf(k.w, vt, s[c][i].w));
            }
          }
        }
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          float y = sum8_of4(o[c], l8);
          y = fmaf(R.x, v[c].x, fmaf(R.y, v[c].y, fmaf(R.z, v[c].z, fmaf(R.w, v[c].w, y))));
          y = fmaf(Tn.x, cc[c].x, fmaf(Tn.y, cc[c].y, fmaf(Tn.z, cc[c].z, fmaf(Tn.w, cc[c].w, y))));
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
        if (col < D) *reinterpret_cast<float4 *>(state + (size_t)col * DP + i * 32 + l8 * 4) = s[c][i];
    }
  }
}

// Norm over every head's outputs, norm weight and gate: LPH lanes per (row, head), each with its channels in registers
// (four consecutive ones at a time where the sizes allow it).
template <int LPH, bool VEC>
__global__ void __launch_bounds__(256) delta_output_kernel(const __grid_constant__ DeltaArgs a, const float *__restrict__ o_buf, void *out, int out_fmt,
                                                           uint32_t ld_out) {
  constexpr int PER = VEC ? 4 : 1, MAXU = VEC ? 2 : 8;  // units per lane: LPH * MAXU * PER >= 256 channels for the widest heads
  pdl_launch_dependents();
  pdl_wait();
  const greta_delta_rule &d = a.d;
  const uint32_t i = (blockIdx.x * 256 + threadIdx.x) / LPH, l = threadIdx.x % LPH, D = d.dim;
  const bool on = i < a.rows.M * d.heads;
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
    const float *g = d.gate + (size_t)m * d.ld + h * D + c, *n = d.norm + (size_t)h * D + c;
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

int check_delta(const char *what, const greta_delta_rule *d, const greta_rows *r) {
  GRETA_REQUIRE(d && r && r->M, "%s: null or empty argument", what);
  GRETA_REQUIRE(d->heads && d->dim && d->dim <= 256, "%s: %u heads of %u channels (1..256)", what, d->heads, d->dim);
  return GRETA_OK;
}

template <int RB, int NC>
int launch_scan(cudaStream_t s, const DeltaArgs &a, float *o_buf, int vec) {
  using C = ScanCfg<RB, NC>;
  // A grid that fits the SMs asks for more than half of an SM's shared memory: CTAs that become resident while the previous
  // kernel drains would otherwise pair up on the SMs that fall idle first, and the pairs would set the pace.
  constexpr size_t ALONE = 118 * 1024;
  static bool attr_set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !attr_set[dev]) {
    GRETA_CUDA_TRY(cudaFuncSetAttribute(delta_scan_kernel<RB, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)std::max(C::SMEM, ALONE)));
    attr_set[dev] = true;
  }
  const dim3 grid(a.d.heads, (a.d.dim + C::COLS - 1) / C::COLS);
  const size_t smem = grid.x * grid.y <= (uint32_t)sm_count() ? std::max(C::SMEM, ALONE) : C::SMEM;
  GRETA_CUDA_TRY(launch_pdl(delta_scan_kernel<RB, NC>, grid, dim3(C::THREADS), smem, s, a, o_buf, vec));
  return launched("delta_scan_kernel");
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
  const DeltaArgs a{*d, *rows};
  cudaStream_t s = (cudaStream_t)stream;
  const int vec = d->dim % 4 == 0 && d->ld % 4 == 0 && d->ld_decay % 4 == 0 && aligned16(d->r) && aligned16(d->k) && aligned16(d->v) && aligned16(d->a) &&
                  aligned16(d->decay);
  switch (dim32(d->dim) / 32) {
    case 1: return launch_scan<1, 2>(s, a, o_buf, vec);
    case 2: return launch_scan<2, 2>(s, a, o_buf, vec);
    case 3: return launch_scan<3, 2>(s, a, o_buf, vec);
    case 4: return launch_scan<4, 2>(s, a, o_buf, vec);
    case 5: return launch_scan<5, 1>(s, a, o_buf, vec);
    case 6: return launch_scan<6, 1>(s, a, o_buf, vec);
    case 7: return launch_scan<7, 1>(s, a, o_buf, vec);
    default: return launch_scan<8, 1>(s, a, o_buf, vec);
  }
}

int greta_cuda_delta_output(greta_stream_t stream, const greta_delta_rule *d, const float *o_buf, uint32_t M, void *out, int out_fmt, uint32_t ld_out) {
  const greta_rows rows{M, 0, 0, nullptr};
  if (int rc = check_delta("delta_output", d, &rows)) return rc;
  GRETA_REQUIRE(o_buf && out && d->norm && d->gate, "delta_output: null pointer");
  const DeltaArgs a{*d, rows};
  cudaStream_t s = (cudaStream_t)stream;
  const uint32_t D = d->dim, pairs = M * d->heads;
  const bool vec = D % 4 == 0 && d->ld % 4 == 0 && ld_out % 4 == 0 && aligned16(o_buf) && aligned16(d->gate) && aligned16(d->norm) && aligned16(out);
  auto grid = [&](uint32_t lanes) { return dim3((pairs + 256 / lanes - 1) / (256 / lanes)); };
  if (vec && D <= 64)
    GRETA_CUDA_TRY(launch_pdl(delta_output_kernel<16, true>, grid(16), dim3(256), 0, s, a, o_buf, out, out_fmt, ld_out));
  else if (vec)
    GRETA_CUDA_TRY(launch_pdl(delta_output_kernel<32, true>, grid(32), dim3(256), 0, s, a, o_buf, out, out_fmt, ld_out));
  else
    GRETA_CUDA_TRY(launch_pdl(delta_output_kernel<32, false>, grid(32), dim3(256), 0, s, a, o_buf, out, out_fmt, ld_out));
  return launched("delta_output_kernel");
}

}  // extern "C"
