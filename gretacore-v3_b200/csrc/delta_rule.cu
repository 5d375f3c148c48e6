// Generalised delta rule (recurrent mixer with a matrix state per head), fp32 throughout:
//   S <- diag(w) S - (a * u)(u^T S) + k v^T,  u = k / sqrt(k.k + 1e-6),  o = S^T r.
// The columns of S (one per value channel) do not mix: column j only needs the scalar c_j = k^T S_j of the old state,
//   S_j <- w * S_j + k v_j - ak c_j,   ak = a * k / (k.k + 1e-6),   o_j = r^T S_j,
// so eight lanes hold one column in registers (row i * 32 + lane8 * 4 + e in register 4 i + e) and a step is two dot
// products over eight lanes and one update.  Rows past dim are padding: every vector is zero there, so they stay zero.
//
// The scan looks one token ahead so that no step waits for a reduction it has just started: with S' the state before token t,
//   k'^T S_j = (k' * w)^T S'_j + (k'.k) v_j - (k'.ak) c_j      (k' the next token's key)
// and the first term needs only S', one step earlier than the state it belongs to.  Producer warps stage the tokens' vectors
// (cp.async), derive ak, k' * w and the two scalars, and write the outputs back, one chunk ahead of and behind the warps that
// hold the state.
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

typedef unsigned long long f32x2;  // two floats for the packed 32-bit arithmetic
__device__ __forceinline__ f32x2 pack2(float a, float b) {
  f32x2 d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(a), "f"(b));
  return d;
}
__device__ __forceinline__ float sum_halves(f32x2 v) {
  float a, b;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v));
  return a + b;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ ulonglong2 lds2(const float *p) { return *reinterpret_cast<const ulonglong2 *>(p); }

// The recurrence over a portion: grid (heads, column groups).  A CTA keeps 32 columns of one head in the registers of its
// first warps, NC columns per group of eight lanes, and walks the tokens in chunks of TC; three chunk buffers rotate.
template <int RB, int NC>
struct ScanCfg {
  static constexpr int DP = RB * 32, COLS = 32;
  static constexpr int TC = RB <= 4 ? 16 : 8;
  static constexpr int ROW = 5 * DP + COLS + 4;   // floats of a staged token: w, k, ak, r, k' * w, v, {k'.k, k'.ak}
  static constexpr int BUF = (TC + 1) * ROW;      // one more token: its key is the last one's k'
  static constexpr int CW = COLS / (4 * NC), PW = 4, THREADS = (CW + PW) * 32;
  static constexpr size_t SMEM = (size_t)(3 * BUF + 2 * TC * COLS) * 4;
  static_assert(SMEM <= 232448, "chunk buffers exceed shared memory");
};
template <int RB, int NC>
__global__ void __launch_bounds__(ScanCfg<RB, NC>::THREADS) delta_scan_kernel(const __grid_constant__ DeltaArgs a, float *__restrict__ o_buf, int vec) {
  using C = ScanCfg<RB, NC>;
  constexpr int DP = C::DP, TC = C::TC, ROW = C::ROW, COLS = C::COLS, BUF = C::BUF;
  extern __shared__ __align__(16) float sm[];
  float *so = sm + 3 * BUF;  // [2][TC][COLS]
  const greta_delta_rule &d = a.d;
  const uint32_t h = blockIdx.x, c0 = blockIdx.y * COLS, D = d.dim, T = a.rows.M;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, l8 = lane & 7;
  const bool producer = warp >= C::CW;
  const int pw = warp - C::CW;
  const uint32_t vcols = min((uint32_t)COLS, D - c0), chunks = (T + TC - 1) / TC;
  float *state = d.state + ((size_t)a.rows.slot0 * d.heads + h) * D * DP;
  for (int i = threadIdx.x; i < 3 * BUF; i += C::THREADS) sm[i] = 0.f;
  pdl_launch_dependents();
  pdl_wait();
  __syncthreads();

  auto stage = [&](uint32_t c) {  // producer warps: the chunk's tokens and one more
    if (c < chunks) {
      const uint32_t t0 = c * TC, n = min((uint32_t)TC + 1, T - t0);
      float *b = sm + (c % 3) * BUF;
      for (uint32_t t = pw; t < n; t += C::PW) {
        const size_t m = t0 + t, at = m * d.ld + (size_t)h * D;
        float *dst = b + t * ROW;
        const float *src[4] = {d.decay + m * d.ld_decay + (size_t)h * D, d.k + at, d.a + at, d.r + at};
        if (vec) {
#pragma unroll
          for (int i = 0; i < 4; ++i)
            for (uint32_t e = lane * 4; e < D; e += 128) cp16(dst + i * DP + e, src[i] + e);
          if (lane * 4 < (int)vcols) cp16(dst + 5 * DP + lane * 4, d.v + at + c0 + lane * 4);
        } else {
#pragma unroll
          for (int i = 0; i < 4; ++i)
            for (uint32_t e = lane; e < D; e += 32) cp4(dst + i * DP + e, src[i] + e);
          if (lane < (int)vcols) cp4(dst + 5 * DP + lane, d.v + at + c0 + lane);
        }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto prepare = [&](uint32_t c) {  // producer warps, once the chunk has landed: ak, k' * w, k'.k, k'.ak
    if (c >= chunks) return;
    const int n = (int)min((uint32_t)TC, T - c * TC);
    float *b = sm + (c % 3) * BUF;
    for (int t = pw; t < TC; t += C::PW) {
      float *row = b + t * ROW;
      if (t >= n) {  // past the end of the portion: a token that leaves the state as it is
        for (int e = lane; e < 5 * DP + COLS + 4; e += 32) row[e] = e < DP ? 1.f : 0.f;
        continue;
      }
      float k[RB], kk = 0.f, next_k = 0.f, next_ak = 0.f;
#pragma unroll
      for (int i = 0; i < RB; ++i) {
        k[i] = row[DP + i * 32 + lane];
        kk = fmaf(k[i], k[i], kk);
      }
      const float inv2 = 1.f / (warp_sum(kk) + 1e-6f);
#pragma unroll
      for (int i = 0; i < RB; ++i) {
        const int e = i * 32 + lane;
        const float k1 = row[ROW + DP + e], ak = row[2 * DP + e] * k[i] * inv2;
        row[2 * DP + e] = ak;
        row[4 * DP + e] = k1 * row[e];
        next_k = fmaf(k1, k[i], next_k);
        next_ak = fmaf(k1, ak, next_ak);
      }
      next_k = warp_sum(next_k);
      next_ak = warp_sum(next_ak);
      if (lane == 0) {
        row[5 * DP + COLS] = next_k;
        row[5 * DP + COLS + 1] = next_ak;
      }
    }
  };
  auto landed = [&]() {  // the chunk before the last one staged is complete for every producer
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    asm volatile("bar.sync 1, %0;" ::"n"(C::PW * 32) : "memory");
  };
  auto write_back = [&](uint32_t c) {
    const uint32_t n = min((uint32_t)TC, T - c * TC);
    const float *src = so + (c & 1) * TC * COLS;
    for (uint32_t t = pw; t < n; t += C::PW)
      if (lane < (int)vcols) o_buf[((size_t)(c * TC + t) * d.heads + h) * D + c0 + lane] = src[t * COLS + lane];
  };

  const int grp = threadIdx.x >> 3;  // state warps: columns c0 + grp * NC ..
  f32x2 s[NC][2 * RB];
  float nc[NC];
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
        const bool on = col < D && a.rows.pos0;
        const ulonglong2 v = on ? *reinterpret_cast<const ulonglong2 *>(state + (size_t)col * DP + i * 32 + l8 * 4) : make_ulonglong2(0ull, 0ull);
        s[c][2 * i] = v.x;
        s[c][2 * i + 1] = v.y;
      }
    }
  }
  __syncthreads();
  if (!producer) {  // the first token's c
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      f32x2 x = 0ull;
#pragma unroll
      for (int i = 0; i < RB; ++i) {
        const ulonglong2 k = lds2(sm + DP + i * 32 + l8 * 4);
        x = fma2(k.x, s[c][2 * i], x);
        x = fma2(k.y, s[c][2 * i + 1], x);
      }
      nc[c] = -sum8(sum_halves(x));
    }
  }
  for (uint32_t ch = 0; ch < chunks; ++ch) {
    if (producer) {
      stage(ch + 2);
      landed();
      prepare(ch + 1);
      if (ch) write_back(ch - 1);
    } else {
      const float *b = sm + (ch % 3) * BUF;
      float *out = so + (ch & 1) * TC * COLS;
#pragma unroll 1
      for (int t8 = 0; t8 < TC; t8 += 8) {  // eight tokens of straight-line code; their outputs leave together
        float o[NC][8];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const float *row = b + (t8 + j) * ROW;
          f32x2 x[NC], y[NC], v2[NC], nc2[NC];
          float v[NC];
#pragma unroll
          for (int c = 0; c < NC; ++c) {
            v[c] = row[5 * DP + grp * NC + c];
            v2[c] = pack2(v[c], v[c]);
            nc2[c] = pack2(nc[c], nc[c]);
            x[c] = y[c] = 0ull;
          }
#pragma unroll
          for (int i = 0; i < RB; ++i) {
            const ulonglong2 kw = lds2(row + 4 * DP + i * 32 + l8 * 4);
#pragma unroll
            for (int c = 0; c < NC; ++c) {
              x[c] = fma2(kw.x, s[c][2 * i], x[c]);
              x[c] = fma2(kw.y, s[c][2 * i + 1], x[c]);
            }
          }
#pragma unroll
          for (int i = 0; i < RB; ++i) {
            const int at = i * 32 + l8 * 4;
            const ulonglong2 w = lds2(row + at), k = lds2(row + DP + at), ak = lds2(row + 2 * DP + at), r = lds2(row + 3 * DP + at);
#pragma unroll
            for (int c = 0; c < NC; ++c) {
              s[c][2 * i] = fma2(ak.x, nc2[c], fma2(k.x, v2[c], mul2(w.x, s[c][2 * i])));
              s[c][2 * i + 1] = fma2(ak.y, nc2[c], fma2(k.y, v2[c], mul2(w.y, s[c][2 * i + 1])));
              y[c] = fma2(r.x, s[c][2 * i], y[c]);
              y[c] = fma2(r.y, s[c][2 * i + 1], y[c]);
            }
          }
          const float2 nx = *reinterpret_cast<const float2 *>(row + 5 * DP + COLS);
#pragma unroll
          for (int c = 0; c < NC; ++c) {
            nc[c] = -(sum8(sum_halves(x[c])) + fmaf(nx.y, nc[c], nx.x * v[c]));
            o[c][j] = sum_halves(y[c]);
          }
        }
        // lane j of the group receives the total of token t8 + j: halves of the tokens change places three times
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          float q4[4], q2[2];
          const bool b4 = l8 & 4, b2 = l8 & 2, b1 = l8 & 1;
#pragma unroll
          for (int j = 0; j < 4; ++j) q4[j] = (b4 ? o[c][j + 4] : o[c][j]) + __shfl_xor_sync(0xffffffffu, b4 ? o[c][j] : o[c][j + 4], 4);
#pragma unroll
          for (int j = 0; j < 2; ++j) q2[j] = (b2 ? q4[j + 2] : q4[j]) + __shfl_xor_sync(0xffffffffu, b2 ? q4[j] : q4[j + 2], 2);
          out[(t8 + l8) * COLS + grp * NC + c] = (b1 ? q2[1] : q2[0]) + __shfl_xor_sync(0xffffffffu, b1 ? q2[0] : q2[1], 1);
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
        if (col < D) *reinterpret_cast<ulonglong2 *>(state + (size_t)col * DP + i * 32 + l8 * 4) = make_ulonglong2(s[c][2 * i], s[c][2 * i + 1]);
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
  static bool attr_set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !attr_set[dev]) {
    GRETA_CUDA_TRY(cudaFuncSetAttribute(delta_scan_kernel<RB, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)C::SMEM));
    attr_set[dev] = true;
  }
  GRETA_CUDA_TRY(launch_pdl(delta_scan_kernel<RB, NC>, dim3(a.d.heads, (a.d.dim + C::COLS - 1) / C::COLS), dim3(C::THREADS), C::SMEM, s, a, o_buf, vec));
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
