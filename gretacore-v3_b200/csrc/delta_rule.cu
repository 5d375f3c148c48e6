// Generalised delta rule (recurrent mixer with a matrix state per head), fp32 throughout:
//   S <- diag(w) S - (a * u)(u^T S) + k v^T,  u = k / sqrt(k.k + 1e-6),  o = S^T r.
// The columns of S (one per value channel) do not mix: column j only needs the scalar c_j = k^T S_j of the old state,
//   S_j <- w * S_j + k v_j - ak c_j,   ak = a * k / (k.k + 1e-6),   o_j = r^T S_j,
// so eight lanes hold one column in registers (row i * 32 + lane8 * 4 + e in register 4 i + e) and a step is two dot
// products over eight lanes and one update.  The scan computes o_t and the next token's c together from the new state:
// one reduction per token.  Rows past dim are padding: every vector is zero there, so they stay zero.
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

// The recurrence over a portion: grid (heads, column groups).  A CTA keeps COLS columns of one head in registers (NC per
// group of eight lanes) and walks the tokens in chunks of TC staged by cp.async, two chunks in shared memory.
template <int RB>
struct ScanCfg {
  static constexpr int DP = RB * 32, COLS = 32;
  static constexpr int TC = RB <= 4 ? 16 : 8;
  static constexpr int ROW = 4 * DP + COLS;  // floats of a staged token: w, k, ak, r, v
  static constexpr size_t SMEM = (size_t)(2 * TC * ROW + TC * COLS) * 4;
};
template <int RB, int NC>
__global__ void __launch_bounds__(ScanCfg<RB>::COLS / NC * 8) delta_scan_kernel(const __grid_constant__ DeltaArgs a, float *__restrict__ o_buf, int vec) {
  using C = ScanCfg<RB>;
  constexpr int DP = C::DP, TC = C::TC, ROW = C::ROW, COLS = C::COLS, THREADS = COLS / NC * 8, NW = THREADS / 32;
  extern __shared__ __align__(16) float sm[];
  float *so = sm + 2 * TC * ROW;  // [TC][COLS]
  const greta_delta_rule &d = a.d;
  const uint32_t h = blockIdx.x, c0 = blockIdx.y * COLS, D = d.dim, T = a.rows.M;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, l8 = lane & 7, grp = threadIdx.x >> 3;
  float *state = d.state + ((size_t)a.rows.slot0 * d.heads + h) * D * DP;
  for (int i = threadIdx.x; i < 2 * TC * ROW; i += THREADS) sm[i] = 0.f;
  pdl_launch_dependents();
  pdl_wait();
  __syncthreads();
  const uint32_t vcols = min((uint32_t)COLS, D - c0);
  auto stage = [&](uint32_t t0, int buf) {
    const uint32_t n = t0 < T ? min((uint32_t)TC, T - t0) : 0;
    float *b = sm + buf * TC * ROW;
    const uint32_t unit = vec ? 4 : 1, per = D / unit, vper = vec ? vcols / 4 : vcols, tok = 4 * per + vper;
    for (uint32_t i = threadIdx.x; i < n * tok; i += THREADS) {
      const uint32_t t = i / tok, j = i % tok, which = j < 4 * per ? j / per : 4, e = (which < 4 ? j % per : j - 4 * per) * unit;
      const size_t m = t0 + t, at = m * d.ld + (size_t)h * D;
      const float *src = which == 0 ? d.decay + m * d.ld_decay + (size_t)h * D + e
                         : which == 1 ? d.k + at + e
                         : which == 2 ? d.a + at + e
                         : which == 3 ? d.r + at + e
                                      : d.v + at + c0 + e;
      float *dst = b + t * ROW + which * DP + e;
      if (vec)
        cp16(dst, src);
      else
        cp4(dst, src);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  float4 s[NC][RB];
  bool on[NC];
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const uint32_t col = c0 + grp * NC + c;
    on[c] = col < D;
#pragma unroll
    for (int i = 0; i < RB; ++i)
      s[c][i] = on[c] && a.rows.pos0 ? *reinterpret_cast<const float4 *>(state + (size_t)col * DP + i * 32 + l8 * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  stage(0, 0);
  for (uint32_t t0 = 0, buf = 0; t0 < T; t0 += TC, buf ^= 1) {
    stage(t0 + TC, buf ^ 1);
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    float *b = sm + buf * TC * ROW;
    const int n = (int)min((uint32_t)TC, T - t0);
    for (int t = warp; t < n; t += NW) {  // ak = a k / (k.k + 1e-6)
      float *row = b + t * ROW;
      float kk = 0.f;
#pragma unroll
      for (int i = 0; i < RB; ++i) kk = fmaf(row[DP + i * 32 + lane], row[DP + i * 32 + lane], kk);
      const float inv2 = 1.f / (warp_sum(kk) + 1e-6f);
#pragma unroll
      for (int i = 0; i < RB; ++i) row[2 * DP + i * 32 + lane] *= row[DP + i * 32 + lane] * inv2;
    }
    __syncthreads();
    float4 k[RB];
    float nc[NC];
#pragma unroll
    for (int i = 0; i < RB; ++i) k[i] = lds4(b + DP + i * 32 + l8 * 4);
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      float x = 0.f;
#pragma unroll
      for (int i = 0; i < RB; ++i) x = dot4(k[i], s[c][i], x);
      nc[c] = -sum8(x);
    }
    for (int t = 0; t < n; ++t) {
      const float *row = b + t * ROW;
      float v[NC], o[NC], x[NC];
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        v[c] = row[4 * DP + grp * NC + c];
        o[c] = x[c] = 0.f;
      }
      const float *next = t + 1 < n ? row + ROW : row;  // the last token's look-ahead is not used
#pragma unroll
      for (int i = 0; i < RB; ++i) {
        const int at = i * 32 + l8 * 4;
        const float4 w = lds4(row + at), ak = lds4(row + 2 * DP + at), r = lds4(row + 3 * DP + at), kn = lds4(next + DP + at);
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          update4(s[c][i], w, k[i], ak, v[c], nc[c]);
          o[c] = dot4(r, s[c][i], o[c]);
          x[c] = dot4(kn, s[c][i], x[c]);
        }
        k[i] = kn;
      }
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        o[c] = sum8(o[c]);
        nc[c] = -sum8(x[c]);
        if (l8 == 0) so[t * COLS + grp * NC + c] = o[c];
      }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n * COLS; i += THREADS) {
      const uint32_t t = i / COLS, c = i % COLS;
      if (c < vcols) o_buf[((size_t)(t0 + t) * d.heads + h) * D + c0 + c] = so[i];
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int c = 0; c < NC; ++c)
#pragma unroll
    for (int i = 0; i < RB; ++i)
      if (on[c]) *reinterpret_cast<float4 *>(state + (size_t)(c0 + grp * NC + c) * DP + i * 32 + l8 * 4) = s[c][i];
}

// Norm over every head's outputs, norm weight and gate: one warp per (row, head).
__global__ void __launch_bounds__(256) delta_output_kernel(const __grid_constant__ DeltaArgs a, const float *__restrict__ o_buf, void *out, int out_fmt,
                                                           uint32_t ld_out) {
  pdl_launch_dependents();
  pdl_wait();
  const greta_delta_rule &d = a.d;
  const uint32_t i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, D = d.dim;
  if (i >= a.rows.M * d.heads) return;
  const uint32_t m = i / d.heads, h = i % d.heads;
  const float *o = o_buf + (size_t)i * D;
  float q = 0.f;
  for (uint32_t c = lane; c < D; c += 32) q = fmaf(o[c], o[c], q);
  const float inv = 1.f / sqrtf(warp_sum(q) / (float)D + d.eps);
  for (uint32_t c = lane; c < D; c += 32)
    store_out(out, out_fmt, (size_t)m * ld_out + h * D + c, o[c] * inv * d.norm[(size_t)h * D + c] * d.gate[(size_t)m * d.ld + h * D + c]);
}

int check_delta(const char *what, const greta_delta_rule *d, const greta_rows *r) {
  GRETA_REQUIRE(d && r && r->M, "%s: null or empty argument", what);
  GRETA_REQUIRE(d->heads && d->dim && d->dim <= 256, "%s: %u heads of %u channels (1..256)", what, d->heads, d->dim);
  return GRETA_OK;
}

template <int RB, int NC>
int launch_scan(cudaStream_t s, const DeltaArgs &a, float *o_buf, int vec) {
  using C = ScanCfg<RB>;
  static bool attr_set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !attr_set[dev]) {
    GRETA_CUDA_TRY(cudaFuncSetAttribute(delta_scan_kernel<RB, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)C::SMEM));
    attr_set[dev] = true;
  }
  GRETA_CUDA_TRY(launch_pdl(delta_scan_kernel<RB, NC>, dim3(a.d.heads, (a.d.dim + C::COLS - 1) / C::COLS), dim3(C::COLS / NC * 8), C::SMEM, s, a, o_buf, vec));
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
    case 1: return launch_scan<1, 1>(s, a, o_buf, vec);
    case 2: return launch_scan<2, 1>(s, a, o_buf, vec);
    case 3: return launch_scan<3, 1>(s, a, o_buf, vec);
    case 4: return launch_scan<4, 1>(s, a, o_buf, vec);
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
  GRETA_CUDA_TRY(launch_pdl(delta_output_kernel, dim3((M * d->heads + 7) / 8), dim3(256), 0, (cudaStream_t)stream, a, o_buf, out, out_fmt, ld_out));
  return launched("delta_output_kernel");
}

}  // extern "C"
