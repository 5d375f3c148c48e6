// Dense linears on few activation rows (decode and short portions): y[m][n] = act(W[n] . LN(x[m]) + bias), weights in bf16
// or fp32 streamed once for up to 8 rows, activations and accumulation in fp32; and the small operators around them
// (layer and root-mean-square norm, embeddings, row gather).  A norm without an offset (ln_b) is the root-mean-square one.
//
// A warp owns R weight rows.  Each lane takes 8 consecutive weights of every row per step (16 bytes of bf16), the
// activations of the same 8 columns come out of shared memory once for all R rows.  There the two float4 halves of every
// 8-column group live in separate planes, so that a warp's reads are conflict-free.  Rows longer than a chunk are staged
// in pieces; the layer norm is applied while staging.  The first weights are requested before the wait on the previous
// kernel (programmatic dependent launch).
#include <algorithm>

#include "dense_device.cuh"

using namespace greta;

namespace {

constexpr int GV_THREADS = 256, GV_WARPS = 8;
constexpr bool PREFETCH = true;

template <typename WT>
struct W8;  // 8 consecutive weights as stored
template <>
struct W8<__nv_bfloat16> {
  uint4 a;
  __device__ __forceinline__ void load(const __nv_bfloat16 *p) { a = ld_stream(p); }
  __device__ __forceinline__ void get(float (&f)[8]) const {
    const uint32_t w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      f[2 * i] = __uint_as_float(w[i] << 16);
      f[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u);
    }
  }
};
template <>
struct W8<float> {
  uint4 a, b;
  __device__ __forceinline__ void load(const float *p) {
    a = ld_stream(p);
    b = ld_stream(p + 4);
  }
  __device__ __forceinline__ void get(float (&f)[8]) const {
    const uint32_t w[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] = __uint_as_float(w[i]);
  }
};

template <typename WT, int MR, int R>
__global__ void __launch_bounds__(GV_THREADS) linear_gemv_kernel(const WT *__restrict__ W, uint32_t N, uint32_t K, uint32_t ldw, Segments sg,
                                                                 const float *x, uint32_t ldx, const float *__restrict__ ln_w,
                                                                 const float *__restrict__ ln_b, float eps, uint32_t M, uint32_t chunk, int vec) {
  extern __shared__ float4 xs[];  // [MR][2][chunk / 8]
  __shared__ float red[32], stat[MR][2];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t n0 = (blockIdx.x * GV_WARPS + warp) * R;
  const WT *wrow[R];
#pragma unroll
  for (int r = 0; r < R; ++r) wrow[r] = W + (size_t)min(n0 + r, N - 1) * ldw + lane * 8;
  W8<WT> first[R];
  const bool any0 = (uint32_t)lane * 8 < ldw;
  if (any0) {
#pragma unroll
    for (int r = 0; r < R; ++r) first[r].load(wrow[r]);
  }
  if (PREFETCH) {  // the rest of the rows starts its way from HBM to L2 while this CTA still waits for its input
    const uint32_t row_bytes = ldw * (uint32_t)sizeof(WT);
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const char *p = reinterpret_cast<const char *>(W + (size_t)min(n0 + r, N - 1) * ldw);
      for (uint32_t b = 512 * sizeof(WT) / 2 + lane * 128; b < min(row_bytes, 16384u); b += 32 * 128)
        asm volatile("prefetch.global.L2 [%0];" ::"l"(p + b));
    }
  }
  pdl_launch_dependents();
  pdl_wait();
  if (ln_w) {
    if (MR == 1) {
      float s = 0.f, mean = 0.f;
      if (ln_b) {
        for (uint32_t k = threadIdx.x; k < K; k += GV_THREADS) s += x[k];
        mean = block_sum_all(s, red) / (float)K;
      }
      float q = 0.f;
      for (uint32_t k = threadIdx.x; k < K; k += GV_THREADS) {
        const float c = x[k] - mean;
        q = fmaf(c, c, q);
      }
      const float var = block_sum_all(q, red) / (float)K;
      if (threadIdx.x == 0) {
        stat[0][0] = mean;
        stat[0][1] = 1.f / sqrtf(var + eps);
      }
    } else if (warp < MR && warp < M) {
      const float *xr = x + (size_t)warp * ldx;
      float s = 0.f, mean = 0.f;
      if (ln_b) {
        for (uint32_t k = lane; k < K; k += 32) s += xr[k];
        mean = warp_sum(s) / (float)K;
      }
      float q = 0.f;
      for (uint32_t k = lane; k < K; k += 32) {
        const float c = xr[k] - mean;
        q = fmaf(c, c, q);
      }
      const float var = warp_sum(q) / (float)K;
      if (lane == 0) {
        stat[warp % MR][0] = mean;
        stat[warp % MR][1] = 1.f / sqrtf(var + eps);
      }
    }
    __syncthreads();
  }
  float acc[MR][R];
#pragma unroll
  for (int m = 0; m < MR; ++m)
#pragma unroll
    for (int r = 0; r < R; ++r) acc[m][r] = 0.f;
  const uint32_t plane = chunk / 8;
  for (uint32_t k0 = 0; k0 < ldw; k0 += chunk) {
    const uint32_t kc = min(chunk, ldw - k0);  // multiple of 64
    if (k0) __syncthreads();
#pragma unroll
    for (int m = 0; m < MR; ++m) {
      float *xd = reinterpret_cast<float *>(xs + (size_t)m * 2 * plane);
      const float *xr = x + (size_t)m * ldx;
      const bool row = (uint32_t)m < M;
      const float mean = ln_w && row ? stat[m][0] : 0.f, inv = ln_w && row ? stat[m][1] : 1.f;
      if (vec && row) {  // four columns are one slot of a plane
        for (uint32_t k = threadIdx.x * 4; k < kc; k += GV_THREADS * 4) {
          const uint32_t col = k0 + k;
          float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
          if (col < K) {
            v = *reinterpret_cast<const float4 *>(xr + col);
            if (ln_w) {
              const float4 w = __ldg(reinterpret_cast<const float4 *>(ln_w + col));
              const float4 b = ln_b ? __ldg(reinterpret_cast<const float4 *>(ln_b + col)) : make_float4(0.f, 0.f, 0.f, 0.f);
              v.x = (v.x - mean) * inv * w.x + b.x;
              v.y = (v.y - mean) * inv * w.y + b.y;
              v.z = (v.z - mean) * inv * w.z + b.z;
              v.w = (v.w - mean) * inv * w.w + b.w;
            }
          }
          reinterpret_cast<float4 *>(xd)[((k >> 2) & 1) * plane + (k >> 3)] = v;
        }
        continue;
      }
      for (uint32_t k = threadIdx.x; k < kc; k += GV_THREADS) {
        const uint32_t col = k0 + k;
        float v = 0.f;
        if (row && col < K) {
          v = xr[col];
          if (ln_w) v = (v - mean) * inv * __ldg(ln_w + col) + (ln_b ? __ldg(ln_b + col) : 0.f);
        }
        xd[((k >> 2) & 1) * plane * 4 + (k >> 3) * 4 + (k & 3)] = v;
      }
    }
    __syncthreads();
    auto step = [&](const W8<WT>(&w)[R], uint32_t k) {
      float4 xa[MR], xb[MR];
#pragma unroll
      for (int m = 0; m < MR; ++m) {
        xa[m] = xs[(size_t)m * 2 * plane + (k >> 3)];
        xb[m] = xs[(size_t)m * 2 * plane + plane + (k >> 3)];
      }
#pragma unroll
      for (int r = 0; r < R; ++r) {
        float f[8];
        w[r].get(f);
#pragma unroll
        for (int m = 0; m < MR; ++m) {
          float a = acc[m][r];
          a = fmaf(f[0], xa[m].x, a);
          a = fmaf(f[1], xa[m].y, a);
          a = fmaf(f[2], xa[m].z, a);
          a = fmaf(f[3], xa[m].w, a);
          a = fmaf(f[4], xb[m].x, a);
          a = fmaf(f[5], xb[m].y, a);
          a = fmaf(f[6], xb[m].z, a);
          acc[m][r] = fmaf(f[7], xb[m].w, a);
        }
      }
    };
    uint32_t k = lane * 8;
    if (k0 == 0 && any0) {
      step(first, k);
      k += 256;
    }
    constexpr int UN = MR > 2 ? (R >= 4 ? 2 : 4) : R >= 4 ? 2 : R == 2 ? 4 : 8;  // steps in flight
    for (; k + (UN - 1) * 256 < kc; k += UN * 256) {
      W8<WT> w[UN][R];
#pragma unroll
      for (int u = 0; u < UN; ++u)
#pragma unroll
        for (int r = 0; r < R; ++r) w[u][r].load(wrow[r] + k0 + u * 256 + (k - lane * 8));
#pragma unroll
      for (int u = 0; u < UN; ++u) step(w[u], k + u * 256);
    }
    for (; k < kc; k += 256) {
      W8<WT> w[R];
#pragma unroll
      for (int r = 0; r < R; ++r) w[r].load(wrow[r] + k0 + (k - lane * 8));
      step(w, k);
    }
  }
  // lane m * R + r finishes row n0 + r of activation row m
  float mine = 0.f;
#pragma unroll
  for (int m = 0; m < MR; ++m)
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const float t = warp_sum(acc[m][r]);
      if (lane == m * R + r) mine = t;
    }
  const uint32_t m = lane / R, row = n0 + lane % R;
  if (m < min(M, (uint32_t)MR) && row < N) store_segment(sg.s[segment_of(sg, row)], row, m, mine);
}

// One CTA per row; rows of up to 8192 columns (a multiple of 4) are read once and kept in registers.  RMS: no mean, no offset.
template <bool RMS>
__global__ void __launch_bounds__(256) norm_kernel(const float *__restrict__ x, uint32_t ldx, const float *__restrict__ w, const float *__restrict__ b,
                                                   float eps, void *out, int out_fmt, uint32_t D, uint32_t ld, int vec) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const float *xr = x + (size_t)blockIdx.x * ldx;
  if (vec) {
    constexpr int U = 8;
    float4 v[U];
    float s = 0.f;
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const uint32_t k = (u * 256 + threadIdx.x) * 4;
      v[u] = k < D ? *reinterpret_cast<const float4 *>(xr + k) : make_float4(0.f, 0.f, 0.f, 0.f);
      s += (v[u].x + v[u].y) + (v[u].z + v[u].w);
    }
    const float mean = RMS ? 0.f : block_sum_all(s, red) / (float)D;
    float q = 0.f;
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if ((u * 256 + threadIdx.x) * 4 >= D) continue;
      v[u].x -= mean, v[u].y -= mean, v[u].z -= mean, v[u].w -= mean;
      q = fmaf(v[u].x, v[u].x, fmaf(v[u].y, v[u].y, fmaf(v[u].z, v[u].z, fmaf(v[u].w, v[u].w, q))));
    }
    const float inv = 1.f / sqrtf(block_sum_all(q, red) / (float)D + eps);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const uint32_t k = (u * 256 + threadIdx.x) * 4;
      if (k >= D) continue;
      const float4 g = *reinterpret_cast<const float4 *>(w + k);
      const float4 h = RMS ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4 *>(b + k);
      const float4 y = make_float4(v[u].x * inv * g.x + h.x, v[u].y * inv * g.y + h.y, v[u].z * inv * g.z + h.z, v[u].w * inv * g.w + h.w);
      const size_t at = (size_t)blockIdx.x * ld + k;
      if (out_fmt == GRETA_OUT_F32) {
        *reinterpret_cast<float4 *>(static_cast<float *>(out) + at) = y;
      } else if (out_fmt == GRETA_OUT_F16) {
        const __half2 lo = __floats2half2_rn(y.x, y.y), hi = __floats2half2_rn(y.z, y.w);
        uint2 p;
        p.x = *reinterpret_cast<const uint32_t *>(&lo);
        p.y = *reinterpret_cast<const uint32_t *>(&hi);
        *reinterpret_cast<uint2 *>(static_cast<__half *>(out) + at) = p;
      } else {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(y.x, y.y), hi = __floats2bfloat162_rn(y.z, y.w);
        uint2 p;
        p.x = *reinterpret_cast<const uint32_t *>(&lo);
        p.y = *reinterpret_cast<const uint32_t *>(&hi);
        *reinterpret_cast<uint2 *>(static_cast<__nv_bfloat16 *>(out) + at) = p;
      }
    }
    return;
  }
  float mean = 0.f;
  if (!RMS) {
    float s = 0.f;
    for (uint32_t k = threadIdx.x; k < D; k += 256) s += xr[k];
    mean = block_sum_all(s, red) / (float)D;
  }
  float q = 0.f;
  for (uint32_t k = threadIdx.x; k < D; k += 256) {
    const float c = xr[k] - mean;
    q = fmaf(c, c, q);
  }
  const float inv = 1.f / sqrtf(block_sum_all(q, red) / (float)D + eps);
  for (uint32_t k = threadIdx.x; k < D; k += 256) store_out(out, out_fmt, (size_t)blockIdx.x * ld + k, (xr[k] - mean) * inv * w[k] + (RMS ? 0.f : b[k]));
}

template <typename T>
__device__ __forceinline__ float table_at(const void *t, size_t i) {
  return (float)static_cast<const T *>(t)[i];
}
template <typename T>
__global__ void embedding_positions_kernel(const int32_t *__restrict__ tokens, const void *__restrict__ table, const void *__restrict__ pos_table,
                                           float *__restrict__ out, uint32_t M, uint32_t D, uint32_t vocab, uint32_t max_positions,
                                           const uint32_t *d_pos, uint32_t pos0) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (size_t)M * D) return;
  const uint32_t m = i / D, c = i % D, p = d_pos ? d_pos[m] : pos0 + m;
  const int32_t t = tokens[m];
  float v = 0.f;
  if (t >= 0 && (uint32_t)t < vocab) v = table_at<T>(table, (size_t)t * D + c);
  if (pos_table && p < max_positions) v += table_at<T>(pos_table, (size_t)p * D + c);
  out[i] = v;
}

template <typename T>
__global__ void embedding_scaled_kernel(const int32_t *__restrict__ tokens, const T *__restrict__ table, uint32_t ld, float scale, float *__restrict__ out,
                                        uint32_t M, uint32_t D, uint32_t vocab) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (size_t)M * D) return;
  const int32_t t = tokens[i / D];
  out[i] = t >= 0 && (uint32_t)t < vocab ? scale * (float)table[(size_t)t * ld + i % D] : 0.f;
}

struct RowList {
  uint32_t r[64];
};
__global__ void gather_rows_kernel(const float *__restrict__ x, uint32_t D, RowList rows, float *__restrict__ out) {
  for (uint32_t c = threadIdx.x; c < D; c += blockDim.x) out[(size_t)blockIdx.x * D + c] = x[(size_t)rows.r[blockIdx.x] * D + c];
}

template <typename WT, int MR, int R>
int launch_gemv(cudaStream_t s, const greta_linear *l, const Segments &sg, const float *x, uint32_t ldx, const float *ln_w, const float *ln_b, float eps,
                uint32_t M) {
  const uint32_t cap = 16384 / MR, chunk = std::min(cap, (l->ldw + 255) / 256 * 256);  // 64 KB of activations at most
  const size_t smem = (size_t)MR * chunk * 4;
  static bool attr_set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !attr_set[dev]) {
    GRETA_CUDA_TRY(cudaFuncSetAttribute(linear_gemv_kernel<WT, MR, R>, cudaFuncAttributeMaxDynamicSharedMemorySize, 65536));
    attr_set[dev] = true;
  }
  const uint32_t grid = (l->N + GV_WARPS * R - 1) / (GV_WARPS * R);
  const int vec = l->K % 4 == 0 && ldx % 4 == 0 && aligned16(x) && (!ln_w || (aligned16(ln_w) && (!ln_b || aligned16(ln_b))));
  GRETA_CUDA_TRY(launch_pdl(linear_gemv_kernel<WT, MR, R>, dim3(grid), dim3(GV_THREADS), smem, s, static_cast<const WT *>(l->w), l->N, l->K, l->ldw, sg, x,
                            ldx, ln_w, ln_b, eps, M, chunk, vec));
  return launched("linear_gemv_kernel");
}
template <typename WT, int MR>
int pick_rows(cudaStream_t s, const greta_linear *l, const Segments &sg, const float *x, uint32_t ldx, const float *ln_w, const float *ln_b, float eps,
              uint32_t M) {
  if (sizeof(WT) == 2 && l->N >= 32u * 2 * 148) return launch_gemv<WT, MR, 4>(s, l, sg, x, ldx, ln_w, ln_b, eps, M);
  if (l->N >= 16u * 148) return launch_gemv<WT, MR, 2>(s, l, sg, x, ldx, ln_w, ln_b, eps, M);
  return launch_gemv<WT, MR, 1>(s, l, sg, x, ldx, ln_w, ln_b, eps, M);
}
template <typename WT>
int pick_m(cudaStream_t s, const greta_linear *l, const Segments &sg, const float *x, uint32_t ldx, const float *ln_w, const float *ln_b, float eps,
           uint32_t M) {
  if (M == 1) return pick_rows<WT, 1>(s, l, sg, x, ldx, ln_w, ln_b, eps, M);
  if (M == 2) return pick_rows<WT, 2>(s, l, sg, x, ldx, ln_w, ln_b, eps, M);
  if (M <= 4) return pick_rows<WT, 4>(s, l, sg, x, ldx, ln_w, ln_b, eps, M);
  return pick_rows<WT, 8>(s, l, sg, x, ldx, ln_w, ln_b, eps, M);
}

}  // namespace

namespace greta {
// Shared argument checks of the dense linears; fills the by-value segment list.
int check_linear(const char *what, const greta_linear *l, Segments *sg) {
  GRETA_REQUIRE(l && l->w && l->N && l->K, "%s: null or empty linear", what);
  GRETA_REQUIRE(l->fmt == GRETA_FMT_BF16 || l->fmt == GRETA_FMT_F32 || l->fmt == GRETA_FMT_F16, "%s: weight format %d is not dense (BF16, F16 or F32)", what,
                l->fmt);
  GRETA_REQUIRE(l->ldw % 64 == 0 && l->ldw >= l->K && aligned16(l->w), "%s: ldw=%u K=%u or a misaligned weight", what, l->ldw, l->K);
  GRETA_REQUIRE(l->n_segments >= 1 && l->n_segments <= GRETA_MAX_SEGMENTS, "%s: %u segments", what, l->n_segments);
  uint32_t row = 0;
  for (uint32_t i = 0; i < l->n_segments; ++i) {
    const greta_out_segment &g = l->seg[i];
    GRETA_REQUIRE(g.row0 == row && g.rows && g.out, "%s: segment %u leaves a gap or has no output", what, i);
    GRETA_REQUIRE(!g.accumulate || g.out_fmt == GRETA_OUT_F32, "%s: segment %u accumulates into a format other than fp32", what, i);
    GRETA_REQUIRE(g.act != GRETA_ACT_SOFTPLUS_DECAY || g.rate, "%s: segment %u has no decay rates", what, i);
    row += g.rows;
    sg->s[i] = g;
  }
  GRETA_REQUIRE(row == l->N, "%s: segments cover %u of %u rows", what, row, l->N);
  sg->n = l->n_segments;
  return GRETA_OK;
}
}  // namespace greta

extern "C" {

int greta_cuda_linear_gemv(greta_stream_t stream, const greta_linear *l, const float *x, uint32_t ldx, const float *ln_w, const float *ln_b, float eps,
                           uint32_t M) {
  Segments sg{};
  if (int rc = check_linear("linear_gemv", l, &sg)) return rc;
  GRETA_REQUIRE(M >= 1 && M <= 8, "linear_gemv: M=%u (1..8)", M);
  GRETA_REQUIRE(x && ldx >= l->K && (ln_w || !ln_b), "linear_gemv: bad activations or norm");
  GRETA_REQUIRE(l->fmt != GRETA_FMT_F16, "linear_gemv: weights must be BF16 or F32");
  cudaStream_t s = (cudaStream_t)stream;
  return l->fmt == GRETA_FMT_BF16 ? pick_m<__nv_bfloat16>(s, l, sg, x, ldx, ln_w, ln_b, eps, M) : pick_m<float>(s, l, sg, x, ldx, ln_w, ln_b, eps, M);
}

int greta_cuda_layer_norm(greta_stream_t stream, const float *x, const float *w, const float *b, float eps, void *out, int out_fmt, uint32_t M, uint32_t D,
                          uint32_t ld_out) {
  if (M == 0) return GRETA_OK;
  GRETA_REQUIRE(x && w && b && out && D && ld_out >= D, "layer_norm: bad argument");
  GRETA_REQUIRE(out_fmt == GRETA_OUT_F32 || out_fmt == GRETA_OUT_F16 || out_fmt == GRETA_OUT_BF16, "layer_norm: output format %d", out_fmt);
  const int vec = D <= 8192 && D % 4 == 0 && ld_out % 4 == 0 && aligned16(x) && aligned16(w) && aligned16(b) && aligned16(out);
  GRETA_CUDA_TRY(launch_pdl(norm_kernel<false>, dim3(M), dim3(256), 0, (cudaStream_t)stream, x, D, w, b, eps, out, out_fmt, D, ld_out, vec));
  return launched("norm_kernel");
}

int greta_cuda_rms_norm(greta_stream_t stream, const float *x, uint32_t ldx, const float *w, float eps, void *out, int out_fmt, uint32_t M, uint32_t D,
                        uint32_t ld_out) {
  if (M == 0) return GRETA_OK;
  GRETA_REQUIRE(x && w && out && D && ldx >= D && ld_out >= D, "rms_norm: bad argument");
  GRETA_REQUIRE(out_fmt == GRETA_OUT_F32 || out_fmt == GRETA_OUT_F16 || out_fmt == GRETA_OUT_BF16, "rms_norm: output format %d", out_fmt);
  const int vec = D <= 8192 && D % 4 == 0 && ldx % 4 == 0 && ld_out % 4 == 0 && aligned16(x) && aligned16(w) && aligned16(out);
  GRETA_CUDA_TRY(launch_pdl(norm_kernel<true>, dim3(M), dim3(256), 0, (cudaStream_t)stream, x, ldx, w, static_cast<const float *>(nullptr), eps, out, out_fmt,
                            D, ld_out, vec));
  return launched("norm_kernel");
}

int greta_cuda_embedding_positions(greta_stream_t stream, const int32_t *tokens, const void *table, const void *pos_table, int fmt, float *out, uint32_t M,
                                   uint32_t D, uint32_t vocab, uint32_t max_positions, const uint32_t *d_pos, uint32_t pos0) {
  if (M == 0 || D == 0) return GRETA_OK;
  GRETA_REQUIRE(tokens && table && out, "embedding_positions: null pointer");
  GRETA_REQUIRE(fmt == GRETA_FMT_BF16 || fmt == GRETA_FMT_F32, "embedding_positions: table format %d", fmt);
  const unsigned grid = (unsigned)(((size_t)M * D + 255) / 256);
  if (fmt == GRETA_FMT_BF16)
    GRETA_CUDA_TRY(launch_pdl(embedding_positions_kernel<__nv_bfloat16>, dim3(grid), dim3(256), 0, (cudaStream_t)stream, tokens, table, pos_table, out, M,
                              D, vocab, max_positions, d_pos, pos0));
  else
    GRETA_CUDA_TRY(launch_pdl(embedding_positions_kernel<float>, dim3(grid), dim3(256), 0, (cudaStream_t)stream, tokens, table, pos_table, out, M, D, vocab,
                              max_positions, d_pos, pos0));
  return launched("embedding_positions_kernel");
}

int greta_cuda_embedding_scaled(greta_stream_t stream, const int32_t *tokens, const void *table, int fmt, uint32_t ld, float scale, float *out, uint32_t M,
                                uint32_t D, uint32_t vocab) {
  if (M == 0 || D == 0) return GRETA_OK;
  GRETA_REQUIRE(tokens && table && out && ld >= D, "embedding_scaled: bad argument");
  GRETA_REQUIRE(fmt == GRETA_FMT_BF16 || fmt == GRETA_FMT_F32, "embedding_scaled: table format %d", fmt);
  const unsigned grid = (unsigned)(((size_t)M * D + 255) / 256);
  if (fmt == GRETA_FMT_BF16)
    GRETA_CUDA_TRY(launch_pdl(embedding_scaled_kernel<__nv_bfloat16>, dim3(grid), dim3(256), 0, (cudaStream_t)stream, tokens,
                              static_cast<const __nv_bfloat16 *>(table), ld, scale, out, M, D, vocab));
  else
    GRETA_CUDA_TRY(launch_pdl(embedding_scaled_kernel<float>, dim3(grid), dim3(256), 0, (cudaStream_t)stream, tokens, static_cast<const float *>(table), ld,
                              scale, out, M, D, vocab));
  return launched("embedding_scaled_kernel");
}

int greta_cuda_gather_rows(greta_stream_t stream, const float *x, uint32_t D, const uint32_t *rows, uint32_t n, float *out) {
  if (n == 0) return GRETA_OK;
  GRETA_REQUIRE(x && rows && out && n <= 64, "gather_rows: bad argument");
  RowList list{};
  for (uint32_t i = 0; i < n; ++i) list.r[i] = rows[i];
  gather_rows_kernel<<<n, 256, 0, (cudaStream_t)stream>>>(x, D, list, out);
  return launched("gather_rows_kernel");
}

}  // extern "C"
