// Norm-after-sum residual stream kept in fp32, and the small element-wise steps around it.
//
//   sum_layer_norm:  z = alpha * x + y  (or z = x when there is no branch output), then the bias-free
//                    layer norm  (z - mean) / sqrt(var + eps) * w * out_scale,  var = mean((z - mean)^2).
//                    The sum, both statistics and the product are fp32; the normalised row is written as
//                    the new fp32 residual stream and, rounded once, as the next projection's bf16 input.
//                    With a row list it gathers (final norm of the rows whose logits are wanted).
//   embed_rows:      token embedding -> fp32 residual stream + bf16 copy.
//   output_norm_join: the residual of a design that norms what a sublayer PUTS OUT, with weight and bias:
//                    z = x + (v - mean(v)) / sqrt(var(v) + eps) * wb + bb;  z is the new fp32 stream and, rounded once,
//                    the next sublayer's input.  v is a row of a projection's output, or (routed form) the sum over
//                    the chosen experts' rows plus the shared expert's row times sigmoid(its gate logit): the combine
//                    of a routed feed-forward, the norm and the sum in one pass.  With a second weight (wa, ba) the
//                    normed z is written instead (final norm), also for a list of wanted rows (gather).
//   embed_sinusoid:  token row + sinusoidal position vector, optionally through the same norm, in one pass.
//   relu2:           max(u, 0)^2, the feed-forward activation between the up and down projections.
// One CTA per row, the row is staged in shared memory once (two-pass variance, no E[z^2] - E[z]^2).
#include "common.cuh"
#include "runtime.h"
#include "../../include/b200.h"

namespace b200 {

__device__ __forceinline__ float pn_f32(float v) { return v; }
__device__ __forceinline__ float pn_f32(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void pn_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void pn_store(bf16* p, float v) { *p = __float2bfloat16_rn(v); }

__device__ __forceinline__ float pn_block_sum(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = (blockDim.x + 31) >> 5;
  __syncthreads();                       // red may still be read by the previous reduction
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = lane < nw ? red[lane] : 0.f;
  return warp_sum(t);
}

template <typename TY, typename TO>
__global__ void __launch_bounds__(256)
sum_layer_norm_kernel(const TY* __restrict__ y, int64_t ldy, const float* x_in, const int32_t* __restrict__ rows,
                      const bf16* __restrict__ w, float* x_out, TO* xb_out, int D, float alpha, float eps,
                      float out_scale) {
  extern __shared__ float zrow[];
  __shared__ float red[32];
  const int r = blockIdx.x;
  const int src = rows != nullptr ? rows[r] : r;
  const float* xr = x_in + (size_t)src * D;
  float s = 0.f;
  for (int i = threadIdx.x; i < D; i += blockDim.x) {
    float z = xr[i];
    if (y != nullptr) z = fmaf(alpha, z, pn_f32(y[(size_t)r * ldy + i]));
    zrow[i] = z;
    s += z;
  }
  const float mean = pn_block_sum(s, red) / (float)D;
  float q = 0.f;
  for (int i = threadIdx.x; i < D; i += blockDim.x) {
    const float d = zrow[i] - mean;
    q = fmaf(d, d, q);
  }
  const float rstd = 1.0f / sqrtf(pn_block_sum(q, red) / (float)D + eps);
  for (int i = threadIdx.x; i < D; i += blockDim.x) {
    const float o = (zrow[i] - mean) * rstd * __bfloat162float(w[i]) * out_scale;
    if (x_out != nullptr) x_out[(size_t)r * D + i] = o;
    if (xb_out != nullptr) pn_store(xb_out + (size_t)r * D + i, o);
  }
}

template <typename TO>
__global__ void embed_rows_kernel(const int32_t* __restrict__ ids, const bf16* __restrict__ table, float* x_out,
                                  TO* xb_out, int T, int D, int V) {
  const size_t n = (size_t)T * D;
  for (size_t i = blockIdx.x * (size_t)blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
    const int t = (int)(i / D), d = (int)(i % D);
    const int id = ids[t];
    const bf16 v = (id >= 0 && id < V) ? table[(size_t)id * D + d] : __float2bfloat16_rn(0.f);
    x_out[i] = __bfloat162float(v);
    if (xb_out != nullptr) pn_store(xb_out + i, __bfloat162float(v));
  }
}

__device__ __forceinline__ float4 pn_ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 pn_ld4(const bf16* p) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  return make_float4(bf16_lo(r.x), bf16_hi(r.x), bf16_lo(r.y), bf16_hi(r.y));
}
__device__ __forceinline__ void pn_st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void pn_st4(bf16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}
template <int V> struct PnVec { float v[V]; };
template <int V, typename T> __device__ __forceinline__ PnVec<V> pn_ldv(const T* p) {
  PnVec<V> r;
  if constexpr (V == 4) {
    const float4 q = pn_ld4(p);
    r.v[0] = q.x; r.v[1] = q.y; r.v[2] = q.z; r.v[3] = q.w;
  } else {
    r.v[0] = pn_f32(p[0]);
  }
  return r;
}
template <int V, typename T> __device__ __forceinline__ void pn_stv(T* p, const PnVec<V>& r) {
  if constexpr (V == 4) pn_st4(p, make_float4(r.v[0], r.v[1], r.v[2], r.v[3]));
  else pn_store(p, r.v[0]);
}

constexpr int kOnjMaxTop = 16;

struct OnjRouted {
  const float* yp;            // [rows of the permuted (token, expert) space][D], weighted expert outputs
  const int32_t* pair_row;    // [T * K]
  int K;
  const float* shared;        // [T][D] or null
  const float* gate;          // logits of the shared expert's gate, one per token at gate[t * ld_gate], or null (no gate)
  int64_t ld_gate;
};

// Two-pass moments of the staged row: every thread reads back only what it staged itself.
template <int V>
__device__ __forceinline__ void row_moments(const float* zrow, float s, int D, float eps, float* red, float& mean, float& rstd) {
  const int i0 = threadIdx.x * V, step = blockDim.x * V;
  mean = pn_block_sum(s, red) / (float)D;
  float q = 0.f;
  for (int i = i0; i < D; i += step) {
    const PnVec<V> z = pn_ldv<V>(zrow + i);
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const float d = z.v[e] - mean;
      q = fmaf(d, d, q);
    }
  }
  rstd = 1.0f / sqrtf(pn_block_sum(q, red) / (float)D + eps);
}

template <typename TO, int V, bool ROUTED>
__global__ void __launch_bounds__(256)
output_norm_join_kernel(const float* x_in, const float* __restrict__ y, OnjRouted ro, const bf16* __restrict__ wb,
                        const bf16* __restrict__ bb, const int32_t* __restrict__ rows, const bf16* __restrict__ wa,
                        const bf16* __restrict__ ba, float* x_out, TO* h_out, int D, float eps) {
  extern __shared__ __align__(16) float zrow[];
  __shared__ float red[32];
  __shared__ int prow[kOnjMaxTop];
  const int r = blockIdx.x;
  const size_t t = rows != nullptr ? rows[r] : r, src = t * D;
  const int i0 = threadIdx.x * V, step = blockDim.x * V;
  float s = 0.f;
  if (ROUTED || y != nullptr) {
    float sg = 1.f;
    if constexpr (ROUTED) {
      if (threadIdx.x < ro.K) prow[threadIdx.x] = ro.pair_row[t * ro.K + threadIdx.x];
      if (ro.gate != nullptr) sg = 1.0f / (1.0f + expf(-ro.gate[t * ro.ld_gate]));
      __syncthreads();
    }
    for (int i = i0; i < D; i += step) {
      PnVec<V> v;
      if constexpr (ROUTED) {
        v = pn_ldv<V>(ro.yp + (size_t)prow[0] * D + i);
        for (int j = 1; j < ro.K; ++j) {
          const PnVec<V> a = pn_ldv<V>(ro.yp + (size_t)prow[j] * D + i);
#pragma unroll
          for (int e = 0; e < V; ++e) v.v[e] += a.v[e];
        }
        if (ro.shared != nullptr) {
          const PnVec<V> a = pn_ldv<V>(ro.shared + src + i);
#pragma unroll
          for (int e = 0; e < V; ++e) v.v[e] = fmaf(sg, a.v[e], v.v[e]);
        }
      } else {
        v = pn_ldv<V>(y + src + i);
      }
      pn_stv<V>(zrow + i, v);
#pragma unroll
      for (int e = 0; e < V; ++e) s += v.v[e];
    }
    float mean, rstd;
    row_moments<V>(zrow, s, D, eps, red, mean, rstd);
    s = 0.f;
    for (int i = i0; i < D; i += step) {
      PnVec<V> v = pn_ldv<V>(zrow + i);
      const PnVec<V> x = pn_ldv<V>(x_in + src + i), w = pn_ldv<V>(wb + i), b = pn_ldv<V>(bb + i);
#pragma unroll
      for (int e = 0; e < V; ++e) {
        v.v[e] = x.v[e] + fmaf((v.v[e] - mean) * rstd, w.v[e], b.v[e]);
        s += v.v[e];
      }
      if (x_out != nullptr) pn_stv<V>(x_out + (size_t)r * D + i, v);
      if (wa != nullptr) pn_stv<V>(zrow + i, v);
      else if (h_out != nullptr) pn_stv<V>(h_out + (size_t)r * D + i, v);
    }
  } else {
    for (int i = i0; i < D; i += step) {
      const PnVec<V> v = pn_ldv<V>(x_in + src + i);
      pn_stv<V>(zrow + i, v);
#pragma unroll
      for (int e = 0; e < V; ++e) s += v.v[e];
    }
  }
  if (wa == nullptr || h_out == nullptr) return;
  float mean, rstd;
  row_moments<V>(zrow, s, D, eps, red, mean, rstd);
  for (int i = i0; i < D; i += step) {
    PnVec<V> v = pn_ldv<V>(zrow + i);
    const PnVec<V> w = pn_ldv<V>(wa + i), b = pn_ldv<V>(ba + i);
#pragma unroll
    for (int e = 0; e < V; ++e) v.v[e] = fmaf((v.v[e] - mean) * rstd, w.v[e], b.v[e]);
    pn_stv<V>(h_out + (size_t)r * D + i, v);
  }
}

// x = table[id] + (sin, cos) pairs of position * freq[i], the angle formed and reduced to [-pi, pi] in fp64;
// w != null: x goes through the layer norm with weight and bias first
template <typename TO>
__global__ void __launch_bounds__(256)
embed_sinusoid_kernel(const int32_t* __restrict__ ids, const int32_t* __restrict__ positions, const bf16* __restrict__ table,
                      const double* __restrict__ freq, const bf16* __restrict__ w, const bf16* __restrict__ b, float* x_out,
                      TO* xb_out, int D, int vocab, float eps) {
  extern __shared__ __align__(16) float zrow[];
  __shared__ float red[32];
  const int t = blockIdx.x;
  int id = ids[t];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const double p = (double)positions[t];
  const bf16* e = table + (size_t)id * D;
  float s = 0.f;
  for (int i = 2 * threadIdx.x; i < D; i += 2 * blockDim.x) {
    const double a = p * freq[i >> 1];
    float sn, cs;
    sincosf((float)(a - rint(a * 0.15915494309189535) * 6.283185307179586), &sn, &cs);
    const float v0 = __bfloat162float(e[i]) + sn;
    zrow[i] = v0;
    s += v0;
    if (i + 1 < D) {
      const float v1 = __bfloat162float(e[i + 1]) + cs;
      zrow[i + 1] = v1;
      s += v1;
    }
  }
  float mean = 0.f, rstd = 1.f;
  if (w != nullptr) {
    mean = pn_block_sum(s, red) / (float)D;
    float q = 0.f;
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
      const float d = zrow[i] - mean;
      q = fmaf(d, d, q);
    }
    rstd = 1.0f / sqrtf(pn_block_sum(q, red) / (float)D + eps);
  } else {
    __syncthreads();
  }
  for (int i = threadIdx.x; i < D; i += blockDim.x) {
    float o = zrow[i];
    if (w != nullptr) o = fmaf((o - mean) * rstd, __bfloat162float(w[i]), __bfloat162float(b[i]));
    x_out[(size_t)t * D + i] = o;
    if (xb_out != nullptr) pn_store(xb_out + (size_t)t * D + i, o);
  }
}

template <typename T>
__global__ void relu2_kernel(const T* __restrict__ u, T* out, size_t n) {
  for (size_t i = blockIdx.x * (size_t)blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
    const float v = fmaxf(pn_f32(u[i]), 0.f);
    pn_store(out + i, v * v);
  }
}

static int ew_blocks(size_t n) {
  size_t b = (n + 255) / 256;
  return (int)(b < 1 ? 1 : (b > 4096 ? 4096 : b));
}

}  // namespace b200

using namespace b200;

extern "C" int b200_sum_layer_norm(const void* y, int y_f32, int64_t ldy, const float* x_in, const int32_t* rows,
                                   const void* w, float* x_out, void* xb_out, int xb_f32, int T, int D, float alpha,
                                   float eps, float out_scale, void* stream) {
  B200_REQUIRE(T >= 0 && D > 0, "sum_layer_norm: bad shape T=%d D=%d", T, D);
  if (T == 0) return B200_OK;
  cudaStream_t s = (cudaStream_t)stream;
  const size_t smem = (size_t)D * sizeof(float);
  B200_REQUIRE(smem <= 48 * 1024, "sum_layer_norm: D=%d exceeds the staged row (12288)", D);
  const bf16* wp = (const bf16*)w;
#define B200_SLN(TY, TO)                                                                                      \
  sum_layer_norm_kernel<TY, TO><<<T, 256, smem, s>>>((const TY*)y, ldy, x_in, rows, wp, x_out, (TO*)xb_out, D, \
                                                     alpha, eps, out_scale)
  if (y_f32 && xb_f32) B200_SLN(float, float);
  else if (y_f32) B200_SLN(float, bf16);
  else if (xb_f32) B200_SLN(bf16, float);
  else B200_SLN(bf16, bf16);
#undef B200_SLN
  return b200_check_launch("b200_sum_layer_norm");
}

extern "C" int b200_embed_rows_f32(const int32_t* ids, const void* table, float* x_out, void* xb_out, int xb_f32,
                                   int T, int D, int V, void* stream) {
  B200_REQUIRE(T >= 0 && D > 0 && V > 0, "embed_rows: bad shape");
  if (T == 0) return B200_OK;
  cudaStream_t s = (cudaStream_t)stream;
  const int blocks = ew_blocks((size_t)T * D);
  if (xb_f32)
    embed_rows_kernel<float><<<blocks, 256, 0, s>>>(ids, (const bf16*)table, x_out, (float*)xb_out, T, D, V);
  else
    embed_rows_kernel<bf16><<<blocks, 256, 0, s>>>(ids, (const bf16*)table, x_out, (bf16*)xb_out, T, D, V);
  return b200_check_launch("b200_embed_rows_f32");
}

extern "C" int b200_relu2(const void* u, void* out, int f32, int64_t n, void* stream) {
  B200_REQUIRE(n >= 0, "relu2: bad size");
  if (n == 0) return B200_OK;
  cudaStream_t s = (cudaStream_t)stream;
  if (f32) relu2_kernel<float><<<ew_blocks((size_t)n), 256, 0, s>>>((const float*)u, (float*)out, (size_t)n);
  else relu2_kernel<bf16><<<ew_blocks((size_t)n), 256, 0, s>>>((const bf16*)u, (bf16*)out, (size_t)n);
  return b200_check_launch("b200_relu2");
}

extern "C" int b200_output_norm_join(const float* x_in, const float* y, const float* yp, const int32_t* pair_row, int top_k,
                                     const float* shared, const float* gate, int64_t ld_gate, const void* wb,
                                     const void* bb, const int32_t* rows, const void* wa, const void* ba, float* x_out,
                                     void* h_out, int h_f32, int T, int D, float eps, void* stream) {
  B200_REQUIRE(T >= 0 && D > 0 && x_in != nullptr, "output_norm_join: bad arguments T=%d D=%d", T, D);
  B200_REQUIRE(y == nullptr || yp == nullptr, "output_norm_join: one source of the sublayer's output");
  B200_REQUIRE((y == nullptr && yp == nullptr) || (wb != nullptr && bb != nullptr), "output_norm_join: the output's norm needs weight and bias");
  B200_REQUIRE(wa == nullptr || (ba != nullptr && h_out != nullptr), "output_norm_join: the final norm needs a bias and an output");
  B200_REQUIRE(rows == nullptr || x_out == nullptr, "output_norm_join: the gather form writes the normed rows only");
  B200_REQUIRE(yp == nullptr || (pair_row != nullptr && top_k >= 1 && top_k <= kOnjMaxTop), "output_norm_join: top_k=%d (1 .. %d)", top_k, kOnjMaxTop);
  if (T == 0) return B200_OK;
  const size_t smem = (size_t)D * sizeof(float);
  B200_REQUIRE(smem <= 48 * 1024, "output_norm_join: D=%d exceeds the staged row (12288)", D);
  cudaStream_t s = (cudaStream_t)stream;
  auto al = [](const void* p, int n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; };
  const bool vec = D % 4 == 0 && al(x_in, 16) && al(y, 16) && al(yp, 16) && al(shared, 16) && al(x_out, 16) && al(wb, 8) &&
                   al(bb, 8) && al(wa, 8) && al(ba, 8) && al(h_out, h_f32 ? 16 : 8);
  const int per = vec ? 4 : 1, want = (D + per - 1) / per;
  const int threads = want >= 256 ? 256 : (want + 31) / 32 * 32;
  const OnjRouted ro{yp, pair_row, top_k, shared, gate, ld_gate};
#define B200_ONJ(TO, V, R)                                                                                                   \
  output_norm_join_kernel<TO, V, R><<<T, threads, smem, s>>>(x_in, y, ro, (const bf16*)wb, (const bf16*)bb, rows,             \
                                                             (const bf16*)wa, (const bf16*)ba, x_out, (TO*)h_out, D, eps)
#define B200_ONJ2(TO)                                                                      \
  do {                                                                                     \
    if (yp != nullptr) { if (vec) B200_ONJ(TO, 4, true); else B200_ONJ(TO, 1, true); }     \
    else { if (vec) B200_ONJ(TO, 4, false); else B200_ONJ(TO, 1, false); }                 \
  } while (0)
  if (h_f32) B200_ONJ2(float);
  else B200_ONJ2(bf16);
#undef B200_ONJ2
#undef B200_ONJ
  return b200_check_launch("b200_output_norm_join");
}

extern "C" int b200_embed_sinusoid(const int32_t* ids, const int32_t* positions, const void* table, const double* freq,
                                   const void* w, const void* b, float* x_out, void* xb_out, int xb_f32, int T, int D,
                                   int vocab, float eps, void* stream) {
  B200_REQUIRE(T >= 0 && D > 0 && vocab > 0, "embed_sinusoid: bad shape");
  B200_REQUIRE(w == nullptr || b != nullptr, "embed_sinusoid: the norm needs weight and bias");
  if (T == 0) return B200_OK;
  const size_t smem = (size_t)D * sizeof(float);
  B200_REQUIRE(smem <= 48 * 1024, "embed_sinusoid: D=%d exceeds the staged row (12288)", D);
  cudaStream_t s = (cudaStream_t)stream;
  if (xb_f32)
    embed_sinusoid_kernel<float><<<T, 256, smem, s>>>(ids, positions, (const bf16*)table, freq, (const bf16*)w, (const bf16*)b,
                                                      x_out, (float*)xb_out, D, vocab, eps);
  else
    embed_sinusoid_kernel<bf16><<<T, 256, smem, s>>>(ids, positions, (const bf16*)table, freq, (const bf16*)w, (const bf16*)b,
                                                     x_out, (bf16*)xb_out, D, vocab, eps);
  return b200_check_launch("b200_embed_sinusoid");
}
