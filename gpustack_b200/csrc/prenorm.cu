// Pre-norm residual stream kept in fp32, for layers whose branches are summed into the stream un-normalised.
//
//   add_rms_norm_f32:  z = x_in + a + b + c   (each of a, b, c optional: the branch outputs of the layer before --
//                      a mixer and a feed-forward that ran side by side on one normed input -- and a third
//                      addend such as the embedding output that a repeated span of layers takes in again),
//                      x_out = z  (the new fp32 stream),   xb_out = z / sqrt(mean(z^2) + eps) * w  (the next
//                      layer's input, rounded once to bf16, or fp32).
//                      The sum, the statistic and the product are fp32 in a fixed order (x, a, b, c).
//                      With a row list it gathers: row r reads x_in / a / b / c at rows[r] and writes row r of
//                      xb_out only (final norm of the rows whose logits are wanted).  Without w nothing is normed
//                      (the sum alone is written).
// One CTA per row; the summed row is staged in shared memory between the statistic and the product.
//
//   prenorm_join:      the same for layers whose mixer and feed-forward each have a norm in front,
//                      z = x_in + c,  x_out = z,  h_out = z / sqrt(mean(z^2) + eps) * w * out_scale, where the contribution c is
//                        * nothing, or one fp32 row y;
//                        * the normed outputs of a pair of mixers, ya * y / rms(y) * wy + yb * y2 / rms(y2) * wy2;
//                        * a routed feed-forward's rows: sum_j yp[pair_row[t K + j]] (+ shared[t]) in a fixed order.
//                      With a row list it gathers (h_out only).  A row lives in the threads' registers from the loads to
//                      the last store: nothing is read twice.
#include "common.cuh"
#include "runtime.h"
#include "../../include/b200.h"

namespace b200 {

__device__ __forceinline__ void prn_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void prn_store(bf16* p, float v) { *p = __float2bfloat16_rn(v); }

template <typename TO, bool VEC>
__global__ void __launch_bounds__(256)
add_rms_norm_f32_kernel(const float* x_in, const float* __restrict__ a, const float* __restrict__ b,
                        const float* __restrict__ c, const int32_t* __restrict__ rows, const bf16* __restrict__ w,
                        float* x_out, TO* xb_out, int D, float eps) {
  extern __shared__ __align__(16) float zrow[];
  __shared__ float red[32];
  const int r = blockIdx.x;
  const size_t src = (size_t)(rows != nullptr ? rows[r] : r) * D;
  float ss = 0.f;
  if (VEC) {
    for (int i = threadIdx.x * 4; i < D; i += blockDim.x * 4) {
      float4 z = *reinterpret_cast<const float4*>(x_in + src + i);
      if (a != nullptr) { const float4 v = *reinterpret_cast<const float4*>(a + src + i); z.x += v.x; z.y += v.y; z.z += v.z; z.w += v.w; }
      if (b != nullptr) { const float4 v = *reinterpret_cast<const float4*>(b + src + i); z.x += v.x; z.y += v.y; z.z += v.z; z.w += v.w; }
      if (c != nullptr) { const float4 v = *reinterpret_cast<const float4*>(c + src + i); z.x += v.x; z.y += v.y; z.z += v.z; z.w += v.w; }
      *reinterpret_cast<float4*>(zrow + i) = z;
      if (x_out != nullptr) *reinterpret_cast<float4*>(x_out + (size_t)r * D + i) = z;
      ss = fmaf(z.x, z.x, fmaf(z.y, z.y, fmaf(z.z, z.z, fmaf(z.w, z.w, ss))));
    }
  } else {
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
      float z = x_in[src + i];
      if (a != nullptr) z += a[src + i];
      if (b != nullptr) z += b[src + i];
      if (c != nullptr) z += c[src + i];
      zrow[i] = z;
      if (x_out != nullptr) x_out[(size_t)r * D + i] = z;
      ss = fmaf(z, z, ss);
    }
  }
  if (w == nullptr || xb_out == nullptr) return;
  ss = warp_sum(ss);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = (blockDim.x + 31) >> 5;
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  float t = lane < nw ? red[lane] : 0.f;
  t = warp_sum(t);
  const float rstd = 1.0f / sqrtf(t / (float)D + eps);
  // every thread reads back only what it staged itself: no barrier between the passes beyond the one above
  if (VEC) {
    for (int i = threadIdx.x * 4; i < D; i += blockDim.x * 4) {
      const float4 z = *reinterpret_cast<const float4*>(zrow + i);
      const uint2 wr = *reinterpret_cast<const uint2*>(w + i);
      const float o0 = z.x * rstd * bf16_lo(wr.x), o1 = z.y * rstd * bf16_hi(wr.x);
      const float o2 = z.z * rstd * bf16_lo(wr.y), o3 = z.w * rstd * bf16_hi(wr.y);
      TO* dst = xb_out + (size_t)r * D + i;
      if (sizeof(TO) == 4) {
        *reinterpret_cast<float4*>(dst) = make_float4(o0, o1, o2, o3);
      } else {
        *reinterpret_cast<uint2*>(dst) = make_uint2(pack_bf16(o0, o1), pack_bf16(o2, o3));
      }
    }
  } else {
    for (int i = threadIdx.x; i < D; i += blockDim.x)
      prn_store(xb_out + (size_t)r * D + i, zrow[i] * rstd * __bfloat162float(w[i]));
  }
}

// ---- prenorm_join
enum { kJoinRow = 0, kJoinPair = 1, kJoinRouted = 2 };
constexpr int kJoinMaxTop = 32;

struct JoinArgs {
  const float* x_in;
  const float* y;                  // kJoinRow (or null), kJoinPair
  const float* y2;                 // kJoinPair
  const bf16* wy;
  const bf16* wy2;
  float ya, yb;
  const float* yp;                 // kJoinRouted: expert rows, the rows of each token, choices per token, shared expert's rows
  const int32_t* pair_row;
  const float* shared;
  int K;
  const int32_t* rows;
  const bf16* w;
  float* x_out;
  void* h_out;
  int D;
  float eps, out_scale;
};

template <int V> struct JoinVec { float v[V]; };
template <int V>
__device__ __forceinline__ JoinVec<V> jn_ld(const float* p) {
  JoinVec<V> r;
  if constexpr (V == 4) { const float4 t = *reinterpret_cast<const float4*>(p); r.v[0] = t.x; r.v[1] = t.y; r.v[2] = t.z; r.v[3] = t.w; }
  else r.v[0] = *p;
  return r;
}
template <int V>
__device__ __forceinline__ JoinVec<V> jn_ld(const bf16* p) {
  JoinVec<V> r;
  if constexpr (V == 4) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    r.v[0] = bf16_lo(t.x); r.v[1] = bf16_hi(t.x); r.v[2] = bf16_lo(t.y); r.v[3] = bf16_hi(t.y);
  } else r.v[0] = __bfloat162float(*p);
  return r;
}
template <int V>
__device__ __forceinline__ void jn_st(float* p, const JoinVec<V>& r) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
  else *p = r.v[0];
}
template <int V>
__device__ __forceinline__ void jn_st(bf16* p, const JoinVec<V>& r) {
  if constexpr (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(r.v[0], r.v[1]), pack_bf16(r.v[2], r.v[3]));
  else *p = __float2bfloat16_rn(r.v[0]);
}

// sums of two values over the CTA, the same in every thread (warps added in order)
__device__ __forceinline__ float2 jn_block_sum(float a, float b, float2* red) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  a = warp_sum(a);
  b = warp_sum(b);
  __syncthreads();                 // the last use of red is over
  if (lane == 0) red[warp] = make_float2(a, b);
  __syncthreads();
  float2 t = lane < nw ? red[lane] : make_float2(0.f, 0.f);
  return make_float2(warp_sum(t.x), warp_sum(t.y));
}

template <typename TO, int V, int MODE>
__global__ void __launch_bounds__(1024)
prenorm_join_kernel(JoinArgs a) {
  constexpr int N = 16 / V;        // pieces a thread can hold
  __shared__ float2 red[32];
  __shared__ int prow[kJoinMaxTop];
  const int r = blockIdx.x, D = a.D;
  const size_t t = a.rows != nullptr ? a.rows[r] : r, src = t * D;
  const int i0 = threadIdx.x * V, step = blockDim.x * V;
  JoinVec<V> z[N];
  if constexpr (MODE == kJoinPair) {
    JoinVec<V> y2[N];
    float s1 = 0.f, s2 = 0.f;
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int i = i0 + n * step;
      if (i >= D) break;
      z[n] = jn_ld<V>(a.y + src + i);
      y2[n] = jn_ld<V>(a.y2 + src + i);
    }
#pragma unroll
    for (int n = 0; n < N; ++n) {
      if (i0 + n * step >= D) break;
#pragma unroll
      for (int e = 0; e < V; ++e) { s1 = fmaf(z[n].v[e], z[n].v[e], s1); s2 = fmaf(y2[n].v[e], y2[n].v[e], s2); }
    }
    const float2 ss = jn_block_sum(s1, s2, red);
    const float f1 = a.ya / sqrtf(ss.x / (float)D + a.eps), f2 = a.yb / sqrtf(ss.y / (float)D + a.eps);
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int i = i0 + n * step;
      if (i >= D) break;
      const JoinVec<V> x = jn_ld<V>(a.x_in + src + i), w1 = jn_ld<V>(a.wy + i), w2 = jn_ld<V>(a.wy2 + i);
#pragma unroll
      for (int e = 0; e < V; ++e) z[n].v[e] = x.v[e] + (z[n].v[e] * f1 * w1.v[e] + y2[n].v[e] * f2 * w2.v[e]);
    }
  } else if constexpr (MODE == kJoinRouted) {
    if (threadIdx.x < a.K) prow[threadIdx.x] = a.pair_row[t * a.K + threadIdx.x];
    __syncthreads();
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int i = i0 + n * step;
      if (i >= D) break;
      JoinVec<V> c = jn_ld<V>(a.yp + (size_t)prow[0] * D + i);
      for (int j = 1; j < a.K; ++j) {
        const JoinVec<V> p = jn_ld<V>(a.yp + (size_t)prow[j] * D + i);
#pragma unroll
        for (int e = 0; e < V; ++e) c.v[e] += p.v[e];
      }
      if (a.shared != nullptr) {
        const JoinVec<V> p = jn_ld<V>(a.shared + src + i);
#pragma unroll
        for (int e = 0; e < V; ++e) c.v[e] += p.v[e];
      }
      z[n] = jn_ld<V>(a.x_in + src + i);
#pragma unroll
      for (int e = 0; e < V; ++e) z[n].v[e] += c.v[e];
    }
  } else {
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int i = i0 + n * step;
      if (i >= D) break;
      z[n] = jn_ld<V>(a.x_in + src + i);
      if (a.y != nullptr) {
        const JoinVec<V> y = jn_ld<V>(a.y + src + i);
#pragma unroll
        for (int e = 0; e < V; ++e) z[n].v[e] += y.v[e];
      }
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int n = 0; n < N; ++n) {
    const int i = i0 + n * step;
    if (i >= D) break;
    if (a.x_out != nullptr) jn_st<V>(a.x_out + (size_t)r * D + i, z[n]);
#pragma unroll
    for (int e = 0; e < V; ++e) ss = fmaf(z[n].v[e], z[n].v[e], ss);
  }
  if (a.h_out == nullptr) return;
  const float f = a.out_scale / sqrtf(jn_block_sum(ss, 0.f, red).x / (float)D + a.eps);
#pragma unroll
  for (int n = 0; n < N; ++n) {
    const int i = i0 + n * step;
    if (i >= D) break;
    const JoinVec<V> w = jn_ld<V>(a.w + i);
#pragma unroll
    for (int e = 0; e < V; ++e) z[n].v[e] *= f * w.v[e];
    jn_st<V>(reinterpret_cast<TO*>(a.h_out) + (size_t)r * D + i, z[n]);
  }
}

}  // namespace b200

using namespace b200;

extern "C" int b200_add_rms_norm_f32(const float* x_in, const float* a, const float* b, const float* c,
                                     const int32_t* rows, const void* w, float* x_out, void* xb_out, int xb_f32, int T,
                                     int D, float eps, void* stream) {
  B200_REQUIRE(T >= 0 && D > 0 && x_in != nullptr, "add_rms_norm_f32: bad arguments T=%d D=%d", T, D);
  B200_REQUIRE(rows == nullptr || x_out == nullptr, "add_rms_norm_f32: the gather form writes the normed rows only");
  if (T == 0) return B200_OK;
  const size_t smem = (size_t)D * sizeof(float);
  B200_REQUIRE(smem <= 48 * 1024, "add_rms_norm_f32: D=%d exceeds the staged row (12288)", D);
  cudaStream_t s = (cudaStream_t)stream;
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool vec = D % 4 == 0 && al(x_in) && al(a) && al(b) && al(c) && al(x_out) && al(xb_out) &&
                   (reinterpret_cast<uintptr_t>(w) & 7) == 0;
#define B200_ARN(TO, V)                                                                                            \
  add_rms_norm_f32_kernel<TO, V><<<T, 256, smem, s>>>(x_in, a, b, c, rows, (const bf16*)w, x_out, (TO*)xb_out, D, eps)
  if (xb_f32) { if (vec) B200_ARN(float, true); else B200_ARN(float, false); }
  else { if (vec) B200_ARN(bf16, true); else B200_ARN(bf16, false); }
#undef B200_ARN
  return b200_check_launch("b200_add_rms_norm_f32");
}

extern "C" int b200_prenorm_join(const float* x_in, const float* y, const float* y2, const void* wy, const void* wy2, float ya,
                                 float yb, const float* yp, const int32_t* pair_row, int top_k, const float* shared,
                                 const int32_t* rows, const void* w, float* x_out, void* h_out, int h_f32, int T, int D, float eps,
                                 float out_scale, void* stream) {
  B200_REQUIRE(T >= 0 && D > 0 && x_in != nullptr && (h_out == nullptr || w != nullptr), "prenorm_join: bad arguments T=%d D=%d", T, D);
  B200_REQUIRE(rows == nullptr || x_out == nullptr, "prenorm_join: the gather form writes the normed rows only");
  B200_REQUIRE(y2 == nullptr || (y != nullptr && wy != nullptr && wy2 != nullptr && yp == nullptr), "prenorm_join: a pair needs two rows and two weights");
  B200_REQUIRE(yp == nullptr || (y == nullptr && pair_row != nullptr && top_k >= 1 && top_k <= kJoinMaxTop), "prenorm_join: bad routed rows (K=%d)", top_k);
  if (T == 0) return B200_OK;
  auto al = [](const void* p, int n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; };
  const bool vec = D % 4 == 0 && al(x_in, 16) && al(y, 16) && al(y2, 16) && al(yp, 16) && al(shared, 16) && al(x_out, 16) && al(h_out, 16) &&
                   al(w, 8) && al(wy, 8) && al(wy2, 8);
  B200_REQUIRE(D <= 16384, "prenorm_join: D=%d exceeds 16384", D);
  // two pieces per thread keep enough loads in flight; wide rows take more pieces, not more than 1024 threads
  const int pieces = vec ? D / 4 : D, per = vec ? 2 : 4;
  int threads = ((pieces + per - 1) / per + 31) / 32 * 32;
  threads = threads < 64 ? 64 : (threads > 1024 ? 1024 : threads);
  const JoinArgs a{x_in, y, y2, (const bf16*)wy, (const bf16*)wy2, ya, yb, yp, pair_row, shared, top_k, rows, (const bf16*)w, x_out, h_out,
                   D, eps, out_scale};
  cudaStream_t s = (cudaStream_t)stream;
#define B200_PJ(TO, V, M) prenorm_join_kernel<TO, V, M><<<T, threads, 0, s>>>(a)
#define B200_PJ2(TO, V)                              \
  do {                                               \
    if (y2 != nullptr) B200_PJ(TO, V, kJoinPair);    \
    else if (yp != nullptr) B200_PJ(TO, V, kJoinRouted); \
    else B200_PJ(TO, V, kJoinRow);                   \
  } while (0)
  if (h_f32) { if (vec) B200_PJ2(float, 4); else B200_PJ2(float, 1); }
  else { if (vec) B200_PJ2(bf16, 4); else B200_PJ2(bf16, 1); }
#undef B200_PJ2
#undef B200_PJ
  return b200_check_launch("b200_prenorm_join");
}
