// Preparation of a softmax-attention mixer whose q, k and v pass a short causal convolution over time, in ONE launch:
// from the projected rows u = [q: H dk | k: G dk | v: G dv] of a step to attention-ready queries and cache pages.
//
//   y_t = sum_j w[:, j] u_(t - taps + 1 + j)         per channel, zeros before the sequence's start, no bias; inputs
//                                                    older than the step come from the sequence's ring
//   q, k:  y / sqrt(mean(y^2) + eps) * weight        per head over dk, one weight vector for all heads (optional)
//   q to its row of q_out, k and v to their pages (slot of the token), heads laid out wk / wv wide (>= dk / dv, the
//   columns behind dk / dv are zeros: a pair of widths that is no tensor-core tile is padded to one);
//   the step's last taps - 1 inputs of every sequence replace the ring's entries: ring[slot][p mod (taps - 1)][channel].
//
// A CTA takes 16 consecutive rows of one sequence and some head slots; the threads that own a channel walk the rows in
// order and keep the last taps - 1 inputs in registers, so a projected row is read once.  Only a sequence's first
// piece can need the ring (a piece is longer than the ring), and the SAME threads that read it there write the step's
// last inputs into it after their reads: no second launch, no race.  The statistics and the convolution are fp32.
#include "common.cuh"
#include "runtime.h"
#include "../../include/b200.h"

namespace b200 {

constexpr int kCapRows = 16;       // rows of one sequence per CTA
constexpr int kCapMaxTaps = 8;
constexpr int kCapWarps = 8;

__device__ __forceinline__ float ca_f32(float v) { return v; }
__device__ __forceinline__ float ca_f32(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void ca_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void ca_store(bf16* p, float v) { *p = __float2bfloat16_rn(v); }

struct CapArgs {
  const void* proj;
  int64_t ld;
  const float* conv_w;             // [C][taps], last column = current token
  const bf16* qnorm_w;             // null: no norm
  const bf16* knorm_w;
  float* ring;                     // [slots][taps - 1][C]; null when taps == 1
  const int32_t* cu_seq;           // every sequence of the step: prompt portions, then single rows
  const int32_t* ctx_lens;
  const int32_t* state_slots;
  const int32_t* tile_seq;         // row tiles of the prompt portions
  const int32_t* tile_q0;
  int n_pieces;                    // tiles * (tile_rows / 16): CTAs [0, n_pieces) along x; then one per single row
  int per_tile;                    // tile_rows / 16
  int n_prompt;                    // sequences with a prompt portion
  const int32_t* slots;            // cache slot of every row (-1: no write)
  void* q_out;
  void* k_cache;
  void* v_cache;
  int H, G, dk, dv, wk, wv, page, taps;
  float eps;
};

// What a CTA works on: rows [row0 + q0, + n) of the projection at positions ctx + q0 ..., of a sequence with qlen new rows
struct CapWork {
  int row0, q0, n, qlen, ctx, slot;
};
__device__ __forceinline__ CapWork cap_work(const CapArgs& a) {
  CapWork m;
  int s, q0 = 0;
  if ((int)blockIdx.x < a.n_pieces) {
    const int tile = blockIdx.x / a.per_tile;
    s = a.tile_seq[tile];
    q0 = a.tile_q0[tile] + kCapRows * (blockIdx.x - tile * a.per_tile);
  } else {
    s = a.n_prompt + (int)blockIdx.x - a.n_pieces;
  }
  m.row0 = a.cu_seq[s];
  m.q0 = q0;
  m.qlen = a.cu_seq[s + 1] - m.row0;
  m.n = min(kCapRows, m.qlen - q0);
  m.ctx = a.ctx_lens[s];
  m.slot = a.ring != nullptr ? a.state_slots[s] : -1;
  return m;
}

// LPH lanes share a head, each owns one 16-byte piece of it.
template <typename TA, int TAPS>
__global__ void __launch_bounds__(kCapWarps * 32)
conv_attn_prep_vec_kernel(CapArgs a, int lph) {
  constexpr int V = 16 / (int)sizeof(TA), R = TAPS - 1;
  const CapWork m = cap_work(a);
  if (m.n <= 0) return;
  const int lane = threadIdx.x & 31, per_warp = 32 / lph;
  const int hs = (blockIdx.y * kCapWarps + (threadIdx.x >> 5)) * per_warp + lane / lph;
  const int n_heads = a.H + 2 * a.G;
  const bool live = hs < n_heads;
  const bool is_q = hs < a.H, is_k = !is_q && hs < a.H + a.G;
  const int width = (is_q || is_k) ? a.dk : a.dv, wide = (is_q || is_k) ? a.wk : a.wv;
  const int col0 = (is_q || is_k) ? hs * a.dk : (a.H + a.G) * a.dk + (hs - a.H - a.G) * a.dv;
  const int d = (lane % lph) * V;
  const bool act = live && d < width, pad = live && !act && d < wide;
  const int c = col0 + d, C = (a.H + a.G) * a.dk + a.G * a.dv;
  const TA* src = reinterpret_cast<const TA*>(a.proj) + (size_t)m.row0 * a.ld + c;
  auto load = [&](int q, float (&x)[V]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(src + (size_t)q * a.ld);
    const TA* rv = reinterpret_cast<const TA*>(&raw);
#pragma unroll
    for (int i = 0; i < V; ++i) x[i] = ca_f32(rv[i]);
  };
  float w[TAPS][V], hist[R > 0 ? R : 1][V], nw[V];     // w[b]: weight of the input b positions back; hist[b]: that input, b + 1 back
  const bf16* norm = is_q ? a.qnorm_w : (is_k ? a.knorm_w : nullptr);
  if (act) {
#pragma unroll
    for (int i = 0; i < V; ++i) {
#pragma unroll
      for (int b = 0; b < TAPS; ++b) w[b][i] = a.conv_w[(size_t)(c + i) * TAPS + (R - b)];
      nw[i] = norm != nullptr ? __bfloat162float(norm[d + i]) : 1.0f;
    }
#pragma unroll
    for (int b = 0; b < R; ++b) {
      const int q = m.q0 - 1 - b, p = m.ctx + q;
      if (q >= 0) {
        load(q, hist[b]);
      } else if (p >= 0 && m.slot >= 0) {
        const float* rp = a.ring + ((size_t)m.slot * R + p % (R > 0 ? R : 1)) * C + c;
#pragma unroll
        for (int i = 0; i < V; ++i) hist[b][i] = rp[i];
      } else {
#pragma unroll
        for (int i = 0; i < V; ++i) hist[b][i] = 0.f;
      }
    }
    if (R > 0 && m.q0 == 0 && m.slot >= 0) {           // the ring has been read by its only readers: this step's last inputs
#pragma unroll
      for (int b = 0; b < R; ++b) {
        const int q = m.qlen - 1 - b;
        if (q < 0) break;
        float x[V];
        load(q, x);
        float* rp = a.ring + ((size_t)m.slot * R + (m.ctx + q) % (R > 0 ? R : 1)) * C + c;
#pragma unroll
        for (int i = 0; i < V; ++i) rp[i] = x[i];
      }
    }
  }
  float nxt[V];
#pragma unroll
  for (int i = 0; i < V; ++i) nxt[i] = 0.f;
  if (act) load(m.q0, nxt);
#pragma unroll 4
  for (int i_row = 0; i_row < m.n; ++i_row) {
    const int q = m.q0 + i_row;
    float cur[V], y[V];
#pragma unroll
    for (int i = 0; i < V; ++i) cur[i] = nxt[i];
    if (act && i_row + 1 < m.n) load(q + 1, nxt);
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < V; ++i) {
      y[i] = 0.f;
      if (act) {
        float v = w[0][i] * cur[i];
#pragma unroll
        for (int b = 0; b < R; ++b) v = fmaf(w[b + 1][i], hist[b][i], v);
        y[i] = v;
        ss = fmaf(v, v, ss);
      }
    }
#pragma unroll
    for (int b = R - 1; b > 0; --b)
#pragma unroll
      for (int i = 0; i < V; ++i) hist[b][i] = hist[b - 1][i];
    if (R > 0) {
#pragma unroll
      for (int i = 0; i < V; ++i) hist[0][i] = cur[i];
    }
    for (int o = lph >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);    // all lanes take part
    if (!act && !pad) continue;
    const float mul = norm != nullptr ? 1.0f / sqrtf(ss / (float)a.dk + a.eps) : 1.0f;
    const size_t row = (size_t)(m.row0 + q);
    TA* dst;
    if (is_q) {
      dst = reinterpret_cast<TA*>(a.q_out) + (row * a.H + hs) * a.wk;
    } else {
      const int slot = a.slots[row];
      if (slot < 0) continue;
      const int g = is_k ? hs - a.H : hs - a.H - a.G;
      dst = reinterpret_cast<TA*>(is_k ? a.k_cache : a.v_cache) + (((size_t)(slot / a.page) * a.G + g) * a.page + (slot % a.page)) * wide;
    }
    uint4 outv;
    TA* ov = reinterpret_cast<TA*>(&outv);
#pragma unroll
    for (int i = 0; i < V; ++i) ca_store(ov + i, act ? (norm != nullptr ? y[i] * mul * nw[i] : y[i]) : 0.f);
    *reinterpret_cast<uint4*>(dst + d) = outv;
  }
}

// Any width, any number of taps: a warp owns a head slot, the lanes its columns in turn, and reads every tap's input anew.
template <typename TA>
__global__ void __launch_bounds__(kCapWarps * 32)
conv_attn_prep_kernel(CapArgs a) {
  constexpr int kPer = 16;                             // columns per lane: widths up to 512
  const CapWork m = cap_work(a);
  const int hs = blockIdx.y * kCapWarps + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (m.n <= 0 || hs >= a.H + 2 * a.G) return;
  const bool is_q = hs < a.H, is_k = !is_q && hs < a.H + a.G;
  const int width = (is_q || is_k) ? a.dk : a.dv, wide = (is_q || is_k) ? a.wk : a.wv;
  const int col0 = (is_q || is_k) ? hs * a.dk : (a.H + a.G) * a.dk + (hs - a.H - a.G) * a.dv;
  const int C = (a.H + a.G) * a.dk + a.G * a.dv, R = a.taps - 1;
  const TA* src = reinterpret_cast<const TA*>(a.proj) + (size_t)m.row0 * a.ld + col0;
  const bf16* norm = is_q ? a.qnorm_w : (is_k ? a.knorm_w : nullptr);
  for (int i_row = 0; i_row < m.n; ++i_row) {
    const int q = m.q0 + i_row;
    float y[kPer], ss = 0.f;
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
      const int d = lane + 32 * i;
      y[i] = 0.f;
      if (d < width) {
        const float* w = a.conv_w + (size_t)(col0 + d) * a.taps;
        float v = 0.f;
        for (int b = 0; b <= R; ++b) {
          const int qq = q - b, p = m.ctx + qq;
          float x = 0.f;
          if (qq >= 0) x = ca_f32(src[(size_t)qq * a.ld + d]);
          else if (p >= 0 && m.slot >= 0) x = a.ring[((size_t)m.slot * R + p % R) * C + col0 + d];
          v = fmaf(w[R - b], x, v);
        }
        y[i] = v;
        ss = fmaf(v, v, ss);
      }
    }
    ss = warp_sum(ss);
    const float mul = norm != nullptr ? 1.0f / sqrtf(ss / (float)a.dk + a.eps) : 1.0f;
    const size_t row = (size_t)(m.row0 + q);
    TA* dst;
    if (is_q) {
      dst = reinterpret_cast<TA*>(a.q_out) + (row * a.H + hs) * a.wk;
    } else {
      const int slot = a.slots[row];
      if (slot < 0) continue;
      const int g = is_k ? hs - a.H : hs - a.H - a.G;
      dst = reinterpret_cast<TA*>(is_k ? a.k_cache : a.v_cache) + (((size_t)(slot / a.page) * a.G + g) * a.page + (slot % a.page)) * wide;
    }
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
      const int d = lane + 32 * i;
      if (d < width) ca_store(dst + d, norm != nullptr ? y[i] * mul * __bfloat162float(norm[d]) : y[i]);
      else if (d < wide) ca_store(dst + d, 0.f);
    }
  }
  if (R > 0 && m.q0 == 0 && m.slot >= 0) {             // every read of the ring by this warp's columns lies behind it
    for (int b = 0; b < R; ++b) {
      const int q = m.qlen - 1 - b;
      if (q < 0) break;
      float* rp = a.ring + ((size_t)m.slot * R + (m.ctx + q) % R) * C + col0;
      for (int d = lane; d < width; d += 32) rp[d] = ca_f32(src[(size_t)q * a.ld + d]);
    }
  }
}

}  // namespace b200

using namespace b200;

extern "C" int b200_conv_attn_prep(const void* proj, int f32, int64_t ld, const float* conv_w, int taps, const void* qnorm_w,
                                   const void* knorm_w, float* ring, const int32_t* cu_seq, const int32_t* ctx_lens,
                                   const int32_t* state_slots, const int32_t* tile_seq, const int32_t* tile_q0, int n_tiles,
                                   int tile_rows, int n_prompt, int n_single, const int32_t* slots, void* q_out,
                                   void* k_cache, void* v_cache, int H, int G, int dk, int dv, int wk, int wv, int page,
                                   float eps, void* stream) {
  B200_REQUIRE(H > 0 && G > 0 && H % G == 0 && dk > 0 && dv > 0 && wk >= dk && wv >= dv && page > 0,
               "conv_attn_prep: bad shape H=%d G=%d dk=%d dv=%d in %d / %d", H, G, dk, dv, wk, wv);
  B200_REQUIRE(taps >= 1 && taps <= kCapMaxTaps, "conv_attn_prep: %d taps (1 .. %d)", taps, kCapMaxTaps);
  B200_REQUIRE(taps == 1 || (ring != nullptr && state_slots != nullptr), "conv_attn_prep: more than one tap needs the sequences' rings");
  B200_REQUIRE(n_tiles == 0 || (tile_rows > 0 && tile_rows % kCapRows == 0), "conv_attn_prep: tiles of %d rows (multiples of %d)",
               tile_rows, kCapRows);
  B200_REQUIRE(n_tiles >= 0 && n_prompt >= 0 && n_single >= 0, "conv_attn_prep: bad counts");
  const int per_tile = n_tiles > 0 ? tile_rows / kCapRows : 1;
  const int n_x = n_tiles * per_tile + n_single;
  if (n_x == 0) return B200_OK;
  const CapArgs a{proj, ld, conv_w, (const bf16*)qnorm_w, (const bf16*)knorm_w, taps > 1 ? ring : nullptr, cu_seq, ctx_lens,
                  state_slots, tile_seq, tile_q0, n_tiles * per_tile, per_tile, n_prompt, slots, q_out, k_cache, v_cache, H, G,
                  dk, dv, wk, wv, page, taps, eps};
  cudaStream_t s = (cudaStream_t)stream;
  const int n_heads = H + 2 * G, esz = f32 ? 4 : 2, vec = 16 / esz, wmax = wk > wv ? wk : wv;
  const bool al = ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(q_out) | reinterpret_cast<uintptr_t>(k_cache) |
                    reinterpret_cast<uintptr_t>(v_cache)) & 15) == 0;
  if (al && taps <= 4 && dk % vec == 0 && dv % vec == 0 && wk % vec == 0 && wv % vec == 0 && ld % vec == 0 && wmax / vec <= 32) {
    int lph = 1;
    while (lph < wmax / vec) lph <<= 1;
    const int per_block = kCapWarps * (32 / lph);
    const dim3 grid(n_x, (n_heads + per_block - 1) / per_block);
#define B200_CAP(TA, N) conv_attn_prep_vec_kernel<TA, N><<<grid, kCapWarps * 32, 0, s>>>(a, lph)
#define B200_CAPT(TA)                        \
  switch (taps) {                            \
    case 1: B200_CAP(TA, 1); break;          \
    case 2: B200_CAP(TA, 2); break;          \
    case 3: B200_CAP(TA, 3); break;          \
    default: B200_CAP(TA, 4);                \
  }
    if (f32) { B200_CAPT(float) } else { B200_CAPT(bf16) }
#undef B200_CAPT
#undef B200_CAP
    return b200_check_launch("b200_conv_attn_prep");
  }
  B200_REQUIRE(wmax <= 512, "conv_attn_prep: head width %d exceeds 512", wmax);
  const dim3 grid(n_x, (n_heads + kCapWarps - 1) / kCapWarps);
  if (f32) conv_attn_prep_kernel<float><<<grid, kCapWarps * 32, 0, s>>>(a);
  else conv_attn_prep_kernel<bf16><<<grid, kCapWarps * 32, 0, s>>>(a);
  return b200_check_launch("b200_conv_attn_prep");
}
