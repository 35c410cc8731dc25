// What the preparation kernels behind a fused projection share: element conversions and the cut of a step's rows into
// pieces of one sequence.  A step lists its sequences as prompt portions (covered by row tiles) followed by single rows; a
// piece is ROWS consecutive rows of a portion, or one single row.
#pragma once
#include "common.cuh"

namespace b200 {

constexpr int kCapRows = 8;        // rows of one sequence per CTA
constexpr int kCapMaxTaps = 8;
constexpr int kCapWarps = 8;

__device__ __forceinline__ float ca_f32(float v) { return v; }
__device__ __forceinline__ float ca_f32(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void ca_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void ca_store(bf16* p, float v) { *p = __float2bfloat16_rn(v); }

// What a CTA works on: rows [row0 + q0, + n) of the projection at positions ctx + q0 ..., of a sequence with qlen new rows
struct CapWork {
  int row0, q0, n, qlen, ctx, slot;
};
template <int ROWS, typename Args>
__device__ __forceinline__ CapWork cap_work(const Args& a) {
  CapWork m;
  int s, q0 = 0;
  if ((int)blockIdx.x < a.n_pieces) {
    const int tile = blockIdx.x / a.per_tile;
    s = a.tile_seq[tile];
    q0 = a.tile_q0[tile] + ROWS * (blockIdx.x - tile * a.per_tile);
  } else {
    s = a.n_prompt + (int)blockIdx.x - a.n_pieces;
  }
  m.row0 = a.cu_seq[s];
  m.q0 = q0;
  m.qlen = a.cu_seq[s + 1] - m.row0;
  m.n = min(ROWS, m.qlen - q0);
  m.ctx = a.ctx_lens[s];
  m.slot = a.ring != nullptr ? a.state_slots[s] : -1;
  return m;
}

// One 16-byte piece (V channels from channel c on) of a work item's rows and of the TAPS - 1 rows before them, as loaded:
// win[R + i] is row q0 + i, win[R - 1 - b] the input b + 1 positions before row q0 -- from this step's rows, else from the
// sequence's ring (a ring entry is an input, so it fits the element type exactly), else zero.  src: row 0 of the sequence.
template <typename TA, int TAPS, int NB>
__device__ __forceinline__ void conv_window(uint4 (&win)[TAPS - 1 + NB], const CapWork& m, const TA* src, int64_t ld,
                                            const float* ring, int c, int C) {
  constexpr int V = 16 / (int)sizeof(TA), R = TAPS - 1, RR = R > 0 ? R : 1;
  static_assert(R <= NB, "a sequence's first piece holds every row that reads the ring");
  const uint4 zero4 = make_uint4(0, 0, 0, 0);
#pragma unroll
  for (int i = 0; i < NB; ++i)
    win[R + i] = i < m.n ? *reinterpret_cast<const uint4*>(src + (int64_t)(m.q0 + i) * ld) : zero4;
  if constexpr (R > 0)
#pragma unroll
  for (int b = 0; b < R; ++b) {
    const int q = m.q0 - 1 - b, p = m.ctx + q;
    win[R - 1 - b] = zero4;
    if (q >= 0) {
      win[R - 1 - b] = *reinterpret_cast<const uint4*>(src + (int64_t)q * ld);
    } else if (p >= 0 && m.slot >= 0) {
      const float* rp = ring + ((size_t)m.slot * R + p % RR) * C + c;
      TA* w = reinterpret_cast<TA*>(&win[R - 1 - b]);
#pragma unroll
      for (int i = 0; i < V; ++i) ca_store(w + i, rp[i]);
    }
  }
}

// The step's last inputs of the piece's channels go to the ring: called by the threads of a sequence's FIRST piece after
// their reads of it (no other piece reads it).
template <typename TA, int TAPS>
__device__ __forceinline__ void conv_ring_put(const CapWork& m, const TA* src, int64_t ld, float* ring, int c, int C) {
  constexpr int V = 16 / (int)sizeof(TA), R = TAPS - 1, RR = R > 0 ? R : 1;
  if (R == 0 || m.q0 != 0 || m.slot < 0) return;
  if constexpr (R > 0)
#pragma unroll
  for (int b = 0; b < R; ++b) {
    const int q = m.qlen - 1 - b;
    if (q < 0) break;
    const uint4 raw = *reinterpret_cast<const uint4*>(src + (int64_t)q * ld);
    const TA* x = reinterpret_cast<const TA*>(&raw);
    float* rp = ring + ((size_t)m.slot * R + (m.ctx + q) % RR) * C + c;
#pragma unroll
    for (int i = 0; i < V; i += 4)
      *reinterpret_cast<float4*>(rp + i) = make_float4(ca_f32(x[i]), ca_f32(x[i + 1]), ca_f32(x[i + 2]), ca_f32(x[i + 3]));
  }
}

// Row i of a window, convolved: w[b] are the weights of the inputs b positions back
template <typename TA, int TAPS, int NB>
__device__ __forceinline__ void conv_row(const uint4 (&win)[TAPS - 1 + NB], int i, const float (&w)[TAPS][16 / (int)sizeof(TA)],
                                         float (&y)[16 / (int)sizeof(TA)]) {
  constexpr int V = 16 / (int)sizeof(TA);
#pragma unroll
  for (int b = 0; b < TAPS; ++b) {
    const TA* x = reinterpret_cast<const TA*>(&win[TAPS - 1 + i - b]);
#pragma unroll
    for (int e = 0; e < V; ++e) y[e] = fmaf(w[b][e], ca_f32(x[e]), y[e]);
  }
}

// The weights of V channels from channel c on: conv_w is [TAPS][C], its last row multiplies the current token
template <int TAPS, int V>
__device__ __forceinline__ void conv_weights(float (&w)[TAPS][V], const float* conv_w, int c, int C) {
#pragma unroll
  for (int b = 0; b < TAPS; ++b)
#pragma unroll
    for (int i = 0; i < V; i += 4)
      *reinterpret_cast<float4*>(&w[b][i]) = *reinterpret_cast<const float4*>(conv_w + (size_t)(TAPS - 1 - b) * C + c + i);
}

// One channel of one row by plain loads (any width, any number of taps): src points at the channel in row 0 of the sequence
template <typename TA>
__device__ __forceinline__ float conv_at(const CapWork& m, int q, const TA* src, int64_t ld, const float* ring, const float* w, int c,
                                         int C, int taps) {
  const int R = taps - 1;
  float v = 0.f;
  for (int b = 0; b <= R; ++b) {
    const int qq = q - b, p = m.ctx + qq;
    float x = 0.f;
    if (qq >= 0) x = ca_f32(src[(int64_t)qq * ld]);
    else if (p >= 0 && m.slot >= 0) x = ring[((size_t)m.slot * R + p % R) * C + c];
    v = fmaf(w[(size_t)(R - b) * C + c], x, v);
  }
  return v;
}

}  // namespace b200
