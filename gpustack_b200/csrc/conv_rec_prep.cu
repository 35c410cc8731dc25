// Preparation of a recurrent mixer whose inputs pass a short causal convolution over time, in ONE launch: from projected
// rows to fp32 rows of the recurrence's inputs.
//
//   y_t = bias + sum_j w[:, j] u_(t - taps + 1 + j)      per channel, zeros before the sequence's start; inputs older than the
//                                                        step come from the sequence's ring
//   y <- silu(y);  optionally per head  y / sqrt(sum(y^2) + eps) * factor
//   rows [segment 0 | segment 1 | segment 2] with every head padded by zeros to a multiple of 4 entries;
//   the step's last taps - 1 inputs of every sequence replace the ring's entries: ring[slot][p mod (taps - 1)][channel].
//
// The channels are up to three segments of equal heads (queries, keys, values of a delta rule; inputs and the two projections
// of a state-space mixer).  The cut into pieces and the ring's protocol are those of the attention preparation
// (conv_prep.cuh); everything behind the loads is fp32.
#include "common.cuh"
#include "conv_prep.cuh"
#include "runtime.h"
#include "../../include/b200.h"

namespace b200 {

struct CrpSegment {
  int heads, width, unit;
  float mul;
};

struct CrpArgs {
  const void* proj;                // column 0 = the first convolved channel
  int64_t ld;
  const float* conv_w;             // [taps][C]
  const float* bias;               // [C] or null
  float* ring;
  const int32_t* cu_seq;
  const int32_t* ctx_lens;
  const int32_t* state_slots;
  const int32_t* tile_seq;
  const int32_t* tile_q0;
  int n_pieces, per_tile, n_prompt;
  CrpSegment seg[3];
  float* out;
  int64_t ldo;
  int C, taps, n_heads;
  float eps;
};

// head slot -> segment, first channel, first output column
struct CrpHead {
  int seg, c, o, width;
};
__device__ __forceinline__ CrpHead crp_head(const CrpArgs& a, int hs) {
  CrpHead h{0, 0, 0, a.seg[0].width};
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    if (h.seg == i && hs >= a.seg[i].heads) {
      hs -= a.seg[i].heads;
      h.c += a.seg[i].heads * a.seg[i].width;
      h.o += a.seg[i].heads * ((a.seg[i].width + 3) & ~3);
      h.seg = i + 1;
      h.width = a.seg[i + 1].width;
    }
  }
  h.c += hs * h.width;
  h.o += hs * ((h.width + 3) & ~3);
  return h;
}

__device__ __forceinline__ float crp_silu(float y) { return y / (1.0f + expf(-y)); }

// LPH lanes share a head, each owns one 16-byte piece of it in NB rows.
template <typename TA, int TAPS, int NB>
__global__ void __launch_bounds__(kCapWarps * 32)
conv_rec_prep_vec_kernel(CrpArgs a, int lph) {
  constexpr int V = 16 / (int)sizeof(TA), R = TAPS - 1;
  const CapWork m = cap_work<NB>(a);
  if (m.n <= 0) return;
  const int lane = threadIdx.x & 31, per_warp = 32 / lph;
  const int hs = (blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5)) * per_warp + lane / lph;
  const bool live = hs < a.n_heads;
  const CrpHead h = crp_head(a, live ? hs : 0);
  const CrpSegment sg = a.seg[h.seg];
  const int d = (lane % lph) * V;
  const bool act = live && d < h.width;
  const int c = h.c + d;
  const TA* src = reinterpret_cast<const TA*>(a.proj) + (size_t)m.row0 * a.ld + c;
  uint4 win[R + NB];
  float w[TAPS][V], bias[V];
  if (act) {
    conv_window<TA, TAPS, NB>(win, m, src, a.ld, a.ring, c, a.C);
    conv_weights<TAPS, V>(w, a.conv_w, c, a.C);
#pragma unroll
    for (int i = 0; i < V; ++i) bias[i] = a.bias != nullptr ? a.bias[c + i] : 0.f;
    conv_ring_put<TA, TAPS>(m, src, a.ld, a.ring, c, a.C);
  }
  float* dst = a.out + (size_t)(m.row0 + m.q0) * a.ldo + h.o + d;
#pragma unroll
  for (int r = 0; r < NB; ++r) {
    if (r >= m.n) break;
    float y[V], ss = 0.f;
#pragma unroll
    for (int i = 0; i < V; ++i) y[i] = 0.f;
    if (act) {
#pragma unroll
      for (int i = 0; i < V; ++i) y[i] = bias[i];
      conv_row<TA, TAPS, NB>(win, r, w, y);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        y[i] = crp_silu(y[i]);
        ss = fmaf(y[i], y[i], ss);
      }
    }
    for (int o = lph >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);    // all lanes take part
    if (!act) continue;
    const float mul = sg.unit ? sg.mul / sqrtf(ss + a.eps) : sg.mul;
#pragma unroll
    for (int i = 0; i < V; i += 4)
      *reinterpret_cast<float4*>(dst + (size_t)r * a.ldo + i) = make_float4(y[i] * mul, y[i + 1] * mul, y[i + 2] * mul, y[i + 3] * mul);
  }
}

// Any width, any number of taps: a warp owns a head slot, the lanes its columns in turn, and reads every tap's input anew.
template <typename TA>
__global__ void __launch_bounds__(kCapWarps * 32)
conv_rec_prep_kernel(CrpArgs a) {
  constexpr int kPer = 16;                             // columns per lane: widths up to 512
  const CapWork m = cap_work<kCapRows>(a);
  const int hs = blockIdx.y * kCapWarps + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (m.n <= 0 || hs >= a.n_heads) return;
  const CrpHead h = crp_head(a, hs);
  const CrpSegment sg = a.seg[h.seg];
  const int R = a.taps - 1, wide = (h.width + 3) & ~3;
  const TA* src = reinterpret_cast<const TA*>(a.proj) + (size_t)m.row0 * a.ld + h.c;
  for (int i_row = 0; i_row < m.n; ++i_row) {
    float y[kPer], ss = 0.f;
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
      const int d = lane + 32 * i;
      y[i] = 0.f;
      if (d < h.width) {
        const float v = conv_at<TA>(m, m.q0 + i_row, src + d, a.ld, a.ring, a.conv_w, h.c + d, a.C, a.taps) +
                        (a.bias != nullptr ? a.bias[h.c + d] : 0.f);
        y[i] = crp_silu(v);
        ss = fmaf(y[i], y[i], ss);
      }
    }
    ss = warp_sum(ss);
    const float mul = sg.unit ? sg.mul / sqrtf(ss + a.eps) : sg.mul;
    float* dst = a.out + (size_t)(m.row0 + m.q0 + i_row) * a.ldo + h.o;
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
      const int d = lane + 32 * i;
      if (d < wide) dst[d] = y[i] * mul;               // zeros behind the head's own columns
    }
  }
  if (R > 0 && m.q0 == 0 && m.slot >= 0) {             // every read of the ring by this warp's columns lies behind it
    for (int b = 0; b < R; ++b) {
      const int q = m.qlen - 1 - b;
      if (q < 0) break;
      float* rp = a.ring + ((size_t)m.slot * R + (m.ctx + q) % R) * a.C + h.c;
      for (int d = lane; d < h.width; d += 32) rp[d] = ca_f32(src[(size_t)q * a.ld + d]);
    }
  }
}

}  // namespace b200

using namespace b200;

extern "C" int b200_conv_rec_prep(const void* proj, int f32, int64_t ld, const float* conv_w, int taps, const float* bias,
                                  float* ring, const int32_t* cu_seq, const int32_t* ctx_lens, const int32_t* state_slots,
                                  const int32_t* tile_seq, const int32_t* tile_q0, int n_tiles, int tile_rows, int n_prompt,
                                  int n_single, const int32_t* seg_heads, const int32_t* seg_width, const int32_t* seg_unit,
                                  const float* seg_mul, float* out, int64_t ldo, float eps, void* stream) {
  B200_REQUIRE(taps >= 1 && taps <= kCapMaxTaps, "conv_rec_prep: %d taps (1 .. %d)", taps, kCapMaxTaps);
  B200_REQUIRE(taps == 1 || (ring != nullptr && state_slots != nullptr), "conv_rec_prep: more than one tap needs the sequences' rings");
  B200_REQUIRE(n_tiles == 0 || (tile_rows > 0 && tile_rows % kCapRows == 0), "conv_rec_prep: tiles of %d rows (multiples of %d)",
               tile_rows, kCapRows);
  B200_REQUIRE(n_tiles >= 0 && n_prompt >= 0 && n_single >= 0, "conv_rec_prep: bad counts");
  CrpArgs a{proj, ld, conv_w, bias, taps > 1 ? ring : nullptr, cu_seq, ctx_lens, state_slots, tile_seq, tile_q0, 0, 1, n_prompt, {}, out, ldo,
            0, taps, 0, eps};
  int wmax = 0, n_out = 0;
  bool unit = false;
  const int esz = f32 ? 4 : 2, vec = 16 / esz;
  bool whole = true;                                   // every head in whole 16-byte pieces
  for (int i = 0; i < 3; ++i) {
    a.seg[i] = CrpSegment{seg_heads[i], seg_width[i], seg_unit[i], seg_mul[i]};
    B200_REQUIRE(seg_heads[i] >= 0 && seg_width[i] > 0 && seg_width[i] <= 512, "conv_rec_prep: segment %d: %d heads of width %d (1 .. 512)", i,
                 seg_heads[i], seg_width[i]);
    a.C += seg_heads[i] * seg_width[i];
    n_out += seg_heads[i] * ((seg_width[i] + 3) & ~3);
    a.n_heads += seg_heads[i];
    unit = unit || seg_unit[i] != 0;
    whole = whole && seg_width[i] % vec == 0;
    wmax = seg_width[i] > wmax ? seg_width[i] : wmax;
  }
  B200_REQUIRE(a.n_heads > 0 && ld >= a.C && ldo >= n_out, "conv_rec_prep: rows of %d channels -> %d columns", a.C, n_out);
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool fast = whole && al(proj) && al(conv_w) && al(out) && al(a.ring) && taps <= 4 && ld % vec == 0 && ldo % 4 == 0 && a.C % 4 == 0 &&
                    (!unit || wmax / vec <= 32);
  const int rows = fast ? 4 : kCapRows;
  a.per_tile = n_tiles > 0 ? tile_rows / rows : 1;
  a.n_pieces = n_tiles * a.per_tile;
  const int n_x = a.n_pieces + n_single;
  if (n_x == 0) return B200_OK;
  cudaStream_t s = (cudaStream_t)stream;
  if (fast) {
    if (!unit && a.seg[0].mul == 1.f && a.seg[1].mul == 1.f && a.seg[2].mul == 1.f) {    // no statistic: the heads do not matter
      a.seg[0] = CrpSegment{a.C / vec, vec, 0, 1.f};
      a.seg[1].heads = a.seg[2].heads = 0;
      a.n_heads = a.C / vec;
      wmax = vec;
    }
    int lph = 1;
    while (lph < wmax / vec) lph <<= 1;
    const int all_warps = (a.n_heads + 32 / lph - 1) / (32 / lph), ny = (all_warps + kCapWarps - 1) / kCapWarps;
    const int warps = (all_warps + ny - 1) / ny;
    const dim3 grid(n_x, ny);
#define B200_CRP(TA, N) conv_rec_prep_vec_kernel<TA, N, 4><<<grid, warps * 32, 0, s>>>(a, lph)
#define B200_CRPT(TA)                        \
  switch (taps) {                            \
    case 1: B200_CRP(TA, 1); break;          \
    case 2: B200_CRP(TA, 2); break;          \
    case 3: B200_CRP(TA, 3); break;          \
    default: B200_CRP(TA, 4);                \
  }
    if (f32) { B200_CRPT(float) } else { B200_CRPT(bf16) }
#undef B200_CRPT
#undef B200_CRP
    return b200_check_launch("b200_conv_rec_prep");
  }
  const dim3 grid(n_x, (a.n_heads + kCapWarps - 1) / kCapWarps);
  if (f32) conv_rec_prep_kernel<float><<<grid, kCapWarps * 32, 0, s>>>(a);
  else conv_rec_prep_kernel<bf16><<<grid, kCapWarps * 32, 0, s>>>(a);
  return b200_check_launch("b200_conv_rec_prep");
}
