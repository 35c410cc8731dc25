// Preparation of a softmax-attention mixer whose q, k and v pass a short causal convolution over time, in ONE launch:
// from the projected rows u = [q: H dk | k: G dk | v: G dv] of a step to attention-ready queries and cache pages.
//
//   y_t = sum_j w[:, j] u_(t - taps + 1 + j)         per channel, zeros before the sequence's start, no bias; inputs
//                                                    older than the step come from the sequence's ring
//   q, k:  y / sqrt(mean(y^2) + eps) * weight        per head over dk, one weight vector for all heads (optional), or over
//                                                    the whole projection (all heads at once) with weights of that size
//   q, k:  rotation of the first `dims` entries by the rows' angles (optional, after the norm); cos and sin come from a table
//          that rot_table fills once per step for all layers with the same frequencies
//   q to its row of q_out, k and v to their pages (slot of the token), heads laid out wk / wv wide (>= dk / dv, the
//   columns behind dk / dv are zeros: a pair of widths that is no tensor-core tile is padded to one);
//   the step's last taps - 1 inputs of every sequence replace the ring's entries: ring[slot][p mod (taps - 1)][channel].
//
// A CTA takes 8 consecutive rows of one sequence and some head slots; the threads that own a channel issue all their loads
// (8 rows and the taps - 1 before them) at once and walk the rows in registers.  Only a sequence's first
// piece can need the ring (a piece is longer than the ring), and the SAME threads that read it there write the step's
// last inputs into it after their reads: no second launch, no race.  The statistics and the convolution are fp32.
#include "common.cuh"
#include "conv_prep.cuh"
#include "runtime.h"
#include "../../include/b200.h"

namespace b200 {

struct CapArgs {
  const void* proj;
  int64_t ld;
  const float* conv_w;             // [taps][C], last row = current token
  const bf16* qnorm_w;             // null: no norm
  const bf16* knorm_w;
  float* ring;                     // [slots][taps - 1][C]; null when taps == 1
  const int32_t* cu_seq;           // every sequence of the step: prompt portions, then single rows
  const int32_t* ctx_lens;
  const int32_t* state_slots;
  const int32_t* tile_seq;         // row tiles of the prompt portions
  const int32_t* tile_q0;
  int n_pieces;                    // tiles * (tile_rows / 8): CTAs [0, n_pieces) along x; then one per single row
  int per_tile;                    // tile_rows / 8
  int n_prompt;                    // sequences with a prompt portion
  const int32_t* slots;            // cache slot of every row (-1: no write)
  void* q_out;
  void* k_cache;
  void* v_cache;
  int H, G, dk, dv, wk, wv, page, page_shift, taps;    // page_shift: log2(page), or -1
  float eps;
  int joint;                       // the norm runs over the whole projection (weights of H dk / G dk entries)
  int dims, half_layout;           // rotation of the first `dims` entries of a q / k head, pairs (i, i + dims/2) or (2i, 2i + 1)
  const float2* cs;                // [rows][dims / 2] (cos, sin)
};

// the (page, head) row of a cache slot, in rows of the cache
__device__ __forceinline__ size_t cap_cache_row(const CapArgs& a, int slot, int g) {
  const int pg = a.page_shift >= 0 ? slot >> a.page_shift : slot / a.page;
  return ((size_t)pg * a.G + g) * a.page + (slot - pg * a.page);
}

// LPH lanes share a head, each owns one 16-byte piece of it.
template <typename TA, int TAPS>
__global__ void __launch_bounds__(kCapWarps * 32, 2)
conv_attn_prep_vec_kernel(CapArgs a, int lph) {
  constexpr int V = 16 / (int)sizeof(TA), R = TAPS - 1, NB = kCapRows;
  static_assert(R <= NB, "a sequence's first piece holds every row that reads the ring");
  const CapWork m = cap_work<kCapRows>(a);
  if (m.n <= 0) return;
  const int lane = threadIdx.x & 31, per_warp = 32 / lph;
  const int hs = (blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5)) * per_warp + lane / lph;
  const bool live = hs < a.H + 2 * a.G;
  const bool is_q = hs < a.H, is_k = !is_q && hs < a.H + a.G;
  const int width = (is_q || is_k) ? a.dk : a.dv, wide = (is_q || is_k) ? a.wk : a.wv;
  const int col0 = (is_q || is_k) ? hs * a.dk : (a.H + a.G) * a.dk + (hs - a.H - a.G) * a.dv;
  const int d = (lane % lph) * V;
  const bool act = live && d < width, pad = live && !act && d < wide;
  const int c = col0 + d, C = (a.H + a.G) * a.dk + a.G * a.dv;
  const TA* src = reinterpret_cast<const TA*>(a.proj) + (size_t)m.row0 * a.ld + c;
  const uint4 zero4 = make_uint4(0, 0, 0, 0);
  auto load = [&](int q) { return *reinterpret_cast<const uint4*>(src + (int64_t)q * a.ld); };
  // win[R + i]: row i of the piece as loaded; win[R - 1 - b]: the input b + 1 positions before it (a ring entry is an
  // input, so it fits the element type exactly)
  uint4 win[R + NB];
#pragma unroll
  for (int i = 0; i < NB; ++i) win[R + i] = (act && i < m.n) ? load(m.q0 + i) : zero4;
#pragma unroll
  for (int b = 0; b < R; ++b) win[b] = zero4;
  const bf16* norm = is_q ? a.qnorm_w : (is_k ? a.knorm_w : nullptr);
  float w[TAPS][V], nw[V];         // w[b]: weight of the input b positions back
  if (act) {
#pragma unroll
    for (int b = 0; b < R; ++b) {
      const int q = m.q0 - 1 - b, p = m.ctx + q;
      if (q >= 0) {
        win[R - 1 - b] = load(q);
      } else if (p >= 0 && m.slot >= 0) {
        const float* rp = a.ring + ((size_t)m.slot * R + p % (R > 0 ? R : 1)) * C + c;
        TA* wv = reinterpret_cast<TA*>(&win[R - 1 - b]);
#pragma unroll
        for (int i = 0; i < V; ++i) ca_store(wv + i, rp[i]);
      }
    }
#pragma unroll
    for (int b = 0; b < TAPS; ++b)
#pragma unroll
      for (int i = 0; i < V; i += 4)
        *reinterpret_cast<float4*>(&w[b][i]) = *reinterpret_cast<const float4*>(a.conv_w + (size_t)(R - b) * C + c + i);
#pragma unroll
    for (int i = 0; i < V; ++i) nw[i] = norm != nullptr ? __bfloat162float(norm[d + i]) : 1.0f;
    if (R > 0 && m.q0 == 0 && m.slot >= 0) {           // the ring has been read by its only readers: this step's last inputs
#pragma unroll
      for (int b = 0; b < R; ++b) {
        const int q = m.qlen - 1 - b;
        if (q < 0) break;
        const uint4 raw = load(q);
        const TA* x = reinterpret_cast<const TA*>(&raw);
        float* rp = a.ring + ((size_t)m.slot * R + (m.ctx + q) % (R > 0 ? R : 1)) * C + c;
#pragma unroll
        for (int i = 0; i < V; i += 4)
          *reinterpret_cast<float4*>(rp + i) = make_float4(ca_f32(x[i]), ca_f32(x[i + 1]), ca_f32(x[i + 2]), ca_f32(x[i + 3]));
      }
    }
  }
  const float inv_dk = 1.0f / (float)a.dk;
  const int g = is_k ? hs - a.H : hs - a.H - a.G;
  TA* const q_dst = reinterpret_cast<TA*>(a.q_out) + ((size_t)(m.row0 + m.q0) * a.H + hs) * a.wk + d;
  TA* const kv_dst = reinterpret_cast<TA*>(is_k ? a.k_cache : a.v_cache) + d;
  const int32_t* slots = a.slots + m.row0 + m.q0;
#pragma unroll
  for (int r = 0; r < NB; ++r) {
    if (r >= m.n) break;
    float y[V], ss = 0.f;
#pragma unroll
    for (int i = 0; i < V; ++i) y[i] = 0.f;
    if (act) {
#pragma unroll
      for (int b = 0; b < TAPS; ++b) {
        const TA* x = reinterpret_cast<const TA*>(&win[R + r - b]);
#pragma unroll
        for (int i = 0; i < V; ++i) y[i] = fmaf(w[b][i], ca_f32(x[i]), y[i]);
      }
#pragma unroll
      for (int i = 0; i < V; ++i) ss = fmaf(y[i], y[i], ss);
    }
    for (int o = lph >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);    // all lanes take part
    if (!act && !pad) continue;
    uint4 outv = zero4;
    if (act) {
      const float mul = norm != nullptr ? rsqrtf(fmaf(ss, inv_dk, a.eps)) : 1.0f;
      TA* ov = reinterpret_cast<TA*>(&outv);
#pragma unroll
      for (int i = 0; i < V; ++i) ca_store(ov + i, y[i] * mul * nw[i]);
    }
    if (is_q) {
      *reinterpret_cast<uint4*>(q_dst + (size_t)r * a.H * a.wk) = outv;
    } else {
      const int slot = slots[r];
      if (slot >= 0) *reinterpret_cast<uint4*>(kv_dst + cap_cache_row(a, slot, g) * wide) = outv;
    }
  }
}

// Any width, any number of taps: a warp owns a head slot, the lanes its columns in turn, and reads every tap's input anew.
template <typename TA>
__global__ void __launch_bounds__(kCapWarps * 32)
conv_attn_prep_kernel(CapArgs a) {
  constexpr int kPer = 16;                             // columns per lane: widths up to 512
  const CapWork m = cap_work<kCapRows>(a);
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
        const float* w = a.conv_w + col0 + d;
        float v = 0.f;
        for (int b = 0; b <= R; ++b) {
          const int qq = q - b, p = m.ctx + qq;
          float x = 0.f;
          if (qq >= 0) x = ca_f32(src[(size_t)qq * a.ld + d]);
          else if (p >= 0 && m.slot >= 0) x = a.ring[((size_t)m.slot * R + p % R) * C + col0 + d];
          v = fmaf(w[(size_t)(R - b) * C], x, v);
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
      dst = reinterpret_cast<TA*>(is_k ? a.k_cache : a.v_cache) + cap_cache_row(a, slot, g) * wide;
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

// (cos, sin) of position * freq[i] for every row of a step: the angle is formed and reduced to [-pi, pi] in fp64, sine and
// cosine of the remainder in fp32
__global__ void __launch_bounds__(256)
rot_table_kernel(const int32_t* __restrict__ positions, const double* __restrict__ freq, float2* __restrict__ out, int half, int n) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const int r = i / half, j = i - r * half;
  const double ang = (double)positions[r] * freq[j];
  float sn, c;
  sincosf((float)(ang - 6.283185307179586 * rint(ang * 0.15915494309189535)), &sn, &c);
  out[i] = make_float2(c, sn);
}

// The form with a rotation and / or a norm over the whole projection.  ONE CTA owns all channels of a run of rows (the joint
// statistic is a sum over the CTA) and walks it two rows at a time; a thread owns one 16-byte piece of a head for the whole
// run, its weights in registers, its inputs in a private ring of eight rows in shared memory that cp.async fills two steps
// ahead.  Per step: convolve, sum the squares over the head's lanes, one barrier, sum over the heads (the same order in every
// warp), scale, rotate -- the partner of an entry sits dims / 2 further, in another lane of the head's group, or beside it --
// and store.
constexpr int kCapRun = 16, kCapJointWarps = 24, kCapSlots = 8;

template <typename TA, int TAPS>
__global__ void __launch_bounds__(kCapJointWarps * 32, 1)
conv_attn_prep_joint_vec_kernel(CapArgs a, int lph) {
  constexpr int V = 16 / (int)sizeof(TA), R = TAPS - 1, RR = R > 0 ? R : 1;
  static_assert(R + 2 + 3 <= kCapSlots, "a step's rows, the ones before and the ones in flight have slots of their own");
  extern __shared__ __align__(16) uint4 raw[];         // [8][threads]
  __shared__ float head_ss[2][2][kCapJointWarps * 32]; // [step parity][row][head slot]
  const CapWork m = cap_work<kCapRun>(a);
  if (m.n <= 0) return;
  const int lane = threadIdx.x & 31, per_warp = 32 / lph, li = lane % lph, d = li * V, half = a.dims >> 1;
  const int hs = (threadIdx.x >> 5) * per_warp + lane / lph;
  const bool live = hs < a.H + 2 * a.G, is_q = hs < a.H, is_k = !is_q && hs < a.H + a.G, qk = is_q || is_k;
  const int width = qk ? a.dk : a.dv, wide = qk ? a.wk : a.wv;
  const bool act = live && d < width, pad = live && !act && d < wide;
  const bool norm = a.qnorm_w != nullptr;
  const int C = (a.H + a.G) * a.dk + a.G * a.dv;
  const int c = (qk ? hs * a.dk : (a.H + a.G) * a.dk + (hs - a.H - a.G) * a.dv) + d;
  const TA* src = reinterpret_cast<const TA*>(a.proj) + (size_t)m.row0 * a.ld + c;
  const uint4 zero4 = make_uint4(0, 0, 0, 0);
  uint4* mine = raw + threadIdx.x;
  auto at = [&](int r) -> uint4* { return mine + ((r + kCapSlots) & (kCapSlots - 1)) * blockDim.x; };      // row r of the run, r >= -R
  auto fetch = [&](int r) {                            // (rows behind the run: zeros)
    if (act && r < m.n)
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((unsigned)__cvta_generic_to_shared(at(r))),
                   "l"(src + (int64_t)(m.q0 + r) * a.ld) : "memory");
    else
      *at(r) = zero4;
  };
  auto commit = [] { asm volatile("cp.async.commit_group;" ::: "memory"); };
  if constexpr (R > 0)
#pragma unroll
  for (int b = 0; b < R; ++b) {                        // the rows before the run
    const int q = m.q0 - 1 - b, p = m.ctx + q;
    uint4 x = zero4;
    if (act && q >= 0) {
      x = *reinterpret_cast<const uint4*>(src + (int64_t)q * a.ld);
    } else if (act && p >= 0 && m.slot >= 0) {
      const float* rp = a.ring + ((size_t)m.slot * R + p % RR) * C + c;
      TA* xv = reinterpret_cast<TA*>(&x);
#pragma unroll
      for (int i = 0; i < V; ++i) ca_store(xv + i, rp[i]);
    }
    *at(-1 - b) = x;
  }
  fetch(0);
  fetch(1);
  commit();
  fetch(2);
  fetch(3);
  commit();
  float w[TAPS][V];
  uint4 nraw = zero4;                                  // norm weights, bf16 (V of them)
  if (act) {
    conv_weights<TAPS, V>(w, a.conv_w, c, C);
    conv_ring_put<TA, TAPS>(m, src, a.ld, a.ring, c, C);
    if (norm && qk) {
      const bf16* nv = (is_q ? a.qnorm_w : a.knorm_w) + (a.joint ? (is_q ? hs : hs - a.H) * a.dk : 0) + d;
      bf16* nr = reinterpret_cast<bf16*>(&nraw);
#pragma unroll
      for (int i = 0; i < V; ++i) nr[i] = nv[i];
    }
  }
  const bool turn = act && qk && d < a.dims;            // (dims is a whole number of pieces)
  const int partner = (turn && a.half_layout) ? (d < half ? lane + half / V : lane - half / V) : lane;
  const int g = is_k ? hs - a.H : hs - a.H - a.G;
  const int row0 = m.row0 + m.q0;
  const float2* table = a.cs + (size_t)row0 * half + (a.half_layout ? (d < half ? d : d - half) : d / 2);
  const bool warp_q = (threadIdx.x >> 5) * per_warp < a.H;                                   // the warp holds query heads
  const bool warp_k = ((threadIdx.x >> 5) + 1) * per_warp > a.H && (threadIdx.x >> 5) * per_warp < a.H + a.G;
  const float inv_q = 1.0f / (float)(a.H * a.dk), inv_k = 1.0f / (float)(a.G * a.dk), inv_dk = 1.0f / (float)a.dk;
  const float sgn = d < half ? -1.0f : 1.0f;
  TA* q_dst = reinterpret_cast<TA*>(a.q_out) + ((size_t)row0 * a.H + hs) * a.wk + d;
  TA* const kv_dst = reinterpret_cast<TA*>(is_k ? a.k_cache : a.v_cache) + d;
  for (int r0 = 0; r0 < m.n; r0 += 2) {
    asm volatile("cp.async.wait_group 1;" ::: "memory");       // (a thread reads only what it fetched itself)
    float y[2][V], f[2] = {1.0f, 1.0f};
#pragma unroll
    for (int r = 0; r < 2; ++r)
#pragma unroll
      for (int i = 0; i < V; ++i) y[r][i] = 0.f;
    if (act) {
#pragma unroll
      for (int k = -R; k < 2; ++k) {                           // input row r0 + k serves rows r0 + k .. r0 + k + R
        const uint4 xr = *at(r0 + k);
        const TA* x = reinterpret_cast<const TA*>(&xr);
#pragma unroll
        for (int i = 0; i < V; ++i) {
          const float v = ca_f32(x[i]);
#pragma unroll
          for (int r = 0; r < 2; ++r)
            if (r - k >= 0 && r - k <= R) y[r][i] = fmaf(w[r - k >= 0 && r - k <= R ? r - k : 0][i], v, y[r][i]);
        }
      }
    }
    fetch(r0 + 4);
    fetch(r0 + 5);
    commit();
    if (norm) {
      float (*hss)[kCapJointWarps * 32] = head_ss[(r0 >> 1) & 1];
      float ss[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        ss[r] = 0.f;
#pragma unroll
        for (int i = 0; i < V; ++i) ss[r] = fmaf(y[r][i], y[r][i], ss[r]);
      }
      if (lph == 16) {                                         // (128-wide heads; all lanes take part)
#pragma unroll
        for (int o = 8; o > 0; o >>= 1)
#pragma unroll
          for (int r = 0; r < 2; ++r) ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], o);
      } else {
        for (int o = lph >> 1; o > 0; o >>= 1)
#pragma unroll
          for (int r = 0; r < 2; ++r) ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], o);
      }
      if (a.joint && li == 0) {
        hss[0][hs] = ss[0];
        hss[1][hs] = ss[1];
      }
      if (a.joint) {
        __syncthreads();                                       // (the other parity's sums may still be read)
        // half a warp sums one row: a fixed order, the same in every warp
        const int hr = lane >> 4, hl = lane & 15;
        float sq = 0.f, sk = 0.f;
        if (warp_q) {
          for (int h = hl; h < a.H; h += 16) sq += hss[hr][h];
#pragma unroll
          for (int o = 8; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
        }
        if (warp_k) {
          for (int h = a.H + hl; h < a.H + a.G; h += 16) sk += hss[hr][h];
#pragma unroll
          for (int o = 8; o > 0; o >>= 1) sk += __shfl_xor_sync(0xffffffffu, sk, o);
        }
        const float fq = rsqrtf(fmaf(sq, inv_q, a.eps)), fk = rsqrtf(fmaf(sk, inv_k, a.eps));
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const float bq = __shfl_sync(0xffffffffu, fq, 16 * r), bk = __shfl_sync(0xffffffffu, fk, 16 * r);
          if (qk) f[r] = is_q ? bq : bk;
        }
      } else if (qk) {
#pragma unroll
        for (int r = 0; r < 2; ++r) f[r] = rsqrtf(fmaf(ss[r], inv_dk, a.eps));
      }
      if (qk) {
        const bf16* nr = reinterpret_cast<const bf16*>(&nraw);
#pragma unroll
        for (int r = 0; r < 2; ++r)
#pragma unroll
          for (int i = 0; i < V; ++i) y[r][i] *= f[r] * __bfloat162float(nr[i]);
      }
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      if (r0 + r >= m.n) break;
      if (a.half_layout && a.dims > 0) {
#pragma unroll
        for (int i = 0; i < V; i += 2) {
          const float o0 = __shfl_sync(0xffffffffu, y[r][i], partner), o1 = __shfl_sync(0xffffffffu, y[r][i + 1], partner);
          if (turn) {
            const float4 t = *reinterpret_cast<const float4*>(table + (size_t)(r0 + r) * half + i);
            y[r][i] = fmaf(o0, sgn * t.y, y[r][i] * t.x);
            y[r][i + 1] = fmaf(o1, sgn * t.w, y[r][i + 1] * t.z);
          }
        }
      } else if (turn) {
#pragma unroll
        for (int i = 0; i < V; i += 2) {
          const float2 t = table[(size_t)(r0 + r) * half + i / 2];
          const float u = y[r][i], v = y[r][i + 1];
          y[r][i] = u * t.x - v * t.y;
          y[r][i + 1] = v * t.x + u * t.y;
        }
      }
      if (!act && !pad) continue;
      uint4 outv;
      TA* ov = reinterpret_cast<TA*>(&outv);
#pragma unroll
      for (int i = 0; i < V; ++i) ca_store(ov + i, y[r][i]);    // (zeros behind the head's own columns)
      if (is_q) {
        *reinterpret_cast<uint4*>(q_dst + (size_t)((r0 + r) * a.H) * a.wk) = outv;
      } else {
        const int slot = a.slots[row0 + r0 + r];
        if (slot >= 0)
          *reinterpret_cast<uint4*>(kv_dst + cap_cache_row(a, slot, g) * wide) = outv;
      }
    }
  }
}

// Any width, any number of taps: warps take the head slots in turn, lanes the columns; a head is staged in shared memory
// between the norm and the rotation.
template <typename TA>
__global__ void __launch_bounds__(kCapWarps * 32)
conv_attn_prep_joint_kernel(CapArgs a) {
  constexpr int NB = kCapRows;
  extern __shared__ __align__(16) float heads[];       // a head per warp
  __shared__ float red[kCapWarps][2][NB], mul[2][NB];
  const CapWork m = cap_work<NB>(a);
  if (m.n <= 0) return;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, half = a.dims >> 1, n_slots = a.H + 2 * a.G, R = a.taps - 1;
  const int C = (a.H + a.G) * a.dk + a.G * a.dv, wmax = a.dk > a.dv ? a.dk : a.dv;
  float* head = heads + warp * wmax;
  const TA* rows = reinterpret_cast<const TA*>(a.proj) + (size_t)m.row0 * a.ld;
  const bool norm = a.qnorm_w != nullptr;
  if (a.joint && norm) {
    float ss[2][NB];
#pragma unroll
    for (int r = 0; r < NB; ++r) ss[0][r] = ss[1][r] = 0.f;
    for (int hs = warp; hs < a.H + a.G; hs += kCapWarps)
      for (int d = lane; d < a.dk; d += 32)
#pragma unroll
        for (int r = 0; r < NB; ++r) {
          if (r >= m.n) break;
          const float y = conv_at<TA>(m, m.q0 + r, rows + hs * a.dk + d, a.ld, a.ring, a.conv_w, hs * a.dk + d, C, a.taps);
          if (hs < a.H) ss[0][r] = fmaf(y, y, ss[0][r]); else ss[1][r] = fmaf(y, y, ss[1][r]);
        }
#pragma unroll
    for (int p = 0; p < 2; ++p)
#pragma unroll
      for (int r = 0; r < NB; ++r) {
        const float v = warp_sum(ss[p][r]);
        if (lane == 0) red[warp][p][r] = v;
      }
    __syncthreads();
    if (threadIdx.x < 2 * NB) {
      const int p = threadIdx.x / NB, r = threadIdx.x % NB;
      float v = 0.f;
      for (int w = 0; w < kCapWarps; ++w) v += red[w][p][r];     // a fixed order
      mul[p][r] = 1.0f / sqrtf(v / (float)((p == 0 ? a.H : a.G) * a.dk) + a.eps);
    }
    __syncthreads();
  }
  for (int hs = warp; hs < n_slots; hs += kCapWarps) {
    const bool is_q = hs < a.H, is_k = !is_q && hs < a.H + a.G, qk = is_q || is_k;
    const int width = qk ? a.dk : a.dv, wide = qk ? a.wk : a.wv;
    const int col0 = qk ? hs * a.dk : (a.H + a.G) * a.dk + (hs - a.H - a.G) * a.dv;
    const int g = is_k ? hs - a.H : hs - a.H - a.G;
    const bf16* nv = is_q ? a.qnorm_w : a.knorm_w;
    if (norm && qk && a.joint) nv += (is_q ? hs : hs - a.H) * a.dk;
    for (int r = 0; r < m.n; ++r) {
      float ss = 0.f;
      for (int d = lane; d < width; d += 32) {
        const float y = conv_at<TA>(m, m.q0 + r, rows + col0 + d, a.ld, a.ring, a.conv_w, col0 + d, C, a.taps);
        head[d] = y;
        ss = fmaf(y, y, ss);
      }
      ss = warp_sum(ss);
      const float f = !(norm && qk) ? 1.0f : (a.joint ? mul[is_q ? 0 : 1][r] : 1.0f / sqrtf(ss / (float)a.dk + a.eps));
      if (norm && qk)
        for (int d = lane; d < width; d += 32) head[d] *= f * __bfloat162float(nv[d]);
      __syncwarp();
      const size_t row = (size_t)(m.row0 + m.q0 + r);
      TA* dst = nullptr;
      if (is_q) {
        dst = reinterpret_cast<TA*>(a.q_out) + (row * a.H + hs) * a.wk;
      } else if (a.slots[row] >= 0) {
        dst = reinterpret_cast<TA*>(is_k ? a.k_cache : a.v_cache) + cap_cache_row(a, a.slots[row], g) * wide;
      }
      if (dst != nullptr)
        for (int d = lane; d < wide; d += 32) {
          float y = d < width ? head[d] : 0.f;
          if (qk && d < a.dims) {
            const bool first = a.half_layout ? d < half : (d & 1) == 0;
            const int j = a.half_layout ? (first ? d : d - half) : d >> 1;
            const float o = head[a.half_layout ? (first ? d + half : d - half) : d ^ 1];
            const float2 t = a.cs[row * half + j];
            y = first ? y * t.x - o * t.y : y * t.x + o * t.y;
          }
          ca_store(dst + d, y);
        }
      __syncwarp();
    }
    if (R > 0 && m.q0 == 0 && m.slot >= 0) {           // every read of the ring by this warp's columns lies behind it
      for (int b = 0; b < R; ++b) {
        const int q = m.qlen - 1 - b;
        if (q < 0) break;
        float* rp = a.ring + ((size_t)m.slot * R + (m.ctx + q) % R) * C + col0;
        for (int d = lane; d < width; d += 32) rp[d] = ca_f32(rows[(size_t)q * a.ld + col0 + d]);
      }
    }
  }
}

}  // namespace b200

using namespace b200;

extern "C" int b200_conv_attn_prep_ex(const void* proj, int f32, int64_t ld, const float* conv_w, int taps, const void* qnorm_w,
                                   const void* knorm_w, float* ring, const int32_t* cu_seq, const int32_t* ctx_lens,
                                   const int32_t* state_slots, const int32_t* tile_seq, const int32_t* tile_q0, int n_tiles,
                                   int tile_rows, int n_prompt, int n_single, const int32_t* slots, void* q_out,
                                   void* k_cache, void* v_cache, int H, int G, int dk, int dv, int wk, int wv, int page,
                                   float eps, int joint_norm, int rot_dims, int half_layout, const float* cos_sin, void* stream) {
  B200_REQUIRE(H > 0 && G > 0 && H % G == 0 && dk > 0 && dv > 0 && wk >= dk && wv >= dv && page > 0,
               "conv_attn_prep: bad shape H=%d G=%d dk=%d dv=%d in %d / %d", H, G, dk, dv, wk, wv);
  B200_REQUIRE(taps >= 1 && taps <= kCapMaxTaps, "conv_attn_prep: %d taps (1 .. %d)", taps, kCapMaxTaps);
  B200_REQUIRE(taps == 1 || (ring != nullptr && state_slots != nullptr), "conv_attn_prep: more than one tap needs the sequences' rings");
  B200_REQUIRE(n_tiles == 0 || (tile_rows > 0 && tile_rows % kCapRows == 0), "conv_attn_prep: tiles of %d rows (multiples of %d)",
               tile_rows, kCapRows);
  B200_REQUIRE(n_tiles >= 0 && n_prompt >= 0 && n_single >= 0, "conv_attn_prep: bad counts");
  B200_REQUIRE(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= dk && (rot_dims == 0 || cos_sin != nullptr),
               "conv_attn_prep: %d rotated entries of %d", rot_dims, dk);
  B200_REQUIRE(!joint_norm || (qnorm_w != nullptr && knorm_w != nullptr), "conv_attn_prep: the joint norm has weights");
  const int per_tile = n_tiles > 0 ? tile_rows / kCapRows : 1;
  const int n_x = n_tiles * per_tile + n_single;
  if (n_x == 0) return B200_OK;
  int shift = 0;
  while ((1 << shift) < page) ++shift;
  CapArgs a{proj, ld, conv_w, (const bf16*)qnorm_w, (const bf16*)knorm_w, taps > 1 ? ring : nullptr, cu_seq, ctx_lens,
                  state_slots, tile_seq, tile_q0, n_tiles * per_tile, per_tile, n_prompt, slots, q_out, k_cache, v_cache, H, G,
                  dk, dv, wk, wv, page, (1 << shift) == page ? shift : -1, taps, eps, joint_norm, rot_dims, half_layout, (const float2*)cos_sin};
  cudaStream_t s = (cudaStream_t)stream;
  const int n_heads = H + 2 * G, esz = f32 ? 4 : 2, vec = 16 / esz, wmax = wk > wv ? wk : wv;
  const int C = (H + G) * dk + G * dv;
  const bool al = ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(q_out) | reinterpret_cast<uintptr_t>(k_cache) |
                    reinterpret_cast<uintptr_t>(v_cache) | reinterpret_cast<uintptr_t>(conv_w) | reinterpret_cast<uintptr_t>(a.ring)) & 15) == 0;
  if (joint_norm || rot_dims > 0) {
    const int piece = half_layout ? 2 * vec : vec;      // the rotated entries in whole pieces (and their partners too)
    int lph = 1;
    while (lph < wmax / vec) lph <<= 1;
    const int warps = lph <= 32 ? (n_heads + 32 / lph - 1) / (32 / lph) : 1 << 20;       // all head slots in one CTA
    const size_t smem_v = sizeof(uint4) * kCapSlots * 32 * (size_t)warps;
    if (al && taps <= 4 && dk % vec == 0 && dv % vec == 0 && wk % vec == 0 && wv % vec == 0 && ld % vec == 0 && C % 4 == 0 &&
        warps <= kCapJointWarps && rot_dims % piece == 0 && (n_tiles == 0 || tile_rows % kCapRun == 0) &&
        (reinterpret_cast<uintptr_t>(cos_sin) & 15) == 0) {
      a.per_tile = n_tiles > 0 ? tile_rows / kCapRun : 1;
      a.n_pieces = n_tiles * a.per_tile;
      const int n_run = a.n_pieces + n_single;
#define B200_CAJ(TA, N)                                                                                                       \
  do {                                                                                                                        \
    if (smem_v > 32 * 1024) {                                                                                                 \
      const cudaError_t e = cudaFuncSetAttribute(conv_attn_prep_joint_vec_kernel<TA, N>,                                      \
                                                 cudaFuncAttributeMaxDynamicSharedMemorySize,                                 \
                                                 (int)(sizeof(uint4) * kCapSlots * 32 * kCapJointWarps));                     \
      if (e != cudaSuccess) {                                                                                                 \
        b200_set_error("conv_attn_prep(joint): %s", cudaGetErrorString(e));                                                   \
        return B200_ERR_CUDA;                                                                                                 \
      }                                                                                                                       \
    }                                                                                                                         \
    conv_attn_prep_joint_vec_kernel<TA, N><<<n_run, warps * 32, smem_v, s>>>(a, lph);                                         \
  } while (0)
#define B200_CAJT(TA)                        \
  switch (taps) {                            \
    case 1: B200_CAJ(TA, 1); break;          \
    case 2: B200_CAJ(TA, 2); break;          \
    case 3: B200_CAJ(TA, 3); break;          \
    default: B200_CAJ(TA, 4);                \
  }
      if (f32) { B200_CAJT(float) } else { B200_CAJT(bf16) }
#undef B200_CAJT
#undef B200_CAJ
      return b200_check_launch("b200_conv_attn_prep(joint)");
    }
    const size_t smem = sizeof(float) * kCapWarps * (dk > dv ? dk : dv);
    B200_REQUIRE(smem <= 40 * 1024, "conv_attn_prep: heads of %d / %d entries exceed the staged head", dk, dv);
    if (f32) conv_attn_prep_joint_kernel<float><<<n_x, kCapWarps * 32, smem, s>>>(a);
    else conv_attn_prep_joint_kernel<bf16><<<n_x, kCapWarps * 32, smem, s>>>(a);
    return b200_check_launch("b200_conv_attn_prep(joint)");
  }
  if (al && taps <= 4 && dk % vec == 0 && dv % vec == 0 && wk % vec == 0 && wv % vec == 0 && ld % vec == 0 && C % 4 == 0 && wmax / vec <= 32) {
    int lph = 1;
    while (lph < wmax / vec) lph <<= 1;
    // warps that cover all head slots, in CTAs of equal size
    const int all_warps = (n_heads + 32 / lph - 1) / (32 / lph), ny = (all_warps + kCapWarps - 1) / kCapWarps;
    const int warps = (all_warps + ny - 1) / ny;
    const dim3 grid(n_x, ny);
#define B200_CAP(TA, N) conv_attn_prep_vec_kernel<TA, N><<<grid, warps * 32, 0, s>>>(a, lph)
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

extern "C" int b200_conv_attn_prep(const void* proj, int f32, int64_t ld, const float* conv_w, int taps, const void* qnorm_w,
                                   const void* knorm_w, float* ring, const int32_t* cu_seq, const int32_t* ctx_lens,
                                   const int32_t* state_slots, const int32_t* tile_seq, const int32_t* tile_q0, int n_tiles,
                                   int tile_rows, int n_prompt, int n_single, const int32_t* slots, void* q_out,
                                   void* k_cache, void* v_cache, int H, int G, int dk, int dv, int wk, int wv, int page,
                                   float eps, void* stream) {
  return b200_conv_attn_prep_ex(proj, f32, ld, conv_w, taps, qnorm_w, knorm_w, ring, cu_seq, ctx_lens, state_slots, tile_seq, tile_q0,
                                n_tiles, tile_rows, n_prompt, n_single, slots, q_out, k_cache, v_cache, H, G, dk, dv, wk, wv, page, eps,
                                0, 0, 0, nullptr, stream);
}

extern "C" int b200_rot_table(const int32_t* positions, const double* freq, float* cos_sin, int T, int half, void* stream) {
  B200_REQUIRE(T >= 0 && half > 0, "rot_table: bad shape");
  if (T == 0) return B200_OK;
  rot_table_kernel<<<(T * half + 255) / 256, 256, 0, (cudaStream_t)stream>>>(positions, freq, (float2*)cos_sin, half, T * half);
  return b200_check_launch("b200_rot_table");
}
