// Recurrences on a matrix state per head with ONE decay per head and token, state in fp32.
//
//   state space:  S_t = g S_(t-1) + beta k_t v_t^T                      g = exp(-rate softplus(a + bias)), beta = softplus(a + bias)
//                 o_t = S_t^T q_t + skip v_t
//   delta rule:   S  <- g S_(t-1);  u = beta (v_t - S^T k_t);  S_t = S + k_t u^T;  o_t = S_t^T q_t
//                 g = exp(-rate softplus(a + bias)), beta = sigmoid(b)
// (S: dk x dv, zero before a sequence's first token; head h reads query / key head h / (H / G).)  Queries, keys and values
// arrive as fp32 rows whose heads are padded with zeros to a multiple of 4 entries (conv_rec_prep.cu); the gates' raw
// projections are fp32 rows, and everything formed from them is fp32.  The state of slot s is S [slots][H][dv][dkp] (key index
// fastest, dkp = dk rounded up to 4).  A sequence whose context is empty starts from zero, whatever its slot held.
//
// Every value column of S is a recurrence of its own, so columns are the unit of work: L lanes share C neighbouring columns,
// lane l holds the key entries 4 (i L + l) .. + 3 (i < R4) of each in registers, and a warp walks its C 32 / L columns
// through the sequence's new rows one token after the other.  Per token: S^T k (a butterfly over the L lanes; delta rule
// only), the update, and the lane's share of S^T q.  Those shares stay in registers for 8 tokens and are then summed over the
// lanes in one transposing exchange (about 2 shuffles a token).  A token's keys and queries are read from shared memory once
// per lane and serve its C columns: with one column that read, not the arithmetic, bounds the walk.  Keys, queries, values and gates are staged 16 or 32 tokens at a time by
// cp.async into two buffers, so the walk never waits for memory; a column's sums do not depend on how a prompt was cut
// beyond the order of the lanes' addends in S^T q.
#include "common.cuh"
#include "runtime.h"
#include "../../include/b200.h"

namespace b200 {

constexpr int kGsWarps = 8;

struct GatedScanArgs {
  const float* x;
  int64_t ld;
  int q_col, k_col, v_col;
  const float* gates;              // [T][ld_g]: delta [b: H | a: H], state space [a: H]
  int64_t ld_g;
  const float* rate;               // [H]
  const float* dt_bias;            // [H]
  const float* skip;               // [H] or null
  const int32_t* cu_seq;
  const int32_t* ctx_lens;
  const int32_t* state_slots;
  float* S;
  float* o;                        // [T][H dv]
  int H, G, dkp, dv, dvp;
};

// two fp32 numbers in one 64-bit register pair: the packed fused multiply-add of sm_100
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float a, float b) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float sum2(f32x2 v) {
  float a, b;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v));
  return a + b;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f32x2 add2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

__device__ __forceinline__ float gs_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// (decay, step) of a token from the raw gates
template <bool DELTA>
__device__ __forceinline__ float2 gs_gate(float a, float b, float rate, float bias) {
  const float sp = gs_softplus(a + bias);
  return make_float2(expf(-rate * sp), DELTA ? 1.0f / (1.0f + expf(-b)) : sp);
}

__device__ __forceinline__ void cp16(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 16;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

template <int L>
__device__ __forceinline__ float lanes_sum(float v) {
#pragma unroll
  for (int o = L / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// the lane's shares of S^T x for C columns
template <int R2, int C>
__device__ __forceinline__ void gs_dot(const f32x2 (&S)[C][R2], const f32x2 (&x)[R2], float (&o)[C]) {
#pragma unroll
  for (int c = 0; c < C; ++c) {
    f32x2 p0 = mul2(S[c][0], x[0]), p1 = mul2(S[c][1], x[1]);
#pragma unroll
    for (int i = 2; i < R2; i += 2) {
      p0 = fma2(S[c][i], x[i], p0);
      p1 = fma2(S[c][i + 1], x[i + 1], p1);
    }
    o[c] = sum2(add2(p0, p1));
  }
}

// sums over the L lanes of a group, in every lane.  Two columns: the lanes' halves take one each and exchange the sums.
template <int L, int C>
__device__ __forceinline__ void gs_lanes_sum(float (&p)[C]) {
  if constexpr (C == 2 && L > 8) {
    const bool hi = threadIdx.x & (L / 2);
    float mine = (hi ? p[1] : p[0]) + __shfl_xor_sync(0xffffffffu, hi ? p[0] : p[1], L / 2);
#pragma unroll
    for (int w = L / 4; w > 0; w >>= 1) mine += __shfl_xor_sync(0xffffffffu, mine, w);
    const float other = __shfl_xor_sync(0xffffffffu, mine, L / 2);
    p[0] = hi ? other : mine;
    p[1] = hi ? mine : other;
  } else {
#pragma unroll
    for (int w = L / 2; w > 0; w >>= 1)
#pragma unroll
      for (int c = 0; c < C; ++c) p[c] += __shfl_xor_sync(0xffffffffu, p[c], w);
  }
}

// One token of C columns: S <- g S + k u^T with u = beta v, or beta (v - g S^T k) for the delta rule.  The read-out of the
// token BEFORE (o, from q; none for a block's first token) and the decay of S need no other lane: they run while the
// butterfly's shuffles are in flight.
template <int L, int R2, int C, bool DELTA, bool READ>
__device__ __forceinline__ void gs_token(f32x2 (&S)[C][R2], const f32x2 (&k)[R2], const f32x2 (&q)[R2], const float (&v)[C], float2 gb,
                                         float (&o)[C]) {
  float p[C];
  if (DELTA) {
    gs_dot<R2, C>(S, k, p);
    gs_lanes_sum<L, C>(p);
  }
  if (READ) gs_dot<R2, C>(S, q, o);
  const f32x2 g2 = pack2(gb.x, gb.x);
#pragma unroll
  for (int c = 0; c < C; ++c)
#pragma unroll
    for (int i = 0; i < R2; ++i) S[c][i] = mul2(g2, S[c][i]);
#pragma unroll
  for (int c = 0; c < C; ++c) {
    const float u = DELTA ? gb.y * (v[c] - gb.x * p[c]) : gb.y * v[c];
    const f32x2 u2 = pack2(u, u);
#pragma unroll
    for (int i = 0; i < R2; ++i) S[c][i] = fma2(k[i], u2, S[c][i]);
  }
}

// 4 R4 entries of a row of key entries: lane l of L takes entries 4 (i L + l) .. + 3
template <int L, int R4>
__device__ __forceinline__ void gs_row(const float* __restrict__ row, int l, f32x2 (&r)[2 * R4]) {
#pragma unroll
  for (int i = 0; i < R4; ++i) {
    const ulonglong2 t = *reinterpret_cast<const ulonglong2*>(row + 4 * (i * L + l));
    r[2 * i] = t.x;
    r[2 * i + 1] = t.y;
  }
}

template <int L, int R4, int C, int TOK, bool DELTA>
__global__ void __launch_bounds__(kGsWarps * 32, C * R4 <= 4 ? 2 : 1)
gated_scan_kernel(GatedScanArgs a) {
  extern __shared__ __align__(16) float smem[];
  constexpr int R2 = 2 * R4, DKP = 4 * R4 * L, CPW = C * 32 / L, COLS = kGsWarps * CPW, OP = COLS + 8;
  float* ks = smem;                                   // [2][TOK][DKP]
  float* qs = ks + 2 * TOK * DKP;                  // [2][TOK][DKP]
  float* vs = qs + 2 * TOK * DKP;                  // [2][TOK][COLS]
  float2* gb = reinterpret_cast<float2*>(vs + 2 * TOK * COLS);   // [2][TOK]
  float* os = reinterpret_cast<float*>(gb + 2 * TOK);            // [TOK][OP]
  const int s = blockIdx.x, h = blockIdx.y, z = blockIdx.z, tid = threadIdx.x;
  const int slot = a.state_slots[s];
  if (slot < 0) return;
  const int t0 = a.cu_seq[s], t1 = a.cu_seq[s + 1];
  if (t1 <= t0) return;
  const int warp = tid >> 5, lane = tid & 31, l = lane % L;
  const int cw = warp * CPW + lane / L * C, col = z * COLS + cw;     // this lane's first column, in the CTA and in the head
  const int hk = h / (a.H / a.G);
  const int dkp = a.dkp;
  float* Sp = a.S + (((size_t)slot * a.H + h) * a.dv + col) * dkp;
  const bool fresh = a.ctx_lens[s] == 0;
  f32x2 S[C][R2];
#pragma unroll
  for (int c = 0; c < C; ++c)
#pragma unroll
    for (int i = 0; i < R4; ++i) {
      ulonglong2 t = make_ulonglong2(0, 0);
      if (!fresh && col + c < a.dv && 4 * (i * L + l) < dkp) t = *reinterpret_cast<const ulonglong2*>(Sp + c * dkp + 4 * (i * L + l));
      S[c][2 * i] = t.x;
      S[c][2 * i + 1] = t.y;
    }
  // key entries behind dkp: zeros in both buffers, written once
  if (dkp < DKP) {
    const int pad = DKP - dkp;
    for (int i = tid; i < 2 * TOK * pad; i += kGsWarps * 32) {
      const int r = i / pad, d = dkp + i % pad;
      ks[r * DKP + d] = 0.f;
      qs[r * DKP + d] = 0.f;
    }
  }
  const float rate = a.rate[h], bias = a.dt_bias[h];
  const float4 zero4 = make_float4(0.f, 0.f, 0.f, 0.f);
  // this thread's share of the staging: entries d0 .. d0 + 3 of rows tt0, tt0 + per_pass, ... (dkp <= 512: at least one pass)
  const int dk4 = dkp >> 2, per_pass = kGsWarps * 32 / dk4, d0 = tid % dk4 * 4;
  const int tt0 = tid / dk4 < per_pass ? tid / dk4 : TOK;
  const float* src = a.x + hk * dkp + d0;
  auto stage = [&](int ch, int buf) {                 // rows ch .. ch + TOK - 1; rows behind the portion are zeros
    const int nt = min(TOK, t1 - ch);
    for (int tt = tt0; tt < TOK; tt += per_pass) {
      const int to = (buf * TOK + tt) * DKP + d0;
      if (tt < nt) {
        const float* row = src + (size_t)(ch + tt) * a.ld;
        cp16(ks + to, row + a.k_col);
        cp16(qs + to, row + a.q_col);
      } else {
        *reinterpret_cast<float4*>(ks + to) = zero4;
        *reinterpret_cast<float4*>(qs + to) = zero4;
      }
    }
    for (int i = tid; i < TOK * (COLS / 4); i += kGsWarps * 32) {
      const int tt = i / (COLS / 4), c = (i - tt * (COLS / 4)) * 4;
      float* to = vs + (buf * TOK + tt) * COLS + c;
      if (tt < nt && z * COLS + c < a.dvp) cp16(to, a.x + (size_t)(ch + tt) * a.ld + a.v_col + h * a.dvp + z * COLS + c);
      else *reinterpret_cast<float4*>(to) = zero4;
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  float ra = 0.f, rb = 0.f;
  auto raw_gates = [&](int ch) {
    if (tid < TOK && ch + tid < t1) {
      const float* g = a.gates + (size_t)(ch + tid) * a.ld_g;
      ra = DELTA ? g[a.H + h] : g[h];
      if (DELTA) rb = g[h];
    }
  };
  auto put_gates = [&](int ch, int buf) {             // rows behind the portion: decay 1, step 0 (the state stays)
    if (tid < TOK) gb[buf * TOK + tid] = ch + tid < t1 ? gs_gate<DELTA>(ra, rb, rate, bias) : make_float2(1.f, 0.f);
  };
  stage(t0, 0);
  raw_gates(t0);
  put_gates(t0, 0);
  int buf = 0;
  for (int ch = t0; ch < t1; ch += TOK, buf ^= 1) {
    const int nt = min(TOK, t1 - ch), next = ch + TOK;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                  // this chunk is staged; the last one's outputs have left os
    if (next < t1) {
      stage(next, buf ^ 1);
      raw_gates(next);
    }
#pragma unroll 1
    for (int tb = 0; tb < nt; tb += 8) {
      float o[8][C];
      f32x2 k[2][R2], q[2][R2];      // this token's and the next one's keys; the last token's and this one's queries
      const float* kr = ks + (buf * TOK + tb) * DKP;
      const float* qr = qs + (buf * TOK + tb) * DKP;
      const float* vr = vs + (buf * TOK + tb) * COLS + cw;
      const float2* gr = gb + buf * TOK + tb;
      gs_row<L, R4>(kr, l, k[0]);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        float v[C];
#pragma unroll
        for (int c = 0; c < C; ++c) v[c] = vr[j * COLS + c];
        if (j < 7) gs_row<L, R4>(kr + (j + 1) * DKP, l, k[(j + 1) & 1]);
        gs_row<L, R4>(qr + j * DKP, l, q[j & 1]);
        if (j == 0) gs_token<L, R2, C, DELTA, false>(S, k[0], q[1], v, gr[0], o[0]);
        else gs_token<L, R2, C, DELTA, true>(S, k[j & 1], q[(j + 1) & 1], v, gr[j], o[j - 1]);
      }
      gs_dot<R2, C>(S, q[1], o[7]);
      // lane l ends with token tb + (l & 7), summed over the columns' lanes
      const bool b4 = l & 4, b2 = l & 2, b1 = l & 1;
      float sum[C];
#pragma unroll
      for (int c = 0; c < C; ++c) {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float mine = b4 ? o[j + 4][c] : o[j][c], other = b4 ? o[j][c] : o[j + 4][c];
          o[j][c] = mine + __shfl_xor_sync(0xffffffffu, other, 4);
        }
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const float mine = b2 ? o[j + 2][c] : o[j][c], other = b2 ? o[j][c] : o[j + 2][c];
          o[j][c] = mine + __shfl_xor_sync(0xffffffffu, other, 2);
        }
        const float mine = b1 ? o[1][c] : o[0][c], other = b1 ? o[0][c] : o[1][c];
        sum[c] = mine + __shfl_xor_sync(0xffffffffu, other, 1);
      }
      if constexpr (C == 2 && L > 8) {                 // the lanes' halves of 8 take one column each
        const bool hi = l & 8;
        float one = (hi ? sum[1] : sum[0]) + __shfl_xor_sync(0xffffffffu, hi ? sum[0] : sum[1], 8);
#pragma unroll
        for (int w = 16; w < L; w <<= 1) one += __shfl_xor_sync(0xffffffffu, one, w);
        if (l < 16) os[(tb + (l & 7)) * OP + cw + (hi ? 1 : 0)] = one;
      } else {
#pragma unroll
        for (int c = 0; c < C; ++c) {
#pragma unroll
          for (int w = 8; w < L; w <<= 1) sum[c] += __shfl_xor_sync(0xffffffffu, sum[c], w);
          if (l < 8) os[(tb + l) * OP + cw + c] = sum[c];
        }
      }
    }
    if (next < t1) put_gates(next, buf ^ 1);
    __syncthreads();
    const float sk = a.skip != nullptr ? a.skip[h] : 0.f;
    for (int i = tid; i < nt * COLS; i += kGsWarps * 32) {
      const int tt = i / COLS, c = i - tt * COLS;
      if (z * COLS + c < a.dv)
        a.o[(size_t)(ch + tt) * a.H * a.dv + h * a.dv + z * COLS + c] =
            fmaf(sk, vs[(buf * TOK + tt) * COLS + c], os[tt * OP + c]);
    }
  }
#pragma unroll
  for (int c = 0; c < C; ++c)
#pragma unroll
    for (int i = 0; i < R4; ++i)
      if (col + c < a.dv && 4 * (i * L + l) < dkp)
        *reinterpret_cast<ulonglong2*>(Sp + c * dkp + 4 * (i * L + l)) = make_ulonglong2(S[c][2 * i], S[c][2 * i + 1]);
}

// Single rows (a decode step): the state, the token's rows and its gates are in flight together; no staging, no barrier.
template <int L, int R4, bool DELTA>
__global__ void __launch_bounds__(kGsWarps * 32, 4)
gated_step_kernel(GatedScanArgs a) {
  constexpr int R2 = 2 * R4, CPW = 32 / L, COLS = kGsWarps * CPW;
  const int s = blockIdx.x, h = blockIdx.y, z = blockIdx.z;
  const int slot = a.state_slots[s];
  if (slot < 0) return;
  const int t = a.cu_seq[s];
  if (a.cu_seq[s + 1] <= t) return;
  const int lane = threadIdx.x & 31, l = lane % L, col = z * COLS + (threadIdx.x >> 5) * CPW + lane / L;
  const int hk = h / (a.H / a.G), dkp = a.dkp;
  const bool live = col < a.dv, fresh = a.ctx_lens[s] == 0;
  float* Sp = a.S + (((size_t)slot * a.H + h) * a.dv + col) * dkp;
  const float* row = a.x + (size_t)t * a.ld;
  f32x2 S[1][R2], k[R2], q[R2];
#pragma unroll
  for (int i = 0; i < R4; ++i) {
    const int d = 4 * (i * L + l);
    ulonglong2 ts = make_ulonglong2(0, 0), tk = ts, tq = ts;
    if (d < dkp) {
      if (live && !fresh) ts = *reinterpret_cast<const ulonglong2*>(Sp + d);
      tk = *reinterpret_cast<const ulonglong2*>(row + a.k_col + hk * dkp + d);
      tq = *reinterpret_cast<const ulonglong2*>(row + a.q_col + hk * dkp + d);
    }
    S[0][2 * i] = ts.x; S[0][2 * i + 1] = ts.y;
    k[2 * i] = tk.x; k[2 * i + 1] = tk.y;
    q[2 * i] = tq.x; q[2 * i + 1] = tq.y;
  }
  const float v[1] = {live ? row[a.v_col + h * a.dvp + col] : 0.f};
  const float* g = a.gates + (size_t)t * a.ld_g;
  const float2 gb = gs_gate<DELTA>(DELTA ? g[a.H + h] : g[h], DELTA ? g[h] : 0.f, a.rate[h], a.dt_bias[h]);
  float o[1];
  gs_token<L, R2, 1, DELTA, false>(S, k, q, v, gb, o);
  gs_dot<R2, 1>(S, q, o);
  o[0] = lanes_sum<L>(o[0]);
  if (!live) return;
#pragma unroll
  for (int i = 0; i < R4; ++i) {
    const int d = 4 * (i * L + l);
    if (d < dkp) *reinterpret_cast<ulonglong2*>(Sp + d) = make_ulonglong2(S[0][2 * i], S[0][2 * i + 1]);
  }
  if (l == 0) a.o[(size_t)t * a.H * a.dv + h * a.dv + col] = a.skip != nullptr ? fmaf(a.skip[h], v[0], o[0]) : o[0];
}

template <int L, int R4, int C, bool DELTA>
int gated_scan_launch(const GatedScanArgs& a, int n_seqs, cudaStream_t s) {
  constexpr int COLS = kGsWarps * C * (32 / L), DKP = 4 * R4 * L;
  constexpr int TOK = DKP <= 128 ? 32 : 16;
  const dim3 grid(n_seqs, a.H, (a.dv + COLS - 1) / COLS);
  constexpr size_t smem = sizeof(float) * (4 * (size_t)TOK * DKP + 2 * TOK * COLS + 4 * TOK + TOK * (COLS + 8));
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(gated_scan_kernel<L, R4, C, TOK, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) {
      b200_set_error("gated_scan: %zu bytes of shared memory: %s", smem, cudaGetErrorString(e));
      return B200_ERR_CUDA;
    }
  }
  gated_scan_kernel<L, R4, C, TOK, DELTA><<<grid, kGsWarps * 32, smem, s>>>(a);
  return b200_check_launch("b200_gated_scan");
}

// L, R4: single rows; PL, PR4: prompt portions (fewer entries of two columns per lane: the same registers, half the reads)
template <int L, int R4, int PL, int PR4, bool DELTA>
int gated_scan_form(const GatedScanArgs& a, int n_seqs, int max_len, cudaStream_t s) {
  if (max_len == 1) {
    constexpr int COLS = kGsWarps * (32 / L);
    gated_step_kernel<L, R4, DELTA><<<dim3(n_seqs, a.H, (a.dv + COLS - 1) / COLS), kGsWarps * 32, 0, s>>>(a);
    return b200_check_launch("b200_gated_scan(step)");
  }
  // too few CTAs to fill the GPU: the widest spread of a column over lanes, the shortest walk per token
  if constexpr (PL == 16 && PR4 == 2) {
    constexpr int COLS = kGsWarps * 2 * (32 / PL);
    if (n_seqs * a.H * ((a.dv + COLS - 1) / COLS) < 148) return gated_scan_launch<32, 1, 2, DELTA>(a, n_seqs, s);
  }
  return gated_scan_launch<PL, PR4, 2, DELTA>(a, n_seqs, s);
}

template <bool DELTA>
int gated_scan_pick(const GatedScanArgs& a, int n_seqs, int max_len, cudaStream_t s) {
  if (a.dkp <= 32) return gated_scan_form<8, 1, 8, 1, DELTA>(a, n_seqs, max_len, s);
  if (a.dkp <= 64) return gated_scan_form<8, 2, 16, 1, DELTA>(a, n_seqs, max_len, s);
  if (a.dkp <= 96) return gated_scan_form<8, 3, 8, 3, DELTA>(a, n_seqs, max_len, s);
  if (a.dkp <= 128) return gated_scan_form<8, 4, 16, 2, DELTA>(a, n_seqs, max_len, s);
  if (a.dkp <= 256) return gated_scan_form<16, 4, 32, 2, DELTA>(a, n_seqs, max_len, s);
  return gated_scan_form<32, 4, 32, 4, DELTA>(a, n_seqs, max_len, s);
}

// ------------------------------------------------------------------------------------------- out
// out = RMSnorm over `parts` equal pieces of (y * silu(z)), times w[channel] -- the gate BEFORE the norm -- or, with the gate
// AFTER it, RMSnorm of the pieces of y times w[place in the piece] (one weight vector for all pieces) times silu(z).  One CTA
// per row; the row is staged in shared memory between the statistic and the product.
template <typename TA>
__device__ __forceinline__ float4 gs_ld4(const TA* p);
template <>
__device__ __forceinline__ float4 gs_ld4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <>
__device__ __forceinline__ float4 gs_ld4<bf16>(const bf16* p) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  return make_float4(bf16_lo(r.x), bf16_hi(r.x), bf16_lo(r.y), bf16_hi(r.y));
}
__device__ __forceinline__ float gs_ld1(const float* p) { return *p; }
__device__ __forceinline__ float gs_ld1(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void gs_st1(float* p, float v) { *p = v; }
__device__ __forceinline__ void gs_st1(bf16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void gs_st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void gs_st4(bf16* p, float4 v) { *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w)); }
__device__ __forceinline__ float gs_silu(float z) { return z / (1.0f + expf(-z)); }

constexpr int kGnThreads = 256;

template <typename TA, bool VEC, bool AFTER>
__global__ void __launch_bounds__(kGnThreads)
gate_norm_kernel(const float* __restrict__ y, const TA* __restrict__ proj, int64_t ld, int z_col, const bf16* __restrict__ w,
                 TA* out, int64_t ldo, int C, int parts, float eps) {
  extern __shared__ __align__(16) float row[];        // [C], then the warps' partial sums
  __shared__ float sums[kGnThreads / 32];
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  constexpr int NW = kGnThreads / 32, V = VEC ? 4 : 1;
  const float* yr = y + (size_t)t * C;
  const TA* zr = proj + (size_t)t * ld + z_col;
  TA* o = out + (size_t)t * ldo;
  const int W = C / parts, per = parts >= NW ? 1 : NW / parts;       // warps that share a part
  for (int p0 = 0; p0 < parts; p0 += NW / per) {
    const int p = p0 + warp / per, sub = warp % per;
    const bool live = p < parts && warp / per < NW / per;
    float ss = 0.f;
    if (live)
      for (int i = (sub * 32 + lane) * V; i < W; i += per * 32 * V) {
        const int c = p * W + i;
        if (VEC) {
          float4 v = *reinterpret_cast<const float4*>(yr + c);
          if (!AFTER) {
            const float4 g = gs_ld4<TA>(zr + c);
            v.x *= gs_silu(g.x); v.y *= gs_silu(g.y); v.z *= gs_silu(g.z); v.w *= gs_silu(g.w);
          }
          *reinterpret_cast<float4*>(row + c) = v;
          ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
        } else {
          const float v = AFTER ? yr[c] : yr[c] * gs_silu(gs_ld1(zr + c));
          row[c] = v;
          ss = fmaf(v, v, ss);
        }
      }
    ss = warp_sum(ss);
    if (per > 1) {
      if (lane == 0) sums[warp] = ss;
      __syncthreads();
      if (live) {
        ss = 0.f;
        for (int i = 0; i < per; ++i) ss += sums[warp - sub + i];    // the same order in every warp
      }
    }
    if (!live) continue;
    const float rstd = 1.0f / sqrtf(ss / (float)W + eps);
    for (int i = (sub * 32 + lane) * V; i < W; i += per * 32 * V) {  // (each thread reads back what it staged itself)
      const int c = p * W + i;
      if (VEC) {
        float4 v = *reinterpret_cast<const float4*>(row + c);
        const float4 g = gs_ld4<bf16>(w + (AFTER ? i : c));
        if (AFTER) {
          const float4 t = gs_ld4<TA>(zr + c);
          v.x *= gs_silu(t.x); v.y *= gs_silu(t.y); v.z *= gs_silu(t.z); v.w *= gs_silu(t.w);
        }
        gs_st4(o + c, make_float4(v.x * rstd * g.x, v.y * rstd * g.y, v.z * rstd * g.z, v.w * rstd * g.w));
      } else {
        gs_st1(o + c, row[c] * rstd * gs_ld1(w + (AFTER ? i : c)) * (AFTER ? gs_silu(gs_ld1(zr + c)) : 1.0f));
      }
    }
  }
}

// Pieces of up to 128 channels (a head): W / 4 neighbouring lanes share one, a thread holds up to 8 of its row's 16-byte
// groups in registers and all their loads are in flight together.
template <typename TA, bool AFTER>
__global__ void __launch_bounds__(kGnThreads)
gate_norm_heads_kernel(const float* __restrict__ y, const TA* __restrict__ proj, int64_t ld, int z_col, const bf16* __restrict__ w, TA* out,
                       int64_t ldo, int C, int W, float eps) {
  constexpr int N = 8;
  const int t = blockIdx.x, i0 = threadIdx.x * 4, step = kGnThreads * 4, lanes = W >> 2;
  const float* yr = y + (size_t)t * C;
  const TA* zr = proj + (size_t)t * ld + z_col;
  TA* o = out + (size_t)t * ldo;
  float4 v[N], g[N];
#pragma unroll
  for (int n = 0; n < N; ++n) {
    const int i = i0 + n * step;
    if (n * step >= C) break;
    v[n] = g[n] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < C) {
      v[n] = *reinterpret_cast<const float4*>(yr + i);
      g[n] = gs_ld4<TA>(zr + i);
    }
  }
#pragma unroll
  for (int n = 0; n < N; ++n) {
    const int i = i0 + n * step;
    if (n * step >= C) break;
    g[n] = make_float4(gs_silu(g[n].x), gs_silu(g[n].y), gs_silu(g[n].z), gs_silu(g[n].w));
    float4 x = v[n];
    if (!AFTER) { x.x *= g[n].x; x.y *= g[n].y; x.z *= g[n].z; x.w *= g[n].w; }
    float ss = fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, x.w * x.w)));
    for (int w_ = lanes >> 1; w_ > 0; w_ >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, w_);
    if (i >= C) continue;
    const float rstd = 1.0f / sqrtf(ss / (float)W + eps);
    const float4 c = gs_ld4<bf16>(w + (AFTER ? i % W : i));
    x = make_float4(x.x * rstd * c.x, x.y * rstd * c.y, x.z * rstd * c.z, x.w * rstd * c.w);
    if (AFTER) { x.x *= g[n].x; x.y *= g[n].y; x.z *= g[n].z; x.w *= g[n].w; }
    gs_st4(o + i, x);
  }
}

}  // namespace b200

using namespace b200;

extern "C" int b200_gated_scan(const float* x, int64_t ld, int q_col, int k_col, int v_col, const float* gates, int64_t ld_g,
                               const float* rate, const float* dt_bias, const float* skip, const int32_t* cu_seq,
                               const int32_t* ctx_lens, const int32_t* state_slots, float* S, float* o_raw, int n_seqs, int H,
                               int G, int dk, int dv, int delta, int max_len, void* stream) {
  B200_REQUIRE(n_seqs >= 0 && H > 0 && G > 0 && H % G == 0 && dk > 0 && dv > 0 && dk <= 512,
               "gated_scan: bad shape H=%d G=%d dk=%d dv=%d (dk <= 512)", H, G, dk, dv);
  B200_REQUIRE(((ld | q_col | k_col | v_col) & 3) == 0 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(S)) & 15) == 0,
               "gated_scan: rows, columns and state in whole 16-byte pieces");
  if (n_seqs == 0) return B200_OK;
  const GatedScanArgs a{x, ld, q_col, k_col, v_col, gates, ld_g, rate, dt_bias, skip, cu_seq, ctx_lens, state_slots, S, o_raw, H, G,
                        (dk + 3) & ~3, dv, (dv + 3) & ~3};
  cudaStream_t s = (cudaStream_t)stream;
  return delta ? gated_scan_pick<true>(a, n_seqs, max_len, s) : gated_scan_pick<false>(a, n_seqs, max_len, s);
}

extern "C" int b200_gate_norm(const float* y, const void* proj, int f32, int64_t ld, int z_col, const void* w, void* out,
                              int64_t ldo, int T, int C, int parts, int gate_after, float eps, void* stream) {
  B200_REQUIRE(T >= 0 && C > 0 && parts > 0 && C % parts == 0, "gate_norm: %d channels in %d parts", C, parts);
  if (T == 0) return B200_OK;
  const size_t smem = sizeof(float) * (size_t)C;
  cudaStream_t s = (cudaStream_t)stream;
  auto al = [](const void* p, int n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; };
  const int n = f32 ? 16 : 8;
  const bool vec = (C / parts) % 4 == 0 && ld % 4 == 0 && ldo % 4 == 0 && z_col % 4 == 0 && al(y, 16) && al(proj, n) && al(out, n) && al(w, 8);
  const int W = C / parts, lanes = W / 4;
  if (vec && lanes <= 32 && (lanes & (lanes - 1)) == 0 && C <= kGnThreads * 4 * 8) {
#define B200_GNH(TA, A) gate_norm_heads_kernel<TA, A><<<T, kGnThreads, 0, s>>>(y, (const TA*)proj, ld, z_col, (const bf16*)w, (TA*)out, ldo, C, W, eps)
    if (f32) { if (gate_after) B200_GNH(float, true); else B200_GNH(float, false); }
    else { if (gate_after) B200_GNH(bf16, true); else B200_GNH(bf16, false); }
#undef B200_GNH
    return b200_check_launch("b200_gate_norm");
  }
  B200_REQUIRE(smem <= 48 * 1024, "gate_norm: %d channels exceed the staged row (12288)", C);
#define B200_GN(TA, V, A) \
  gate_norm_kernel<TA, V, A><<<T, kGnThreads, smem, s>>>(y, (const TA*)proj, ld, z_col, (const bf16*)w, (TA*)out, ldo, C, parts, eps)
#define B200_GN2(TA)                                                                                     \
  do {                                                                                                   \
    if (gate_after) { if (vec) B200_GN(TA, true, true); else B200_GN(TA, false, true); }                 \
    else { if (vec) B200_GN(TA, true, false); else B200_GN(TA, false, false); }                          \
  } while (0)
  if (f32) B200_GN2(float);
  else B200_GN2(bf16);
#undef B200_GN2
#undef B200_GN
  return b200_check_launch("b200_gate_norm");
}
