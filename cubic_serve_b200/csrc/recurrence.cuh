// Linear recurrences over the tokens of a request: gated delta rule (delta_rule.cu), gated linear attention and state-space
// duality (linear_recurrence.cu), of any head size, with one decay per head or one per key channel.
//
//   recurrence_prepare_kernel  everything of a token that does not depend on the state, all tokens in parallel: depthwise
//                              causal convolution of any number of taps + SiLU (or none), q, k (unit for the delta rule) and
//                              k . q, step sizes and decays; the last taps - 1 inputs of every channel are the request's
//                              convolution state
//   recurrence_walk_kernel     the recurrence, per (head, segment, slice of value rows), token by token:
//                                  S <- g S;  u = beta v, or beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//   recurrence_step_kernel     the same for segments of one token (decode), with the gated RMS norm of the head's output
//   gated_norm_kernel          that norm as a kernel of its own
//
// S^T q is taken from the decayed state before the write: o = S^T q + (k . q) u, so that all reductions over the key
// channels of a token happen at once.  The state [slot][head][value row][key channel] is fp32 and stays in registers for
// a whole segment; everything is computed in fp32 and what passes between the kernels is fp32, except the value rows,
// which keep the activation type.
#pragma once
#include "launch.cuh"
#include "mma.cuh"
#include "short_conv.cuh"

namespace cb {

__device__ __forceinline__ float gate_of(float z, int sigmoid) { return (sigmoid ? 1.f : z) / (1.f + expf(-z)); }
// ------------------------------------------------------------------ preparation
static constexpr int kPrepRows = 16;       // tokens per warp
static constexpr int kPrepWarps = 4;

// The recurrences of a state S [key channel, value channel] per head:
//   kDelta  gated delta rule: unit q and k, a write of beta (v - S^T k), decays exp(-exp(A_log) softplus(a + dt_bias))
//   kGated  gated linear attention: q times d^-1/2, a write of v, decays sigmoid(a + dt_bias)^rate per key channel
//   kSsd    state-space duality: q and k as convolved, a write of dt v, decays exp(-exp(A_log) dt), dt = softplus(a + dt_bias)
enum Rule : int { kDelta = 0, kGated = 1, kSsd = 2 };

template <typename T>
struct RecPrep {
  ShortConv<T> cv;            // projections (before the convolution, if there is one)
  int q_off, k_off, v_off;    // columns of q [G d], k [G d] and v [H e] among them
  const T* b; int ldb;        // [H] step size logits (kDelta)
  const T* a; int lda;        // decay logits: [H] or [H d]; kSsd: step sizes [H]
  const float* a_log;         // [H] (not kGated)
  const float* dt_bias;       // [H] or [H d]
  float rate;                 // kGated
  float* q;                   // [T, G, ds]
  float* k;                   // [T, G, ds]
  float* kq;                  // [T, G] k . q
  T* v;                       // [T, H, es]
  float2* coef;               // [T, H] {step size, decay per head (1 with channel decays)}
  float* g;                   // [T, H, ds] channel decays or null
  const T* low;               // kGated, bf16: [H d, low_k]: a holds low_rank inner columns of the logits, this makes the logits; or null
  int low_k, low_rank;
  int H, G, d, e, ds, es;
  Segments sg;
};

// 32 channel decays (from channel n0 of head h on) of up to 16 tokens from the inner columns of their low-rank logits (bf16
// models): the second product runs here on the tensor cores, its result stays fp32.  Lane (g, t4) feeds the columns 8 t4 .. + 7 of
// a chunk of 32 to two steps: which column goes to which place of a step is the same for both operands, so 16-byte loads make the
// fragments.
template <typename F>
__device__ __forceinline__ void low_rank_decays(const RecPrep<__nv_bfloat16>& p, int h, int n0, size_t row, int tokens, F decay_of) {
  const int lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  const __nv_bfloat16* w = p.low + static_cast<size_t>(h) * p.d * p.low_k;
  float acc[4][4] = {};
  for (int kc = 0; kc < p.low_rank; kc += 64) {                // the whole warp together; two chunks' loads in flight
    uint4 a[2][2], b[2][4];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int k = kc + 32 * u + 8 * t4;
      const bool there = kc + 32 * u < p.low_rank;             // low_k is a multiple of 32
#pragma unroll
      for (int i = 0; i < 2; ++i)
        a[u][i] = there && g + 8 * i < tokens ? *reinterpret_cast<const uint4*>(p.a + (row + g + 8 * i) * p.lda + k) : make_uint4(0, 0, 0, 0);
#pragma unroll
      for (int j = 0; j < 4; ++j)
        b[u][j] = there && n0 + 8 * j + g < p.d ? *reinterpret_cast<const uint4*>(w + static_cast<size_t>(n0 + 8 * j + g) * p.low_k + k)
                                                : make_uint4(0, 0, 0, 0);
    }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const uint32_t a0[4] = {a[u][0].x, a[u][1].x, a[u][0].y, a[u][1].y}, a1[4] = {a[u][0].z, a[u][1].z, a[u][0].w, a[u][1].w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        mma_bf16(acc[j], a0, b[u][j].x, b[u][j].y);
        mma_bf16(acc[j], a1, b[u][j].z, b[u][j].w);
      }
    }
  }
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int c = n0 + 8 * j + 2 * t4;
    if (c >= p.ds) continue;                                   // ds is a multiple of 4
    const float b0 = c < p.d ? p.dt_bias[h * p.d + c] : 0.f, b1 = c + 1 < p.d ? p.dt_bias[h * p.d + c + 1] : 0.f;
#pragma unroll
    for (int i = 0; i < 2; ++i)
      if (g + 8 * i < tokens)
        *reinterpret_cast<float2*>(p.g + ((row + g + 8 * i) * p.H + h) * p.ds + c) =
            make_float2(c < p.d ? decay_of(acc[j][2 * i] + b0) : 0.f, c + 1 < p.d ? decay_of(acc[j][2 * i + 1] + b1) : 0.f);
  }
}

// A warp per (slot, tile of kPrepRows tokens).  The first G slots are key heads (q and k), then come value channels (64 VP of them
// a slot), step sizes and decays (32 heads a slot) and the channel decays (a head a slot, with low-rank logits 32 channels of one).  NP: channel pairs per lane of a key head
// (d <= 64 NP).  STEP: segments of one token (decode): nothing is read ahead, which leaves registers for more channels at once.
template <bool STEP> constexpr int value_pairs() { return STEP ? 4 : 2; }
template <typename T, int NP, int TAPS, bool STEP, int RULE>
__global__ void __launch_bounds__(32 * kPrepWarps)
recurrence_prepare_kernel(const RecPrep<T> p) {
  using Pair = ConvPair<T, TAPS, RULE == kSsd>;
  constexpr int VP = value_pairs<STEP>();
  const ShortConv<T>& cvp = p.cv;
  const int vslots = (p.H * p.e + 64 * VP - 1) / (64 * VP), cslots = (p.H + 31) / 32;
  pdl_wait();
  pdl_launch_dependents();
  const int slot = blockIdx.x * kPrepWarps + (threadIdx.x >> 5);
  auto low_rank_slot = [&](size_t row, int tokens) {
    if constexpr (RULE == kGated && sizeof(T) == 2) {
      const int chunks = (p.ds + 31) / 32, i = slot - p.G - vslots - cslots;
      if (i < p.H * chunks)
        low_rank_decays(p, i / chunks, i % chunks * 32, row, tokens,
                        [&](float logit) { return exp_of<T>(-p.rate * softplus_of<T>(-logit)); });
    }
  };
  if (RULE == kGated && STEP && p.low && slot >= p.G + vslots + cslots) {
    // decays do not depend on what request a token belongs to: 16 rows of the step at a time
    if ((blockIdx.y & 15) == 0) low_rank_slot(blockIdx.y, min(16, p.sg.num - static_cast<int>(blockIdx.y)));
    return;
  }
  int s, off;
  if (!find_tile(p.sg, kPrepRows, blockIdx.y, s, off)) return;
  const int lane = threadIdx.x & 31;
  if (slot >= p.G + vslots + cslots + (p.g ? p.H * (p.low ? (p.ds + 31) / 32 : 1) : 0)) return;
  const int count = p.sg.count[s], end = min(count, off + kPrepRows);
  const bool fresh = p.sg.pos0[s] == 0;
  const size_t row0 = p.sg.row0[s];
  const T* xr = cvp.x + row0 * cvp.ldx;
  T* st = TAPS < 0 ? nullptr : cvp.state + static_cast<size_t>(p.sg.slot[s]) * (cvp.taps - 1) * cvp.ldw;
  if (slot < p.G) {
    const int qb = p.q_off + slot * p.d, kb = p.k_off + slot * p.d;
    const float scale = RULE == kSsd ? 1.f : 1.f / sqrtf(static_cast<float>(p.d));
    Pair cq[NP], ck[NP];
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      cq[i].begin(cvp, xr, st, fresh, qb, 2 * lane + 64 * i, p.d, off);
      ck[i].begin(cvp, xr, st, fresh, kb, 2 * lane + 64 * i, p.d, off);
    }
    constexpr int AH = STEP ? 1 : NP == 1 ? 8 : NP == 2 ? 4 : 2;  // tokens whose inputs are read at once
    for (int t0 = off; t0 < end; t0 += AH) {
      float2 xq[AH][NP], xk[AH][NP];
#pragma unroll
      for (int u = 0; u < AH; ++u)
#pragma unroll
        for (int i = 0; i < NP; ++i) {
          xq[u][i] = cq[i].ahead(t0 + u, end);
          xk[u][i] = ck[i].ahead(t0 + u, end);
        }
#pragma unroll
      for (int u = 0; u < AH; ++u) {
      const int t = t0 + u;
      if (t >= end) break;
      float2 q[NP], k[NP];
      float qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        q[i] = cq[i].token(t, xq[u][i]);
        k[i] = ck[i].token(t, xk[u][i]);
        if constexpr (RULE == kDelta) {
          qq = fmaf(q[i].x, q[i].x, qq); qq = fmaf(q[i].y, q[i].y, qq);
          kk = fmaf(k[i].x, k[i].x, kk); kk = fmaf(k[i].y, k[i].y, kk);
        }
        qk = fmaf(q[i].x, k[i].x, qk); qk = fmaf(q[i].y, k[i].y, qk);
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        if constexpr (RULE == kDelta) {
          qq += __shfl_xor_sync(0xffffffffu, qq, o);
          kk += __shfl_xor_sync(0xffffffffu, kk, o);
        }
        qk += __shfl_xor_sync(0xffffffffu, qk, o);
      }
      const float qi = RULE == kDelta ? 1.f / sqrtf(qq + 1e-6f) * scale : scale, ki = RULE == kDelta ? 1.f / sqrtf(kk + 1e-6f) : 1.f;
      const size_t o = ((row0 + t) * p.G + slot) * p.ds;
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        const int c = 2 * lane + 64 * i;             // columns [d, ds) get zeros
        if (c < p.ds) {
          *reinterpret_cast<float2*>(p.q + o + c) = make_float2(q[i].x * qi, q[i].y * qi);
          *reinterpret_cast<float2*>(p.k + o + c) = make_float2(k[i].x * ki, k[i].y * ki);
        }
      }
      if (lane == 0) p.kq[(row0 + t) * p.G + slot] = qk * qi * ki;
      }
    }
    if (off == 0) {
      if constexpr (TAPS > 0) {
#pragma unroll
        for (int i = 0; i < NP; ++i) {
          cq[i].save(st, count, end == count);
          ck[i].save(st, count, end == count);
        }
      } else if constexpr (TAPS == 0) {
        conv_state(cvp, xr, st, fresh, count, qb, p.d);
        conv_state(cvp, xr, st, fresh, count, kb, p.d);
      }
    }
  } else if (slot < p.G + vslots) {
    // 64 VP neighbouring value channels, whatever heads they belong to
    const int c0 = (slot - p.G) * 64 * VP, lim = p.H * p.e;
    constexpr int AH = STEP ? 1 : 4;
    Pair cv[VP];
    int at0[VP], at1[VP];                                      // places of the pair's channels in a row of v
#pragma unroll
    for (int i = 0; i < VP; ++i) {
      const int c = c0 + 2 * lane + 64 * i;
      cv[i].begin(cvp, xr, st, fresh, p.v_off, c, lim, off);
      at0[i] = p.es == p.e ? c : c / p.e * p.es + c % p.e;
      at1[i] = p.es == p.e || (p.e & 1) == 0 ? at0[i] + 1 : (c + 1) / p.e * p.es + (c + 1) % p.e;
    }
    for (int t0 = off; t0 < end; t0 += AH) {
      float2 xv[AH][VP];
#pragma unroll
      for (int u = 0; u < AH; ++u)
#pragma unroll
        for (int i = 0; i < VP; ++i) xv[u][i] = cv[i].ahead(t0 + u, end);
#pragma unroll
      for (int u = 0; u < AH; ++u) {
        const int t = t0 + u;
        if (t >= end) break;
        T* dst = p.v + (row0 + t) * p.H * p.es;
#pragma unroll
        for (int i = 0; i < VP; ++i) {
          const float2 v = cv[i].token(t, xv[u][i]);
          if (!cv[i].ok) continue;
          if constexpr (Pair::ODD) {
            dst[at0[i]] = from_f<T>(v.x);
            if (cv[i].ok1) dst[at1[i]] = from_f<T>(v.y);
          } else if constexpr (sizeof(T) == 2) {
            *reinterpret_cast<uint32_t*>(dst + at0[i]) = pack_bf16x2(v.x, v.y);
          } else {
            *reinterpret_cast<float2*>(dst + at0[i]) = v;
          }
        }
      }
    }
    if constexpr (TAPS > 0) {
      if (off == 0) {
#pragma unroll
        for (int i = 0; i < VP; ++i) cv[i].save(st, count, end == count);
      }
    } else if constexpr (TAPS == 0) {
      if (off == 0) conv_state(cvp, xr, st, fresh, count, p.v_off + c0, min(64 * VP, lim - c0));
    }
  } else if (slot < p.G + vslots + cslots) {
    // step sizes and decays of 32 heads
    const int h = (slot - p.G - vslots) * 32 + lane;
    if (h >= p.H) return;
    const float rate = RULE == kGated ? 0.f : -expf(p.a_log[h]);
    const float bias = RULE == kGated || p.g ? 0.f : p.dt_bias[h];
    for (int t = off; t < end; ++t) {
      const size_t r = row0 + t;
      float beta = 1.f, decay = 1.f;
      if constexpr (RULE == kSsd) {
        beta = softplus_of<float>(to_f(p.a[r * p.lda + h]) + bias);
        decay = expf(rate * beta);
      } else if constexpr (RULE == kDelta) {
        beta = 1.f / (1.f + expf(-to_f(p.b[r * p.ldb + h])));
        if (!p.g) decay = expf(rate * softplus_of<float>(to_f(p.a[r * p.lda + h]) + bias));
      }
      p.coef[r * p.H + h] = make_float2(beta, decay);
    }
  } else if (RULE == kGated && p.low) {
    low_rank_slot(row0 + off, end - off);
  } else if constexpr (RULE != kSsd) {
    const int h = slot - p.G - vslots - cslots;
    // sigmoid(x)^rate = exp(-rate softplus(-x))
    const float rate = RULE == kGated ? -p.rate : -expf(p.a_log[h]), sign = RULE == kGated ? -1.f : 1.f;
    auto decay_of = [&](float logit) { return exp_of<T>(rate * softplus_of<T>(sign * logit)); };
    constexpr int AH = STEP ? 1 : 4;
    for (int c0 = lane; c0 < p.ds; c0 += 128) {                // four channels x AH tokens read at once
      float dt[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) dt[i] = c0 + 32 * i < p.d ? p.dt_bias[h * p.d + c0 + 32 * i] : 0.f;
      float* dst = p.g + (row0 * p.H + h) * p.ds + c0;
      const T* src = p.a + row0 * p.lda + h * p.d + c0;
      for (int t0 = off; t0 < end; t0 += AH) {
        float v[AH][4];
#pragma unroll
        for (int u = 0; u < AH; ++u)
#pragma unroll
          for (int i = 0; i < 4; ++i)
            v[u][i] = c0 + 32 * i < p.d && t0 + u < end ? to_f(src[static_cast<size_t>(t0 + u) * p.lda + 32 * i]) : 0.f;
#pragma unroll
        for (int u = 0; u < AH; ++u)
#pragma unroll
          for (int i = 0; i < 4; ++i)
            if (t0 + u < end && c0 + 32 * i < p.ds)
              dst[static_cast<size_t>(t0 + u) * p.H * p.ds + 32 * i] = c0 + 32 * i < p.d ? decay_of(v[u][i] + dt[i]) : 0.f;
      }
    }
  }
}

// ------------------------------------------------------------------ recurrence
template <typename T>
struct RecWalk {
  const float* q; const float* k; const float* kq;
  const T* v; const float2* coef; const float* g;     // as written by the preparation
  const float* skip;                                  // [H] value rows pass to the output times this, or null
  const T* z; int ldz;                                // output gate [H e] (recurrence_step_kernel)
  const float* norm_w;                                // [e]
  float* state;                                       // [slots, H, e, ds]
  T* out; int ldo;                                    // [H e]
  float* raw;                                         // fp32 [T, H e]: outputs before the norm, or null
  int H, G, d, e, ds, es;
  float eps;
  int sigmoid_gate;                                   // output gate sigmoid(z) instead of silu(z)
  Segments sg;
};

// KD: key channels covered by a row's lanes (d <= KD).  LPR = KD / 16 lanes share a state row, lane l holds the float4
// chunks l + LPR c (c < 4); a thread holds RPT rows.
template <int KD> struct RecShape {
  static constexpr int LPR = KD / 16;
  static constexpr int NB = KD <= 128 ? 16 : 8;       // tokens staged at a time
};

template <int LPR, int RPT>
__device__ __forceinline__ void load_state(const float* sp, int ds, int e, int v_first, int v_step, int l, bool use, float2 (&S)[RPT][8]) {
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int v = v_first + i * v_step;
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const int col = 4 * (l + LPR * c);
      float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
      if (use && v < e && col < ds) t = *reinterpret_cast<const float4*>(sp + static_cast<size_t>(v) * ds + col);
      S[i][2 * c] = make_float2(t.x, t.y);
      S[i][2 * c + 1] = make_float2(t.z, t.w);
    }
  }
}
template <int LPR, int RPT>
__device__ __forceinline__ void store_state(float* sp, int ds, int e, int v_first, int v_step, int l, const float2 (&S)[RPT][8]) {
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int v = v_first + i * v_step;
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const int col = 4 * (l + LPR * c);
      if (v < e && col < ds)
        *reinterpret_cast<float4*>(sp + static_cast<size_t>(v) * ds + col) =
            make_float4(S[i][2 * c].x, S[i][2 * c].y, S[i][2 * c + 1].x, S[i][2 * c + 1].y);
    }
  }
}

// One token: decays the state, updates it with (k, v) and returns the output of ONE of the thread's rows: row l of the
// thread for its row's lanes l < RPT (a lane l >= RPT repeats row l % RPT).  `get(which, c)` yields the float4 chunk c of q (0), k (1), g (2).
// DELTA: the write is beta (v - S^T k), else beta v.
template <int LPR, int RPT, bool CHANNEL, bool DELTA, typename Get>
__device__ __forceinline__ float recurrence_token(float2 (&S)[RPT][8], Get get, float beta, float decay, float kq, float skip,
                                                  const float (&va)[RPT]) {
  float o[RPT];
  float2 k2[8], aa[RPT], bb[RPT], a2[RPT], b2[RPT];   // two chains per sum
  const float2 g1 = make_float2(decay, decay);
#pragma unroll
  for (int i = 0; i < RPT; ++i) aa[i] = bb[i] = a2[i] = b2[i] = make_float2(0.f, 0.f);
#pragma unroll
  for (int c = 0; c < 4; ++c) {
    const float4 q4 = get(0, c), k4 = get(1, c);
    float2 ga = g1, gb = g1;
    if constexpr (CHANNEL) {
      const float4 g4 = get(2, c);
      ga = make_float2(g4.x, g4.y);
      gb = make_float2(g4.z, g4.w);
    }
    k2[2 * c] = make_float2(k4.x, k4.y);
    k2[2 * c + 1] = make_float2(k4.z, k4.w);
    const float2 q0 = make_float2(q4.x, q4.y), q1 = make_float2(q4.z, q4.w);
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      S[i][2 * c] = mul2(S[i][2 * c], ga);
      S[i][2 * c + 1] = mul2(S[i][2 * c + 1], gb);
      bb[i] = fma2(S[i][2 * c], q0, bb[i]);
      if constexpr (RPT == 1) b2[i] = fma2(S[i][2 * c + 1], q1, b2[i]);
      else bb[i] = fma2(S[i][2 * c + 1], q1, bb[i]);
      if constexpr (DELTA) {
        aa[i] = fma2(S[i][2 * c], k2[2 * c], aa[i]);
        if constexpr (RPT == 1) a2[i] = fma2(S[i][2 * c + 1], k2[2 * c + 1], a2[i]);
        else aa[i] = fma2(S[i][2 * c + 1], k2[2 * c + 1], aa[i]);
      }
    }
  }
  float sa[RPT];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    if constexpr (RPT == 1) {
      aa[i].x += a2[i].x; aa[i].y += a2[i].y;
      bb[i].x += b2[i].x; bb[i].y += b2[i].y;
    }
    sa[i] = aa[i].x + aa[i].y;
    o[i] = bb[i].x + bb[i].y;
  }
  if constexpr (RPT == 4 && LPR >= 4) {
    // the four rows' sums are dealt over the lanes while they are added (2 + 1 exchanges instead of 4 per step), then
    // spread back: lane l ends with the totals of row l & 3
    const int l = threadIdx.x % LPR;
    const bool b0 = l & 1, b1 = l & 2;
    const float o01 = (b0 ? o[1] : o[0]) + __shfl_xor_sync(0xffffffffu, b0 ? o[0] : o[1], 1);
    const float o23 = (b0 ? o[3] : o[2]) + __shfl_xor_sync(0xffffffffu, b0 ? o[2] : o[3], 1);
    float r = (b1 ? o23 : o01) + __shfl_xor_sync(0xffffffffu, b1 ? o01 : o23, 2);
#pragma unroll
    for (int sh = 4; sh < LPR; sh <<= 1) r += __shfl_xor_sync(0xffffffffu, r, sh);
    if constexpr (DELTA) {
      const float a01 = (b0 ? sa[1] : sa[0]) + __shfl_xor_sync(0xffffffffu, b0 ? sa[0] : sa[1], 1);
      const float a23 = (b0 ? sa[3] : sa[2]) + __shfl_xor_sync(0xffffffffu, b0 ? sa[2] : sa[3], 1);
      float a = (b1 ? a23 : a01) + __shfl_xor_sync(0xffffffffu, b1 ? a01 : a23, 2);
#pragma unroll
      for (int sh = 4; sh < LPR; sh <<= 1) a += __shfl_xor_sync(0xffffffffu, a, sh);
#pragma unroll
      for (int i = 0; i < 4; ++i) sa[i] = __shfl_sync(0xffffffffu, a, i, 4);
    }
    o[0] = r;                                        // the total of row l & 3: the caller's lane l stores that row
  } else {
#pragma unroll
    for (int sh = 1; sh < LPR; sh <<= 1)
#pragma unroll
      for (int i = 0; i < RPT; ++i) {
        if constexpr (DELTA) sa[i] += __shfl_xor_sync(0xffffffffu, sa[i], sh);
        o[i] += __shfl_xor_sync(0xffffffffu, o[i], sh);
      }
  }
  float mine = 0.f, direct = 0.f;
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const float u = DELTA ? beta * (va[i] - sa[i]) : beta * va[i];
    if (RPT == 1 || (static_cast<int>(threadIdx.x) & 3) == i) {
      mine = u;
      direct = va[i];
    }
    const float2 u2 = make_float2(u, u);
#pragma unroll
    for (int c = 0; c < 8; ++c) S[i][c] = fma2(k2[c], u2, S[i][c]);
  }
  const float out = fmaf(kq, mine, o[0]);
  return DELTA ? out : fmaf(skip, direct, out);
}

template <int B>
__device__ __forceinline__ void cp_async(void* dst, const void* src) {
  if constexpr (B == 16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
  else asm volatile("cp.async.ca.shared.global [%0], [%1], %2;" ::"r"(smem_u32(dst)), "l"(src), "n"(B) : "memory");
}

// Segments of many tokens: NB tokens' operands arrive by cp.async while the previous NB are walked; one barrier per NB
// tokens.  Outputs leave through shared memory, before the norm.  With one row per thread (few blocks: the chain of tokens
// is what takes the time) kHelpers more threads do the copies in and out.
static constexpr int kHelpers = 128;
template <int RPT> constexpr int helper_threads() { return RPT == 1 ? kHelpers : 0; }

template <typename T, int KD, int RPT, bool CHANNEL, bool DELTA>
__global__ void __launch_bounds__(256 + helper_threads<RPT>(), RPT == 1 ? 1 : 2)
recurrence_walk_kernel(const RecWalk<T> p) {
  constexpr int LPR = RecShape<KD>::LPR, NB = RecShape<KD>::NB, OPS = CHANNEL ? 3 : 2;
  extern __shared__ __align__(16) float sm[];
  pdl_wait();
  pdl_launch_dependents();
  const int head = blockIdx.x, s = blockIdx.y;
  const int n = p.sg.count[s];
  if (n <= 0) return;
  constexpr int HELP = helper_threads<RPT>();
  const int row_threads = blockDim.x - HELP;
  const int VT = row_threads / LPR * RPT;             // value rows of this block
  const int v0 = blockIdx.z * VT, e_here = min(VT, p.e - v0);
  const int es = p.es;
  // per buffer: operands [OPS][NB][KD], coefficients [NB] float4, value rows [NB][es] (the whole head's, T)
  const int buf_floats = NB * (OPS * KD + 4) + NB * es * static_cast<int>(sizeof(T)) / 4;
  float* const obuf = sm + 2 * buf_floats;            // [2][NB][VT]
  const int tid = threadIdx.x;
  const int l = tid % LPR, grp = tid / LPR, ngrp = row_threads / LPR;
  const bool rower = tid < row_threads, copier = HELP == 0 || !rower;
  const size_t row0 = p.sg.row0[s];
  const int hq = head / (p.H / p.G);
  const float skip = !DELTA && p.skip ? p.skip[head] : 0.f;
  float* sp = p.state + (static_cast<size_t>(p.sg.slot[s]) * p.H + head) * p.e * p.ds;
  float2 S[RPT][8];
  load_state<LPR, RPT>(sp, p.ds, p.e, v0 + grp, ngrp, l, rower && p.sg.pos0[s] != 0, S);

  auto coefs = [&](int b) { return sm + b * buf_floats + NB * OPS * KD; };
  auto values = [&](int b) { return reinterpret_cast<T*>(sm + b * buf_floats + NB * (OPS * KD + 4)); };
  const int chunks = p.ds / 4, vchunks = es * static_cast<int>(sizeof(T)) / 16;
  const int warp = (tid - (HELP ? row_threads : 0)) >> 5, lane = tid & 31, warps = (HELP ? HELP : row_threads) >> 5;
  auto fetch = [&](int blk) {                         // a warp per token row
    const int t0 = blk * NB, nb = min(NB, n - t0), b = blk & 1;
    float* buf = sm + b * buf_floats;
    T* vs = values(b);
    for (int j = warp; j < nb; j += warps) {
      const size_t r = row0 + t0 + j;
      const float* qr = p.q + (r * p.G + hq) * p.ds;
      const float* kr = p.k + (r * p.G + hq) * p.ds;
#pragma unroll
      for (int i = 0; i < (KD + 127) / 128; ++i) {
        const int c = lane + 32 * i;
        if (c < chunks) {
          cp_async<16>(buf + j * KD + c * 4, qr + c * 4);
          cp_async<16>(buf + (NB + j) * KD + c * 4, kr + c * 4);
          if constexpr (CHANNEL) cp_async<16>(buf + (2 * NB + j) * KD + c * 4, p.g + (r * p.H + head) * p.ds + c * 4);
        }
      }
      const T* vr = p.v + (r * p.H + head) * es;
      for (int c = lane; c < vchunks; c += 32) {
        constexpr int E = 16 / static_cast<int>(sizeof(T));
        cp_async<16>(vs + j * es + c * E, vr + c * E);
      }
      if (lane == 0) cp_async<8>(coefs(b) + j * 4, p.coef + r * p.H + head);
      if (lane == 1) cp_async<4>(coefs(b) + j * 4 + 2, p.kq + r * p.G + hq);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // columns [ds, KD) of the operand rows are never fetched: zero once
  if (p.ds < KD)
    for (int i = tid; i < 2 * OPS * NB * (KD - p.ds); i += blockDim.x) {
      const int rowi = i / (KD - p.ds), c = p.ds + i % (KD - p.ds);
      (sm + (rowi / (OPS * NB)) * buf_floats)[(rowi % (OPS * NB)) * KD + c] = 0.f;
    }
  auto put = [&](int blk) {                           // outputs of block blk to memory
    const int t0 = blk * NB, nb = min(NB, n - t0);
    const float* ob = obuf + (blk & 1) * NB * VT;
    for (int j = warp; j < nb; j += warps) {
      float* dst = p.raw + (row0 + t0 + j) * (static_cast<size_t>(p.H) * p.e) + head * p.e + v0;
      for (int v = lane; v < e_here; v += 32) dst[v] = ob[j * VT + v];
    }
  };
  const int blocks = (n + NB - 1) / NB;
  if (copier) fetch(0);
  for (int blk = 0; blk < blocks; ++blk) {
    const int b = blk & 1, nb = min(NB, n - blk * NB);
    if (copier) asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();                                  // operands of blk are here; everybody has left blk - 1
    if (copier) {
      if (blk + 1 < blocks) fetch(blk + 1);
      if (blk > 0) put(blk - 1);
    }
    if (HELP && !rower) continue;
    const float* buf = sm + b * buf_floats;
    const float* cf = coefs(b);
    const T* vs = values(b) + v0 + grp;
    float* ob = obuf + b * NB * VT + grp;
#pragma unroll (RPT == 1 ? 4 : 1)
    for (int j = 0; j < nb; ++j) {
      const float4 co = *reinterpret_cast<const float4*>(cf + j * 4);
      float va[RPT];
#pragma unroll
      for (int i = 0; i < RPT; ++i) va[i] = v0 + grp + i * ngrp < p.e ? to_f(vs[j * es + i * ngrp]) : 0.f;
      const float o = recurrence_token<LPR, RPT, CHANNEL, DELTA>(
          S, [&](int w, int c) { return *reinterpret_cast<const float4*>(buf + (w * NB + j) * KD + 4 * (l + LPR * c)); },
          co.x, co.y, co.z, skip, va);
      if (l < RPT) ob[j * VT + l * ngrp] = o;
    }
  }
  __syncthreads();
  if (copier) put(blocks - 1);
  if (rower) store_state<LPR, RPT>(sp, p.ds, p.e, v0 + grp, ngrp, l, S);
}

// Segments of one token.  The state's loads go out first; the operands are a few cached rows.
template <typename T, int KD, int RPT, bool CHANNEL, bool DELTA>
__global__ void __launch_bounds__(256, 2)
recurrence_step_kernel(const RecWalk<T> p) {
  constexpr int LPR = RecShape<KD>::LPR;
  extern __shared__ __align__(16) float sm[];         // [VT]
  __shared__ float red[8];
  const int head = blockIdx.x, s = blockIdx.y, tid = threadIdx.x;
  const int VT = blockDim.x / LPR * RPT, v0 = blockIdx.z * VT;
  const int l = tid % LPR, grp = tid / LPR, ngrp = blockDim.x / LPR;
  pdl_wait();
  pdl_launch_dependents();
  if (p.sg.count[s] <= 0) return;
  const size_t r = p.sg.row0[s];
  const int hq = head / (p.H / p.G);
  const float skip = !DELTA && p.skip ? p.skip[head] : 0.f;
  float* sp = p.state + (static_cast<size_t>(p.sg.slot[s]) * p.H + head) * p.e * p.ds;
  float2 S[RPT][8];
  load_state<LPR, RPT>(sp, p.ds, p.e, v0 + grp, ngrp, l, p.sg.pos0[s] != 0, S);
  const float* qr = p.q + (r * p.G + hq) * p.ds;
  const float* kr = p.k + (r * p.G + hq) * p.ds;
  const float* gr = CHANNEL ? p.g + (r * p.H + head) * p.ds : nullptr;
  const float2 co = p.coef[r * p.H + head];
  const float kq = p.kq[r * p.G + hq];
  float va[RPT];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int v = v0 + grp + i * ngrp;
    va[i] = v < p.e ? to_f(p.v[(r * p.H + head) * p.es + v]) : 0.f;
  }
  const float o = recurrence_token<LPR, RPT, CHANNEL, DELTA>(
      S,
      [&](int w, int c) {
        const int col = 4 * (l + LPR * c);
        const float* src = w == 0 ? qr : w == 1 ? kr : gr;
        return col < p.ds ? *reinterpret_cast<const float4*>(src + col) : make_float4(0.f, 0.f, 0.f, 0.f);
      },
      co.x, co.y, kq, skip, va);
  store_state<LPR, RPT>(sp, p.ds, p.e, v0 + grp, ngrp, l, S);
  const int v_mine = v0 + grp + l * ngrp;              // the row this lane has the output of
  const bool has = l < RPT && v_mine < p.e;
  if (p.raw) {
    if (has) p.raw[(r * p.H + head) * p.e + v_mine] = o;
    return;
  }
  // gated norm: the whole head is in this block
  if (has) sm[v_mine] = o;
  float ss = has ? o * o : 0.f;
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  ss = 0.f;
  for (int w = 0; w < static_cast<int>(blockDim.x >> 5); ++w) ss += red[w];
  const float inv = 1.f / sqrtf(ss / static_cast<float>(p.e) + p.eps);
  for (int v = tid; v < p.e; v += blockDim.x)
    p.out[r * p.ldo + head * p.e + v] =
        from_f<T>(sm[v] * inv * p.norm_w[v] * gate_of(to_f(p.z[r * p.ldz + head * p.e + v]), p.sigmoid_gate));
}

// out = raw / rms(raw) * norm_w * gate(z) per (token, head); a warp each.
template <typename T>
__global__ void __launch_bounds__(256)
gated_norm_kernel(const float* __restrict__ raw, const T* __restrict__ z, int ldz, const float* __restrict__ w,
                  T* __restrict__ out, int ldo, int rows, int H, int e, float eps, int sigmoid_gate) {
  pdl_wait();
  pdl_launch_dependents();
  const long long item = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (item >= static_cast<long long>(rows) * H) return;
  const size_t t = static_cast<size_t>(item / H);
  const int h = static_cast<int>(item % H);
  const float* o = raw + static_cast<size_t>(item) * e;
  const T* zr = z + t * ldz + h * e;
  T* dst = out + t * ldo + h * e;
  float v[8], g[8], ss = 0.f;                        // up to 256 columns in registers
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int c = lane + 32 * i;
    v[i] = c < e ? o[c] : 0.f;
    g[i] = c < e ? to_f(zr[c]) : 0.f;
    ss = fmaf(v[i], v[i], ss);
  }
  for (int c = lane + 256; c < e; c += 32) ss = fmaf(o[c], o[c], ss);
  const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(e) + eps);
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int c = lane + 32 * i;
    if (c < e) dst[c] = from_f<T>(v[i] * inv * w[c] * gate_of(g[i], sigmoid_gate));
  }
  for (int c = lane + 256; c < e; c += 32) dst[c] = from_f<T>(o[c] * inv * w[c] * gate_of(to_f(zr[c]), sigmoid_gate));
}

// ------------------------------------------------------------------ host
template <typename T, int KD, int RPT, bool CHANNEL, bool DELTA, bool STEP>
static int recurrence_go(const RecWalk<T>& p, int threads, int vtiles, cudaStream_t st) {
  const int VT = threads / RecShape<KD>::LPR * RPT;
  const dim3 grid(p.H, p.sg.num, vtiles);
  if constexpr (STEP) {
    return static_cast<int>(launch(recurrence_step_kernel<T, KD, RPT, CHANNEL, DELTA>, grid, dim3(threads), sizeof(float) * VT, st, p));
  } else {
    constexpr int NB = RecShape<KD>::NB;
    const size_t smem = 2 * (sizeof(float) * NB * ((CHANNEL ? 3 : 2) * KD + 4 + VT) + sizeof(T) * NB * p.es);
    auto kernel = recurrence_walk_kernel<T, KD, RPT, CHANNEL, DELTA>;
    static bool configured[64] = {};     // per device
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -18;
    if (!configured[dev]) {
      const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
      if (e != cudaSuccess) return static_cast<int>(e);
      configured[dev] = true;
    }
    if (smem > 200 * 1024) return -14;
    return static_cast<int>(launch(kernel, grid, dim3(threads + helper_threads<RPT>()), smem, st, p));
  }
}

// `p.norm_w` null: the outputs leave as they are, in `raw`.
template <typename T, int KD, bool DELTA>
static int recurrence_kd(RecWalk<T> p, bool channel, bool step, int tokens, float* raw, cudaStream_t st) {
  constexpr int LPR = RecShape<KD>::LPR;
  // four rows per thread amortise the operand loads; one row per thread spreads a head over more blocks when the step
  // has too few (head, request) pairs to fill the device
  const int max1 = 256 / LPR, max4 = max1 * 4;
  const bool spread = !step && static_cast<long long>(p.H) * p.sg.num < 74;
  const int rpt = (spread || p.e <= max1 / 2) ? 1 : 4;
  int max_rows = rpt == 4 ? max4 : max1;
  if (spread) {
    // a head over as many blocks as still give every block an SM of its own
    const int warp_rows = 32 / LPR, blocks = 148 / (p.H * p.sg.num);
    const int rows = ((p.e + blocks - 1) / blocks + warp_rows - 1) / warp_rows * warp_rows;
    max_rows = rows < 2 * warp_rows ? 2 * warp_rows : rows > max1 ? max1 : rows;
  }
  const int parts = (p.e + max_rows - 1) / max_rows;
  const int rows = (p.e + parts - 1) / parts;
  const int threads = ((rows + rpt - 1) / rpt * LPR + 31) / 32 * 32;
  const int vt = threads / LPR * rpt;
  const int vtiles = (p.e + vt - 1) / vt;
  const bool apart = !step || vtiles > 1 || !p.norm_w;       // the norm, if any, runs as a kernel of its own
  p.raw = apart ? raw : nullptr;
  if (apart && !raw) return -13;
  int rc;
  if (step) {
    if (rpt == 4) rc = channel ? recurrence_go<T, KD, 4, true, DELTA, true>(p, threads, vtiles, st) : recurrence_go<T, KD, 4, false, DELTA, true>(p, threads, vtiles, st);
    else rc = channel ? recurrence_go<T, KD, 1, true, DELTA, true>(p, threads, vtiles, st) : recurrence_go<T, KD, 1, false, DELTA, true>(p, threads, vtiles, st);
  } else if (rpt == 4) {
    rc = channel ? recurrence_go<T, KD, 4, true, DELTA, false>(p, threads, vtiles, st) : recurrence_go<T, KD, 4, false, DELTA, false>(p, threads, vtiles, st);
  } else {
    rc = channel ? recurrence_go<T, KD, 1, true, DELTA, false>(p, threads, vtiles, st) : recurrence_go<T, KD, 1, false, DELTA, false>(p, threads, vtiles, st);
  }
  if (rc || !apart || !p.norm_w) return rc;
  const long long items = static_cast<long long>(tokens) * p.H;
  return static_cast<int>(launch(gated_norm_kernel<T>, dim3(static_cast<unsigned>((items + 7) / 8)), dim3(256), 0, st,
                                 static_cast<const float*>(raw), p.z, p.ldz, p.norm_w, p.out, p.ldo, tokens, p.H, p.e, p.eps,
                                 p.sigmoid_gate));
}

}  // namespace cb

extern "C" {

// Operands of the preparation and of the recurrence (RecPrep, RecWalk); `f32`: activations and convolution state are fp32.
struct CbRecPrep {
  const void* x; int ldx;
  const void* w;
  const void* bias; int ldw, taps;                   // taps 0: no convolution
  void* state;
  int q_off, k_off, v_off;
  const void* b; int ldb;
  const void* a; int lda;
  const void* a_log;
  const void* dt_bias;
  float rate;
  void* q;
  void* k;
  void* kq;
  void* v;
  void* coef;
  void* g;
  const void* low; int low_k, low_rank;
  int H, G, d, e, ds, es, tokens, f32;
};

struct CbRecWalk {
  const void* q;
  const void* k;
  const void* kq;
  const void* v;
  const void* coef;
  const void* g;
  const void* skip;
  const void* z; int ldz;
  const void* norm_w;
  void* state;
  void* out; int ldo;
  void* raw;
  int H, G, d, e, ds, es;
  float eps;
  int sigmoid_gate, decode, tokens, f32;
};

}  // extern "C"

namespace cb {

template <typename T>
static RecPrep<T> rec_prep(const CbRecPrep* a, const CbSegments* seg) {
  RecPrep<T> p;
  p.cv.x = static_cast<const T*>(a->x); p.cv.ldx = a->ldx;
  p.cv.w = static_cast<const float*>(a->w); p.cv.bias = static_cast<const float*>(a->bias);
  p.cv.ldw = a->ldw; p.cv.taps = a->taps;
  p.cv.state = static_cast<T*>(a->state);
  p.q_off = a->q_off; p.k_off = a->k_off; p.v_off = a->v_off;
  p.b = static_cast<const T*>(a->b); p.ldb = a->ldb;
  p.a = static_cast<const T*>(a->a); p.lda = a->lda;
  p.a_log = static_cast<const float*>(a->a_log);
  p.dt_bias = static_cast<const float*>(a->dt_bias);
  p.rate = a->rate;
  p.q = static_cast<float*>(a->q); p.k = static_cast<float*>(a->k); p.kq = static_cast<float*>(a->kq);
  p.v = static_cast<T*>(a->v);
  p.coef = static_cast<float2*>(a->coef);
  p.g = static_cast<float*>(a->g);
  p.low = static_cast<const T*>(a->low); p.low_k = a->low_k; p.low_rank = a->low_rank;
  p.H = a->H; p.G = a->G; p.d = a->d; p.e = a->e; p.ds = a->ds; p.es = a->es;
  p.sg = make_segments(seg, a->tokens);
  return p;
}

template <typename T>
static RecWalk<T> rec_walk(const CbRecWalk* a, const CbSegments* seg) {
  RecWalk<T> p;
  p.q = static_cast<const float*>(a->q); p.k = static_cast<const float*>(a->k); p.kq = static_cast<const float*>(a->kq);
  p.v = static_cast<const T*>(a->v);
  p.coef = static_cast<const float2*>(a->coef);
  p.g = static_cast<const float*>(a->g);
  p.skip = static_cast<const float*>(a->skip);
  p.z = static_cast<const T*>(a->z); p.ldz = a->ldz;
  p.norm_w = static_cast<const float*>(a->norm_w);
  p.state = static_cast<float*>(a->state);
  p.out = static_cast<T*>(a->out); p.ldo = a->ldo;
  p.raw = nullptr;
  p.H = a->H; p.G = a->G; p.d = a->d; p.e = a->e; p.ds = a->ds; p.es = a->es;
  p.eps = a->eps; p.sigmoid_gate = a->sigmoid_gate;
  p.sg = make_segments(seg, a->tokens);
  return p;
}

// The preparation kernel of key width NP * 64 for every supported tap count of the rule.
template <typename T, int NP, int TAPS, int RULE>
static int prep_go(const RecPrep<T>& p, int tiles, cudaStream_t st) {
  auto go = [&](auto kernel, int vp) {
    const int slots = p.G + (p.H * p.e + 64 * vp - 1) / (64 * vp) + (p.H + 31) / 32 + (p.g ? p.H * (p.low ? (p.ds + 31) / 32 : 1) : 0);
    return static_cast<int>(launch(kernel, dim3((slots + kPrepWarps - 1) / kPrepWarps, tiles), dim3(32 * kPrepWarps), 0, st, p));
  };
  if (p.sg.single) return go(recurrence_prepare_kernel<T, NP, TAPS, true, RULE>, value_pairs<true>());
  return go(recurrence_prepare_kernel<T, NP, TAPS, false, RULE>, value_pairs<false>());
}
template <typename T, int NP, int RULE>
static int prep_taps(const RecPrep<T>& p, int tiles, cudaStream_t st) {
  const bool even = ((p.d | p.e | p.q_off | p.k_off | p.v_off) & 1) == 0;
  if constexpr (RULE == kGated) {
    return even ? prep_go<T, NP, kPlain, RULE>(p, tiles, st) : prep_go<T, NP, kPlainOdd, RULE>(p, tiles, st);
  } else {
    if (!even) return prep_go<T, NP, 0, RULE>(p, tiles, st);
    if constexpr (NP <= 2) {
      if (p.cv.taps == 2) return prep_go<T, NP, 2, RULE>(p, tiles, st);
      if (p.cv.taps == 3) return prep_go<T, NP, 3, RULE>(p, tiles, st);
    }
    return p.cv.taps == 4 ? prep_go<T, NP, 4, RULE>(p, tiles, st) : prep_go<T, NP, 0, RULE>(p, tiles, st);
  }
}
template <typename T, int RULE>
static int prep_typed(const CbRecPrep* a, const CbSegments* seg, cudaStream_t st) {
  const RecPrep<T> p = rec_prep<T>(a, seg);
  const int tiles = max_tiles(a->tokens, seg->num, kPrepRows);
  if (tiles > 65535) return -11;
  if (a->d <= 64) return prep_taps<T, 1, RULE>(p, tiles, st);
  if (a->d <= 128) return prep_taps<T, 2, RULE>(p, tiles, st);
  return prep_taps<T, 4, RULE>(p, tiles, st);
}

template <typename T, bool DELTA>
static int walk_typed(const CbRecWalk* a, const CbSegments* seg, cudaStream_t st) {
  const RecWalk<T> p = rec_walk<T>(a, seg);
  const bool channel = a->g != nullptr, step = a->decode != 0;
  float* raw = static_cast<float*>(a->raw);
  if (a->d <= 64) return recurrence_kd<T, 64, DELTA>(p, channel, step, a->tokens, raw, st);
  if (a->d <= 128) return recurrence_kd<T, 128, DELTA>(p, channel, step, a->tokens, raw, st);
  return recurrence_kd<T, 256, DELTA>(p, channel, step, a->tokens, raw, st);
}

static inline bool recurrence_sizes_ok(int H, int G, int d, int e, int ds, int es, const CbSegments* seg) {
  return H > 0 && G > 0 && (H % G) == 0 && d > 0 && d <= 256 && e > 0 && ds >= d && (ds & 3) == 0 && es >= e && (es & 7) == 0 &&
         seg->num <= 65535;
}
// `ldw` (channels of a weight row and of a state row) and `ldx` are even.
static inline bool convolution_ok(const CbRecPrep* a) {
  return a->taps >= 1 && a->taps <= kPrepRows && (a->ldx & 1) == 0 && (a->ldw & 1) == 0 && a->ldw >= 2 * a->G * a->d + a->H * a->e;
}

}  // namespace cb
