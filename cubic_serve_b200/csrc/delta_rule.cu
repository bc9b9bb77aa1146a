// Gated delta rule layers of any head size, with one decay per head or one per key channel, and the short causal
// convolution in front of them (the fixed 128 x 128, four-tap form of the hybrid family is gdn.cu).
//
//   conv_silu_kernel     depthwise causal convolution of any number of taps + SiLU; token tiles run in parallel, the
//                        last taps - 1 inputs of every channel are the request's convolution state
//   delta_rule_kernel    per (head, segment, slice of value rows): unit q / k, beta = sigmoid(b),
//                        g = exp(-exp(A_log) softplus(a + dt_bias)) per head or per (head, key channel), then per token
//                            S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//                        and the gated RMS norm of a head's output
//   gated_norm_kernel    that norm as a kernel of its own, when a head's value rows are split over several blocks
//
// S^T q is taken from the decayed state before the write: o = S^T q + (k . q) u, so that both reductions over the key
// channels of a token happen at once.  The state [slot][head][value row][key channel] is fp32 and stays in registers for
// a whole segment; all arithmetic is fp32.  Only the projections and the convolution's outputs have the activation type.
#include "segments.cuh"
#include "launch.cuh"

namespace cb {

// ------------------------------------------------------------------ short convolution
static constexpr int kConvRows = 16;       // tokens per block
static constexpr int kConvThreads = 128;   // two channels per thread

template <typename T> struct Pair2;
template <> struct Pair2<__nv_bfloat16> { using type = __nv_bfloat162; };
template <> struct Pair2<float> { using type = float2; };
__device__ __forceinline__ float2 to_f2(__nv_bfloat162 v) { return __bfloat1622float2(v); }
__device__ __forceinline__ float2 to_f2(float2 v) { return v; }
__device__ __forceinline__ void store2(__nv_bfloat16* p, float2 v) { *reinterpret_cast<__nv_bfloat162*>(p) = __float22bfloat162_rn(v); }
__device__ __forceinline__ void store2(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ float silu_exact(float x) { return x / (1.f + expf(-x)); }

// The block that holds a segment's first tokens also replaces the convolution state: it is the only one that reads it.
template <typename T, int TAPS>
__global__ void __launch_bounds__(kConvThreads)
conv_silu_kernel(const T* __restrict__ x, int ldx, T* __restrict__ y, int ldy, const float* __restrict__ w,   // [C, TAPS]
                 T* __restrict__ state,                                                                       // [slots, TAPS - 1, C]
                 Segments sg, int C) {
  using P = typename Pair2<T>::type;
  pdl_wait();
  pdl_launch_dependents();
  int s, off;
  if (!find_tile(sg, kConvRows, blockIdx.y, s, off)) return;
  const int c = (blockIdx.x * kConvThreads + threadIdx.x) * 2;
  if (c >= C) return;
  const int n = sg.count[s];
  const T* xp = x + static_cast<size_t>(sg.row0[s]) * ldx + c;
  T* yp = y + static_cast<size_t>(sg.row0[s]) * ldy + c;
  float2 wv[TAPS];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) wv[j] = make_float2(w[static_cast<size_t>(c) * TAPS + j], w[static_cast<size_t>(c + 1) * TAPS + j]);
  constexpr int H = TAPS - 1;
  float2 hist[H > 0 ? H : 1];               // inputs at t - H .. t - 1
  T* st = state + static_cast<size_t>(sg.slot[s]) * H * C + c;
  if (off == 0) {
    const bool fresh = sg.pos0[s] == 0;
#pragma unroll
    for (int j = 0; j < H; ++j)
      hist[j] = fresh ? make_float2(0.f, 0.f) : to_f2(*reinterpret_cast<const P*>(st + static_cast<size_t>(j) * C));
    // new state: inputs n - H .. n - 1, where negative indices are entries of the old state
#pragma unroll
    for (int j = 0; j < H; ++j) {
      const int t = n - H + j;
      float2 v = make_float2(0.f, 0.f);
      if (t >= 0) {
        v = to_f2(*reinterpret_cast<const P*>(xp + static_cast<size_t>(t) * ldx));
      } else {
#pragma unroll
        for (int i = 0; i < H; ++i) if (i == t + H) v = hist[i];
      }
      store2(st + static_cast<size_t>(j) * C, v);
    }
  } else {
#pragma unroll
    for (int j = 0; j < H; ++j) {            // a tile that is not the first starts at least kConvRows >= H tokens in
      hist[j] = to_f2(*reinterpret_cast<const P*>(xp + static_cast<size_t>(off - H + j) * ldx));
    }
  }
  const int end = min(n, off + kConvRows);
#pragma unroll 4
  for (int t = off; t < end; ++t) {
    const float2 v = to_f2(*reinterpret_cast<const P*>(xp + static_cast<size_t>(t) * ldx));
    float2 a = make_float2(wv[H].x * v.x, wv[H].y * v.y);
#pragma unroll
    for (int j = 0; j < H; ++j) { a.x = fmaf(wv[j].x, hist[j].x, a.x); a.y = fmaf(wv[j].y, hist[j].y, a.y); }
    store2(yp + static_cast<size_t>(t) * ldy, make_float2(silu_exact(a.x), silu_exact(a.y)));
#pragma unroll
    for (int j = 0; j + 1 < H; ++j) hist[j] = hist[j + 1];
    if (H > 0) hist[H - 1] = v;
  }
}

// ------------------------------------------------------------------ delta rule
template <typename T>
struct DeltaRule {
  const T* qkv; int ldq;      // after the convolution: q [G d] | k [G d] | v [H e]
  const T* b; int ldb;        // [H] step size logits
  const T* a; int lda;        // decay logits: [H] or [H d]
  const T* z; int ldz;        // output gate [H e]
  const float* a_log;         // [H]
  const float* dt_bias;       // [H] or [H d]
  const float* norm_w;        // [e]
  float* state;               // [slots, H, e, ds]
  T* out; int ldo;            // [H e]
  float* raw;                 // fp32 [T, H e]: outputs before the norm (value rows split over blocks), or null
  int H, G, d, e, ds;         // ds: row stride of the state, d rounded up to 4
  float eps;
  int sigmoid_gate;           // output gate sigmoid(z) instead of silu(z)
  Segments sg;
};

__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) { return __ffma2_rn(a, b, c); }
__device__ __forceinline__ float2 mul2(float2 a, float2 b) { return __fmul2_rn(a, b); }
__device__ __forceinline__ float gate_of(float z, int sigmoid) { return (sigmoid ? 1.f : z) / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_of(float x) { return x > 20.f ? x + log1pf(expf(-x)) : log1pf(expf(x)); }

// KD: key channels covered by a row's lanes (d <= KD).  LPR = KD / 16 lanes share a state row, lane l holds the float4
// chunks l + LPR c (c < 4); a thread holds RPT rows.  NB tokens are prepared at a time.
//
// PIPE: the block has kPrepWarps more warps that prepare the operands of the next NB tokens and normalise the outputs
// of the previous NB while the other warps walk the recurrence (two shared-memory buffers, one barrier per NB tokens).
// Without it (decode: one token per segment) all warps do both in turn, and two blocks share an SM so that one's
// state traffic overlaps the other's arithmetic.
static constexpr int kPrepWarps = 8;

template <int KD> struct DeltaShape {
  static constexpr int LPR = KD / 16;
  static constexpr int NB = KD <= 128 ? 16 : 8;
  static constexpr int kMaxRowThreads = 256;
};

template <typename T, int KD, int RPT, bool CHANNEL, bool PIPE>
__global__ void __launch_bounds__(PIPE ? 256 + 32 * kPrepWarps : 256, PIPE ? 1 : 2)
delta_rule_kernel(const DeltaRule<T> p) {
  constexpr int LPR = DeltaShape<KD>::LPR, NB = PIPE ? DeltaShape<KD>::NB : 1;
  constexpr int KV = KD / 32;
  constexpr int OPS = CHANNEL ? 3 : 2;                    // q, k (, g) rows per token
  extern __shared__ __align__(16) float sm[];
  pdl_wait();
  pdl_launch_dependents();
  const int head = blockIdx.x, s = blockIdx.y;
  const int n = p.sg.count[s];
  if (n <= 0) return;
  const int row_threads = PIPE ? blockDim.x - 32 * kPrepWarps : blockDim.x;
  const int VT = row_threads / LPR * RPT;                 // value rows of this block
  const int v0 = blockIdx.z * VT;
  const int e_here = min(VT, p.e - v0);
  const int buf_floats = NB * (OPS * KD + VT + 4);
  float* const obuf = sm + (PIPE ? 2 : 1) * buf_floats;   // [PIPE ? 2 : 1][NB][VT]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const bool rower = tid < row_threads;
  const int l = tid % LPR, grp = tid / LPR, ngrp = row_threads / LPR;
  const size_t row0 = p.sg.row0[s];
  const int hq = head / (p.H / p.G);
  const float rate = -expf(p.a_log[head]);

  // the state's loads are issued first: their latency covers the preparation of the first tokens
  float* sp = p.state + (static_cast<size_t>(p.sg.slot[s]) * p.H + head) * p.e * p.ds;
  float2 S[RPT][8];
  const bool fresh = p.sg.pos0[s] == 0;
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int v = v0 + grp + i * ngrp;
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const int col = 4 * (l + LPR * c);
      float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
      if (rower && !fresh && v < p.e && col < p.ds) t = *reinterpret_cast<const float4*>(sp + static_cast<size_t>(v) * p.ds + col);
      S[i][2 * c] = make_float2(t.x, t.y);
      S[i][2 * c + 1] = make_float2(t.z, t.w);
    }
  }

  auto bufq = [&](int b) { return sm + b * buf_floats; };
  auto bufc = [&](int b) { return sm + b * buf_floats + NB * OPS * KD; };          // float4 per token: 16-byte aligned
  auto bufv = [&](int b) { return sm + b * buf_floats + NB * (OPS * KD + 4); };

  // operands of token t (of the segment) into slot j of buffer b: `part` 0 unit q and k, beta, k . q, scalar decay;
  // 1 the value rows; 2 the channel decays
  auto prep = [&](int t, int j, int b, int part) {
    const size_t r = row0 + t;
    const T* row = p.qkv + r * p.ldq;
    if (part == 0) {
      float q[KV], k[KV];
#pragma unroll
      for (int i = 0; i < KV; ++i) {
        const int c = lane + 32 * i;
        q[i] = c < p.d ? to_f(row[hq * p.d + c]) : 0.f;
        k[i] = c < p.d ? to_f(row[(p.G + hq) * p.d + c]) : 0.f;
      }
      const float bl = to_f(p.b[r * p.ldb + head]);
      const float al = CHANNEL ? 0.f : to_f(p.a[r * p.lda + head]) + p.dt_bias[head];
      float qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
      for (int i = 0; i < KV; ++i) { qq = fmaf(q[i], q[i], qq); kk = fmaf(k[i], k[i], kk); }
      qq = warp_sum(qq);
      kk = warp_sum(kk);
      const float qi = 1.f / sqrtf(qq + 1e-6f) * (1.f / sqrtf(static_cast<float>(p.d))), ki = 1.f / sqrtf(kk + 1e-6f);
      float* qs = bufq(b) + j * KD;
      float* ks = qs + NB * KD;
#pragma unroll
      for (int i = 0; i < KV; ++i) {
        q[i] *= qi;
        k[i] *= ki;
        qs[lane + 32 * i] = q[i];
        ks[lane + 32 * i] = k[i];
        qk = fmaf(q[i], k[i], qk);
      }
      qk = warp_sum(qk);
      if (lane == 0)
        *reinterpret_cast<float4*>(bufc(b) + j * 4) =
            make_float4(1.f / (1.f + expf(-bl)), CHANNEL ? 1.f : expf(rate * softplus_of(al)), qk, 0.f);
    } else if (part == 1) {
      float* vs = bufv(b) + j * VT;
      const T* vr = row + 2 * p.G * p.d + head * p.e + v0;
      for (int c = lane; c < e_here; c += 32) vs[c] = to_f(vr[c]);
    } else {
      float* gs = bufq(b) + (2 * NB + j) * KD;
      const T* ar = p.a + r * p.lda + head * p.d;
#pragma unroll
      for (int i = 0; i < KV; ++i) {
        const int c = lane + 32 * i;
        gs[c] = c < p.d ? expf(rate * softplus_of(to_f(ar[c]) + p.dt_bias[head * p.d + c])) : 0.f;
      }
    }
  };

  // gated norm of token t's outputs (slot j of buffer b), or their raw store when the head is split
  auto finish = [&](int t, int j, int b) {
    const float* o = obuf + (b * NB + j) * VT;
    const size_t r = row0 + t;
    if (p.raw) {
      float* dst = p.raw + r * (static_cast<size_t>(p.H) * p.e) + head * p.e + v0;
      for (int c = lane; c < e_here; c += 32) dst[c] = o[c];
      return;
    }
    float ss = 0.f;
    for (int c = lane; c < p.e; c += 32) ss = fmaf(o[c], o[c], ss);
    const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(p.e) + p.eps);
    const T* zr = p.z + r * p.ldz + head * p.e;
    T* dst = p.out + r * p.ldo + head * p.e;
    for (int c = lane; c < p.e; c += 32)
      dst[c] = from_f<T>(o[c] * inv * p.norm_w[c] * gate_of(to_f(zr[c]), p.sigmoid_gate));
  };

  // the recurrence over nb tokens of buffer b
  auto walk = [&](int nb, int b) {
    const float* qb = bufq(b);
    const float* vb = bufv(b);
    const float* cb_ = bufc(b);
    float* ob = obuf + b * NB * VT;
#pragma unroll 1
    for (int j = 0; j < nb; ++j) {
      const float4 co = *reinterpret_cast<const float4*>(cb_ + j * 4);
      const float2 g1 = make_float2(co.y, co.y);
      float2 k2[8], aa[RPT], bb[RPT];
      float va[RPT];
#pragma unroll
      for (int i = 0; i < RPT; ++i) {
        aa[i] = make_float2(0.f, 0.f);
        bb[i] = make_float2(0.f, 0.f);
        va[i] = vb[j * VT + grp + i * ngrp];
      }
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int col = 4 * (l + LPR * c);
        const float4 q4 = *reinterpret_cast<const float4*>(qb + j * KD + col);
        const float4 k4 = *reinterpret_cast<const float4*>(qb + (NB + j) * KD + col);
        float2 ga = g1, gb = g1;
        if constexpr (CHANNEL) {
          const float4 g4 = *reinterpret_cast<const float4*>(qb + (2 * NB + j) * KD + col);
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
          aa[i] = fma2(S[i][2 * c], k2[2 * c], aa[i]);
          bb[i] = fma2(S[i][2 * c], q0, bb[i]);
          aa[i] = fma2(S[i][2 * c + 1], k2[2 * c + 1], aa[i]);
          bb[i] = fma2(S[i][2 * c + 1], q1, bb[i]);
        }
      }
      float sa[RPT], sb[RPT];
#pragma unroll
      for (int i = 0; i < RPT; ++i) { sa[i] = aa[i].x + aa[i].y; sb[i] = bb[i].x + bb[i].y; }
#pragma unroll
      for (int sh = 1; sh < LPR; sh <<= 1)
#pragma unroll
        for (int i = 0; i < RPT; ++i) {
          sa[i] += __shfl_xor_sync(0xffffffffu, sa[i], sh);
          sb[i] += __shfl_xor_sync(0xffffffffu, sb[i], sh);
        }
#pragma unroll
      for (int i = 0; i < RPT; ++i) {
        const float u = co.x * (va[i] - sa[i]);
        if (l == 0) ob[j * VT + grp + i * ngrp] = fmaf(co.z, u, sb[i]);
        const float2 u2 = make_float2(u, u);
#pragma unroll
        for (int c = 0; c < 8; ++c) S[i][c] = fma2(k2[c], u2, S[i][c]);
      }
    }
  };

  if constexpr (PIPE) {
    const int pw = warp - (row_threads >> 5);
    const int blocks = (n + NB - 1) / NB;
    auto prep_block = [&](int blk) {
      const int t0 = blk * NB, nb = min(NB, n - t0), b = blk & 1;
      // a token per warp and turn, its parts back to back so that their loads are in flight together
#pragma unroll 2
      for (int j = pw; j < nb; j += kPrepWarps) {
        prep(t0 + j, j, b, 0);
        prep(t0 + j, j, b, 1);
        if constexpr (CHANNEL) prep(t0 + j, j, b, 2);
      }
    };
    auto finish_block = [&](int blk) {
      const int t0 = blk * NB, nb = min(NB, n - t0);
      for (int j = pw; j < nb; j += kPrepWarps) finish(t0 + j, j, blk & 1);
    };
    if (!rower) prep_block(0);
    __syncthreads();
    for (int blk = 0; blk < blocks; ++blk) {
      if (rower) {
        walk(min(NB, n - blk * NB), blk & 1);
      } else {
        if (blk > 0) finish_block(blk - 1);
        if (blk + 1 < blocks) prep_block(blk + 1);
      }
      __syncthreads();
    }
    if (!rower) finish_block(blocks - 1);
  } else {
    const int nwarps = blockDim.x >> 5;
    for (int t = 0; t < n; ++t) {
      for (int part = warp; part < OPS; part += nwarps) prep(t, 0, 0, part);
      __syncthreads();
      walk(1, 0);
      __syncthreads();
      if (warp == 0) finish(t, 0, 0);
      // the outputs of this token are read by warp 0 while the others prepare the next one; they are overwritten only
      // after the next barrier
    }
  }
  if (!rower) return;
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int v = v0 + grp + i * ngrp;
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const int col = 4 * (l + LPR * c);
      if (v < p.e && col < p.ds)
        *reinterpret_cast<float4*>(sp + static_cast<size_t>(v) * p.ds + col) =
            make_float4(S[i][2 * c].x, S[i][2 * c].y, S[i][2 * c + 1].x, S[i][2 * c + 1].y);
    }
  }
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
  float ss = 0.f;
  for (int c = lane; c < e; c += 32) ss = fmaf(o[c], o[c], ss);
  const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(e) + eps);
  for (int c = lane; c < e; c += 32)
    out[t * ldo + h * e + c] = from_f<T>(o[c] * inv * w[c] * gate_of(to_f(z[t * ldz + h * e + c]), sigmoid_gate));
}

// ------------------------------------------------------------------ host
template <typename T>
static int conv_launch(const void* x, int ldx, void* y, int ldy, const void* w, void* state, const Segments& sg, int C,
                       int taps, int tokens, cudaStream_t st) {
  const dim3 grid((C / 2 + kConvThreads - 1) / kConvThreads, max_tiles(tokens, sg.num, kConvRows));
  auto go = [&](auto kernel) {
    return static_cast<int>(launch(kernel, grid, dim3(kConvThreads), 0, st, static_cast<const T*>(x), ldx,
                                   static_cast<T*>(y), ldy, static_cast<const float*>(w), static_cast<T*>(state), sg, C));
  };
  switch (taps) {
    case 1: return go(conv_silu_kernel<T, 1>);
    case 2: return go(conv_silu_kernel<T, 2>);
    case 3: return go(conv_silu_kernel<T, 3>);
    case 4: return go(conv_silu_kernel<T, 4>);
    case 5: return go(conv_silu_kernel<T, 5>);
    case 6: return go(conv_silu_kernel<T, 6>);
    case 7: return go(conv_silu_kernel<T, 7>);
    case 8: return go(conv_silu_kernel<T, 8>);
  }
  return -12;
}

template <typename T, int KD, int RPT, bool CHANNEL, bool PIPE>
static int delta_go(const DeltaRule<T>& p, int row_threads, int vtiles, cudaStream_t st) {
  constexpr int NB = PIPE ? DeltaShape<KD>::NB : 1;
  const int VT = row_threads / DeltaShape<KD>::LPR * RPT;
  const size_t smem = sizeof(float) * (PIPE ? 2 : 1) * NB * ((CHANNEL ? 3 : 2) * KD + 2 * VT + 4);
  auto kernel = delta_rule_kernel<T, KD, RPT, CHANNEL, PIPE>;
  static bool configured[64] = {};     // per device
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -18;
  if (!configured[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured[dev] = true;
  }
  return static_cast<int>(launch(kernel, dim3(p.H, p.sg.num, vtiles), dim3(row_threads + (PIPE ? 32 * kPrepWarps : 0)), smem,
                                 st, p));
}

template <typename T, int KD>
static int delta_kd(DeltaRule<T> p, bool channel, bool decode, int tokens, float* raw, cudaStream_t st) {
  constexpr int LPR = DeltaShape<KD>::LPR;
  // rows per thread: four amortise the operand loads from shared memory; one spreads a head over more blocks when the
  // step has too few (head, request) pairs to fill the device
  const int max_rows4 = 256 / LPR * 4, max_rows1 = 256 / LPR;
  const bool spread = !decode && static_cast<long long>(p.H) * p.sg.num < 148;
  const int rpt = (spread || p.e <= max_rows1 / 2) ? 1 : 4;
  const int max_rows = rpt == 4 ? max_rows4 : max_rows1;
  const int vtiles = (p.e + max_rows - 1) / max_rows;
  const int rows = (p.e + vtiles - 1) / vtiles;
  int row_threads = (rows + rpt - 1) / rpt * LPR;
  row_threads = (row_threads + 31) / 32 * 32;
  // blocks cover row_threads / LPR * rpt rows each
  const int vt = row_threads / LPR * rpt;
  const int tiles = (p.e + vt - 1) / vt;
  p.raw = tiles > 1 ? raw : nullptr;
  if (tiles > 1 && !raw) return -13;
  int rc;
  if (decode) {
    if (rpt == 4) rc = channel ? delta_go<T, KD, 4, true, false>(p, row_threads, tiles, st) : delta_go<T, KD, 4, false, false>(p, row_threads, tiles, st);
    else rc = channel ? delta_go<T, KD, 1, true, false>(p, row_threads, tiles, st) : delta_go<T, KD, 1, false, false>(p, row_threads, tiles, st);
  } else if (rpt == 4) {
    rc = channel ? delta_go<T, KD, 4, true, true>(p, row_threads, tiles, st) : delta_go<T, KD, 4, false, true>(p, row_threads, tiles, st);
  } else {
    rc = channel ? delta_go<T, KD, 1, true, true>(p, row_threads, tiles, st) : delta_go<T, KD, 1, false, true>(p, row_threads, tiles, st);
  }
  if (rc || tiles == 1) return rc;
  const long long items = static_cast<long long>(tokens) * p.H;
  return static_cast<int>(launch(gated_norm_kernel<T>, dim3(static_cast<unsigned>((items + 7) / 8)), dim3(256), 0, st,
                                 static_cast<const float*>(raw), p.z, p.ldz, p.norm_w, p.out, p.ldo, tokens, p.H, p.e, p.eps,
                                 p.sigmoid_gate));
}

}  // namespace cb

extern "C" {

struct CbDeltaRule {
  const void* qkv; int ldq;
  const void* b; int ldb;
  const void* a; int lda;
  const void* z; int ldz;
  const void* a_log;
  const void* dt_bias;
  const void* norm_w;
  void* state;
  void* out; int ldo;
  void* raw;
  int H, G, d, e, ds;
  float eps;
  int sigmoid_gate, channel, decode, tokens, f32;
};

// `C` and the row strides are even; `taps` 1..8.  `f32`: activations and state are fp32.
int cb_conv_silu(const void* x, int ldx, void* y, int ldy, const void* w, void* state, const CbSegments* seg, int C, int taps,
                 int tokens, int f32, void* stream) {
  using namespace cb;
  if (!seg || seg->num <= 0 || tokens <= 0) return 0;
  if (C <= 0 || (C & 1) || (ldx & 1) || (ldy & 1) || taps < 1 || taps > 8) return -10;
  const int tiles = max_tiles(tokens, seg->num, kConvRows);
  if (tiles > 65535) return -11;
  const Segments sg = make_segments(seg);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return f32 ? conv_launch<float>(x, ldx, y, ldy, w, state, sg, C, taps, tokens, st)
             : conv_launch<__nv_bfloat16>(x, ldx, y, ldy, w, state, sg, C, taps, tokens, st);
}

}  // extern "C"

namespace cb {
template <typename T>
static int delta_typed(const CbDeltaRule* a, const CbSegments* seg, cudaStream_t st) {
  DeltaRule<T> p;
  p.qkv = static_cast<const T*>(a->qkv); p.ldq = a->ldq;
  p.b = static_cast<const T*>(a->b); p.ldb = a->ldb;
  p.a = static_cast<const T*>(a->a); p.lda = a->lda;
  p.z = static_cast<const T*>(a->z); p.ldz = a->ldz;
  p.a_log = static_cast<const float*>(a->a_log);
  p.dt_bias = static_cast<const float*>(a->dt_bias);
  p.norm_w = static_cast<const float*>(a->norm_w);
  p.state = static_cast<float*>(a->state);
  p.out = static_cast<T*>(a->out); p.ldo = a->ldo;
  p.raw = nullptr;
  p.H = a->H; p.G = a->G; p.d = a->d; p.e = a->e; p.ds = a->ds;
  p.eps = a->eps; p.sigmoid_gate = a->sigmoid_gate;
  p.sg = make_segments(seg);
  float* raw = static_cast<float*>(a->raw);
  if (a->d <= 64) return delta_kd<T, 64>(p, a->channel != 0, a->decode != 0, a->tokens, raw, st);
  if (a->d <= 128) return delta_kd<T, 128>(p, a->channel != 0, a->decode != 0, a->tokens, raw, st);
  return delta_kd<T, 256>(p, a->channel != 0, a->decode != 0, a->tokens, raw, st);
}
}  // namespace cb

extern "C" {

// `decode`: every segment has at most one row.  `raw`: fp32 scratch [tokens, H e].
int cb_delta_rule(const CbDeltaRule* a, const CbSegments* seg, void* stream) {
  if (!a || !seg || seg->num <= 0 || a->tokens <= 0) return 0;
  if (a->H <= 0 || a->G <= 0 || (a->H % a->G) != 0 || a->d <= 0 || a->d > 256 || a->e <= 0 || a->ds < a->d || (a->ds & 3) ||
      seg->num > 65535)
    return -10;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return a->f32 ? cb::delta_typed<float>(a, seg, st) : cb::delta_typed<__nv_bfloat16>(a, seg, st);
}

}  // extern "C"
