// Short causal convolution + SiLU over the tokens of a request, the building block of the recurrences' preparation
// (recurrence.cuh), and the fp32 helpers it shares with them.
#pragma once
#include "segments.cuh"

namespace cb {

template <typename T> struct Pair2;
template <> struct Pair2<__nv_bfloat16> { using type = __nv_bfloat162; };
template <> struct Pair2<float> { using type = float2; };
__device__ __forceinline__ float2 to_f2(__nv_bfloat162 v) { return __bfloat1622float2(v); }
__device__ __forceinline__ float2 to_f2(float2 v) { return v; }
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) { return __ffma2_rn(a, b, c); }
__device__ __forceinline__ float2 mul2(float2 a, float2 b) { return __fmul2_rn(a, b); }

// Exponential and softplus of the decays.  In a bf16 model the logits are bf16: the fast forms' absolute error (1e-7 and a
// few ulp of the exponential) is far below what the logits carry; fp32 models use the exact ones.
template <typename T> __device__ __forceinline__ float exp_of(float x) { return sizeof(T) == 2 ? __expf(x) : expf(x); }
template <typename T> __device__ __forceinline__ float softplus_of(float x) {
  const float e = exp_of<T>(-fabsf(x));
  return fmaxf(x, 0.f) + (sizeof(T) == 2 ? __logf(1.f + e) : log1pf(e));
}
template <typename T> __device__ __forceinline__ float silu_of(float x) { return sizeof(T) == 2 ? silu_fast(x) : x / (1.f + expf(-x)); }

// Two neighbouring channels p[0], p[1] where `ok`, zeros elsewhere: one predicated load, so that the loads of a whole tile can
// be in flight at once.  ODD: the pair may start at an odd channel and its second channel exists only where `ok1`.
template <typename T, bool ODD>
__device__ __forceinline__ float2 load_pair(const T* p, bool ok, bool ok1) {
  using P = typename Pair2<T>::type;
  if constexpr (ODD) return make_float2(ok ? to_f(p[0]) : 0.f, ok1 ? to_f(p[1]) : 0.f);
  float2 v = make_float2(0.f, 0.f);
  if (ok) v = to_f2(*reinterpret_cast<const P*>(p));
  return v;
}

// A causal depthwise convolution over the tokens of a segment, with the request's last taps - 1 inputs as its state.  Channel
// c is column c of x, of the weights and of the state.
template <typename T>
struct ShortConv {
  const T* x; int ldx;
  const float* w;             // [taps][ldw], the last row multiplies the current input
  const float* bias;          // [ldw] or null
  int ldw, taps;
  T* state;                   // [slots, taps - 1, ldw]
};

// Convolution + SiLU of one channel pair along a segment's tokens.  TAPS > 0: weights and the last inputs in registers; the
// caller reads the inputs of several tokens ahead and feeds them in order (heads of even width).  TAPS 0: any number of taps
// and any width, everything is read again for every token.  TAPS < 0: no convolution, the inputs pass (kPlain: heads of even
// width, kPlainOdd: any).
static constexpr int kPlain = -1, kPlainOdd = -2;
template <typename T, int TAPS, bool BIAS>
struct ConvPair {
  static constexpr int R = TAPS > 0 ? TAPS : 1;
  static constexpr bool ODD = TAPS == 0 || TAPS == kPlainOdd;
  float2 w[R], hist[R], b;
  const ShortConv<T>* p;
  const T* xr;
  const T* st;
  bool fresh, ok, ok1;
  int col;                                                        // first channel of the pair

  __device__ __forceinline__ float2 input(int t) const {          // input at token t of the segment, t >= -(taps - 1)
    const T* src = t >= 0 ? xr + static_cast<ptrdiff_t>(t) * p->ldx : st + static_cast<ptrdiff_t>(t + p->taps - 1) * p->ldw;
    const bool there = t >= 0 || !fresh;
    return load_pair<T, ODD>(src + col, ok && there, ok1 && there);
  }
  __device__ __forceinline__ float2 weight(int j) const {
    return load_pair<float, ODD>(p->w + static_cast<size_t>(j) * p->ldw + col, ok, ok1);
  }
  __device__ __forceinline__ void begin(const ShortConv<T>& prm, const T* x, const T* state, bool fr, int base, int c, int lim,
                                        int t0) {
    p = &prm; xr = x; st = state; fresh = fr; col = base + c; ok = c < lim; ok1 = c + 1 < lim;
    if constexpr (BIAS) b = load_pair<float, ODD>(p->bias + col, ok, ok1);
    if constexpr (TAPS > 0) {
#pragma unroll
      for (int j = 0; j < TAPS; ++j) w[j] = weight(j);
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) hist[j] = input(t0 - (TAPS - 1) + j);
    }
  }
  __device__ __forceinline__ float2 ahead(int t, int end) const { // the input `token` wants, t >= 0; nothing behind the tile
    if constexpr (TAPS == 0) return make_float2(0.f, 0.f);
    return load_pair<T, ODD>(xr + static_cast<ptrdiff_t>(t) * p->ldx + col, ok && t < end, ok1 && t < end);
  }
  __device__ __forceinline__ float2 token(int t, float2 v) {      // tokens in order from t0 on
    if constexpr (TAPS < 0) return v;
    float2 a;
    if constexpr (TAPS > 0) {
      if constexpr (BIAS) a = fma2(w[TAPS - 1], v, b);
      else a = mul2(w[TAPS - 1], v);
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) a = fma2(w[j], hist[j], a);
#pragma unroll
      for (int j = 0; j + 1 < TAPS - 1; ++j) hist[j] = hist[j + 1];
      if constexpr (TAPS > 1) hist[TAPS - 2] = v;
    } else {
      a = BIAS ? b : make_float2(0.f, 0.f);
#pragma unroll 1
      for (int j = 0; j < p->taps; ++j) a = fma2(weight(j), input(t - (p->taps - 1) + j), a);
    }
    return make_float2(silu_of<T>(a.x), silu_of<T>(a.y));
  }
  // The pair's new convolution state, written by the tile that holds the segment's first tokens (the only reader of the old
  // one): from the registers when it holds the last tokens too, else from the inputs.
  __device__ __forceinline__ void save(T* state, int count, bool whole) const {
    if constexpr (TAPS > 1) {
      float2 v[TAPS - 1];
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) v[j] = whole ? hist[j] : input(count - (TAPS - 1) + j);
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) {
        T* dst = state + static_cast<ptrdiff_t>(j) * p->ldw + col;
        if (ok) dst[0] = from_f<T>(v[j].x);
        if (ok1) dst[1] = from_f<T>(v[j].y);
      }
    }
  }
};

// The convolution state of channels [base, base + n) becomes the segment's last taps - 1 inputs.  Called after the
// outputs that need the old state, by the warp that produced them.
template <typename T>
__device__ __forceinline__ void conv_state(const ShortConv<T>& p, const T* xr, T* st, bool fresh, int count, int base, int n) {
  const int H = p.taps - 1;
  __syncwarp();                              // read in pairs, replaced channel by channel
  for (int c = threadIdx.x & 31; c < n; c += 32)
    for (int j = 0; j < H; ++j) {            // entry j moves down from entry j + count, which is read before it is written
      const int t = count - H + j;
      T v = from_f<T>(0.f);
      if (t >= 0) v = xr[static_cast<ptrdiff_t>(t) * p.ldx + base + c];
      else if (!fresh) v = st[static_cast<ptrdiff_t>(t + H) * p.ldw + base + c];
      st[static_cast<ptrdiff_t>(j) * p.ldw + base + c] = v;
    }
}

}  // namespace cb
