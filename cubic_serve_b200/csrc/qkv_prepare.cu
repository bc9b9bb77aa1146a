// Queries, keys and values of the layered decoders' attention on their way from the projection to the padded queries and the paged
// cache of gqa_attn.cu (values of their own; gqa_attn.cu prepares the layers whose values are raw keys).
//
//   conv_qkv_kernel   short causal convolution over time on every channel, rotary positions on the halves of a head's first
//                     channels, every query and key head over its root mean square
//   norm_qkv_kernel   queries and keys of a token over the root mean square of their whole projection, times a weight per channel;
//                     queries times a factor that grows with the position
//   head_qkv_kernel   every query and key head, or map of it, over its root mean square, times a weight per channel, rotary positions
//                     on the halves of its first channels
//
// In the first two a warp takes a head, lane l the channels 4 l .. and 128 + 4 l ..; in the last, rows of 32 or 64 columns share a
// warp.  Everything between the projection and the stored row is fp32.
#include <type_traits>

#include "segments.cuh"
#include "launch.cuh"

namespace cb {

static constexpr int kQkvPage = 16;
static constexpr int kQkvWarps = 4;
static constexpr int kQkvTokens = 16;       // of a conv_qkv_kernel block; at least the convolution's history (taps - 1)

// Four channels c .. c + 3 of a row of d; `vec`: rows start at multiples of four elements and d is one
__device__ __forceinline__ float4 load_four(const float* p, int c, int d, bool vec) {
  if (vec) return c < d ? *reinterpret_cast<const float4*>(p + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  return make_float4(c < d ? p[c] : 0.f, c + 1 < d ? p[c + 1] : 0.f, c + 2 < d ? p[c + 2] : 0.f, c + 3 < d ? p[c + 3] : 0.f);
}
// ... of an activation row as they are stored, and as numbers
__device__ __forceinline__ float4 load_raw(const float* p, int c, int d, bool vec) { return load_four(p, c, d, vec); }
__device__ __forceinline__ uint2 load_raw(const __nv_bfloat16* p, int c, int d, bool vec) {
  uint2 u = make_uint2(0u, 0u);
  if (vec) {
    if (c < d) u = *reinterpret_cast<const uint2*>(p + c);
  } else {
    u.x = pack_bf16x2(c < d ? to_f(p[c]) : 0.f, c + 1 < d ? to_f(p[c + 1]) : 0.f);
    u.y = pack_bf16x2(c + 2 < d ? to_f(p[c + 2]) : 0.f, c + 3 < d ? to_f(p[c + 3]) : 0.f);
  }
  return u;
}
__device__ __forceinline__ float4 unpack_four(float4 v) { return v; }
__device__ __forceinline__ float4 unpack_four(uint2 u) {
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
template <typename T> struct RawFour;
template <> struct RawFour<float> { using type = float4; };
template <> struct RawFour<__nv_bfloat16> { using type = uint2; };
__device__ __forceinline__ float4 load_four(const __nv_bfloat16* p, int c, int d, bool vec) { return unpack_four(load_raw(p, c, d, vec)); }
__device__ __forceinline__ void store_four(float* p, int c, float4 v) { *reinterpret_cast<float4*>(p + c) = v; }
__device__ __forceinline__ void store_four(__nv_bfloat16* p, int c, float4 v) {
  *reinterpret_cast<uint2*>(p + c) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}
__device__ __forceinline__ float4 fma_four(float4 a, float4 b, float4 c) {
  return make_float4(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y), fmaf(a.z, b.z, c.z), fmaf(a.w, b.w, c.w));
}
__device__ __forceinline__ float4 mul_four(float4 a, float s) { return make_float4(a.x * s, a.y * s, a.z * s, a.w * s); }
__device__ __forceinline__ float dot_four(float4 a, float4 b) { return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, a.w * b.w))); }

template <typename T>
struct QkvPrep {
  const T* x; int ldx;        // projections
  int q_off, k_off, v_off;    // columns of q [H d], k [G d] and v [G e]
  T* q;                       // [T, H, P]
  T* cache;                   // [pages][G][key, value][16][P]
  const int* slots;           // [T] cache row, < 0: none
  int H, G, d, e, P;
  float eps;
  int vec;                    // four channels at a time

  // Where token t's row of item `it` (H queries, G keys, G values) goes, null: nowhere
  __device__ __forceinline__ T* row(int it, size_t t, int slot) const {
    if (it < H) return q + (t * H + it) * P;
    if (slot < 0) return nullptr;
    const bool value = it >= H + G;
    const int g = it - H - (value ? G : 0);
    return cache + (((static_cast<size_t>(slot / kQkvPage) * G + g) * 2 + value) * kQkvPage + slot % kQkvPage) * P;
  }
  __device__ __forceinline__ int col(int it) const { return it < H ? q_off + it * d : it < H + G ? k_off + (it - H) * d : v_off + (it - H - G) * e; }
  __device__ __forceinline__ int width(int it) const { return it < H + G ? d : e; }
};

template <typename T>
struct ConvQkv {
  QkvPrep<T> a;
  const float* w;             // [taps][ldw], column 0 is the first query's; the last row multiplies the current input
  int ldw, taps;
  T* state;                   // [slots, taps - 1, ldw]: a request's last inputs
  const float* freq;          // [2][pairs] radians per position, and what they were rounded by
  int pairs;
  const int* positions;
  Segments sg;
};

// A block takes a tile of tokens of one segment and the heads blockIdx.y, + gridDim.y, ... by warps.  TAPS: 0 any number.  NJ: 128-channel
// chunks of a head.  BATCH: tokens a warp has in flight (1: steps of one token per segment).
template <typename T, int TAPS, int NJ, int BATCH>
__global__ void __launch_bounds__(32 * kQkvWarps, NJ > 1 ? 1 : BATCH > 1 ? 5 : 8)
conv_qkv_kernel(const ConvQkv<T> p) {
  constexpr int R = TAPS > 0 ? TAPS : 1, ROW = 128 * NJ, TOKS = BATCH == 1 ? 1 : kQkvTokens;
  using Raw = typename RawFour<T>::type;
  extern __shared__ __align__(16) float lsm[];                         // cosines and sines [tokens][half], then the warps' rows
  __shared__ long long place[TOKS];                                    // first element of a token's first key in the cache, -1: none
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait();
  pdl_launch_dependents();
  int s, off;
  if (!find_tile(p.sg, kQkvTokens, blockIdx.x, s, off)) return;
  const QkvPrep<T>& a = p.a;
  const int count = p.sg.count[s], toks = BATCH == 1 ? 1 : min(kQkvTokens, count - off);
  const size_t row0 = p.sg.row0[s];                                    // first row of the segment
  const bool fresh = p.sg.pos0[s] == 0;
  const int hist_rows = p.taps - 1;
  T* st = p.state + static_cast<size_t>(p.sg.slot[s]) * hist_rows * p.ldw;
  const int half = p.pairs, dims = 2 * half, hp = (half + 3) & ~3;     // hp: a token's cosines start at multiples of 16 bytes
  float* cosine = lsm;
  float* sine = lsm + TOKS * hp;
  for (int i = threadIdx.x; i < toks * half; i += 32 * kQkvWarps) {
    const int t = BATCH == 1 ? 0 : i / half, j = i - t * half;
    // the rounding error of the product is put back: angles of far positions keep their fraction of a turn
    const float pos = static_cast<float>(p.positions[row0 + off + t]), f = p.freq[j];
    const float ang = pos * f, e = fmaf(pos, f, -ang) + pos * p.freq[half + j];
    float sn, cs;
    sincosf(ang, &sn, &cs);
    const float ce = fmaf(-0.5f * e, e, 1.f), se = e * fmaf(e * (-1.f / 6.f), e, 1.f);
    cosine[t * hp + j] = cs * ce - sn * se;
    sine[t * hp + j] = fmaf(sn, ce, cs * se);
  }
  if (static_cast<int>(threadIdx.x) < toks) {
    const int slot = a.slots[row0 + off + threadIdx.x];
    place[threadIdx.x] = slot < 0 ? -1 : (static_cast<long long>(slot / kQkvPage) * a.G * 2 * kQkvPage + slot % kQkvPage) * a.P;
  }
  __syncthreads();
  float* swap = lsm + 2 * TOKS * hp + warp * BATCH * ROW;
  const bool vec = a.vec, vec_turn = (half & 3) == 0;
  for (int it = blockIdx.y * kQkvWarps + warp; it < a.H + 2 * a.G; it += kQkvWarps * gridDim.y) {
    const int d = a.width(it), col = a.col(it), wc = col - a.q_off;
    const bool query = it < a.H, value = it >= a.H + a.G;
    const T* xr = a.x + row0 * a.ldx + col;
    const float inv_d = 1.f / static_cast<float>(d);
    // where token t's row goes, by its entry of `place`
    T* const dst0 = query ? a.q + ((row0 + off) * a.H + it) * a.P
                          : a.cache + static_cast<size_t>(2 * (it - a.H - (value ? a.G : 0)) + value) * kQkvPage * a.P;
    // input at token t of the segment (t >= -(taps - 1)), channels of chunk j
    auto raw = [&](int t, int j) { return load_raw(xr + static_cast<size_t>(t) * a.ldx, 4 * lane + 128 * j, d, vec); };
    auto input = [&](int t, int j) {
      if (t >= 0) return unpack_four(raw(t, j));
      if (fresh) return make_float4(0.f, 0.f, 0.f, 0.f);
      return load_four(st + static_cast<size_t>(t + hist_rows) * p.ldw + wc, 4 * lane + 128 * j, d, vec);
    };
    auto tap = [&](int k, int j) { return load_four(p.w + static_cast<size_t>(k) * p.ldw + wc, 4 * lane + 128 * j, d, vec); };
    float4 w[R][NJ], hist[R][NJ];
    Raw next[BATCH][NJ];                                               // the inputs of the tokens that come next
    if constexpr (TAPS > 0) {
#pragma unroll
      for (int k = 0; k < TAPS - 1; ++k)
#pragma unroll
        for (int j = 0; j < NJ; ++j) hist[k][j] = input(off + k - (TAPS - 1), j);
#pragma unroll
      for (int b = 0; b < BATCH; ++b)
#pragma unroll
        for (int j = 0; j < NJ; ++j) next[b][j] = raw(off + min(b, toks - 1), j);
#pragma unroll
      for (int k = 0; k < TAPS; ++k)
#pragma unroll
        for (int j = 0; j < NJ; ++j) w[k][j] = tap(k, j);
    }
    // tokens t0 .. + BATCH - 1 of the tile; FULL: all of them exist
    auto batch = [&](int t0, auto full) {
      constexpr bool FULL = decltype(full)::value;
      float4 v[BATCH][NJ];
      if constexpr (TAPS > 0) {
#pragma unroll
        for (int b = 0; b < BATCH; ++b) {
#pragma unroll
          for (int j = 0; j < NJ; ++j) {
            const float4 in = unpack_four(next[b][j]);
            float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int k = 0; k < TAPS - 1; ++k) acc = fma_four(w[k][j], hist[k][j], acc);
            v[b][j] = fma_four(w[TAPS - 1][j], in, acc);
            if (FULL || t0 + b < toks) {
#pragma unroll
              for (int k = 0; k + 1 < TAPS - 1; ++k) hist[k][j] = hist[k + 1][j];
              if constexpr (TAPS > 1) hist[TAPS - 2][j] = in;
            }
          }
        }
        if (t0 + BATCH < toks) {                                       // nothing behind the tile
#pragma unroll
          for (int b = 0; b < BATCH; ++b)
#pragma unroll
            for (int j = 0; j < NJ; ++j) next[b][j] = raw(off + min(t0 + BATCH + b, toks - 1), j);
        }
      } else {
#pragma unroll
        for (int b = 0; b < BATCH; ++b)
#pragma unroll
          for (int j = 0; j < NJ; ++j) {
            v[b][j] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (!FULL && t0 + b >= toks) continue;
#pragma unroll 1
            for (int k = 0; k < p.taps; ++k) v[b][j] = fma_four(tap(k, j), input(off + t0 + b - hist_rows + k, j), v[b][j]);
          }
      }
      if (!value) {
        if (half) {
          __syncwarp();                                                // the rows before these were read
#pragma unroll
          for (int b = 0; b < BATCH; ++b)
#pragma unroll
            for (int j = 0; j < NJ; ++j) store_four(swap, b * ROW + 4 * lane + 128 * j, v[b][j]);
          __syncwarp();
#pragma unroll
          for (int j = 0; j < NJ; ++j) {
            const int c = 4 * lane + 128 * j;
            if (c >= dims) continue;
            if (vec_turn) {                                            // four channels turn with four neighbours
              const bool hi = c >= half;
              const float sg = hi ? 1.f : -1.f;
              const int other = hi ? c - half : c + half, low = hi ? c - half : c;
#pragma unroll
              for (int b = 0; b < BATCH; ++b) {
                const int at = (FULL || t0 + b < toks ? t0 + b : 0) * hp + low;
                const float4 o = *reinterpret_cast<const float4*>(swap + b * ROW + other);
                const float4 cs = *reinterpret_cast<const float4*>(cosine + at), sn = *reinterpret_cast<const float4*>(sine + at);
                float4& u = v[b][j];
                u = make_float4(fmaf(u.x, cs.x, sg * o.x * sn.x), fmaf(u.y, cs.y, sg * o.y * sn.y), fmaf(u.z, cs.z, sg * o.z * sn.z),
                                fmaf(u.w, cs.w, sg * o.w * sn.w));
              }
            } else {
#pragma unroll
              for (int b = 0; b < BATCH; ++b) {
                const int at = (FULL || t0 + b < toks ? t0 + b : 0) * hp;
                float* vp = &v[b][j].x;
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                  const int ch = c + i;
                  if (ch >= dims) continue;
                  const bool hi = ch >= half;
                  const int low = hi ? ch - half : ch;
                  const float o = swap[b * ROW + (hi ? low : ch + half)];
                  vp[i] = fmaf(vp[i], cosine[at + low], (hi ? o : -o) * sine[at + low]);
                }
              }
            }
          }
        }
        float ss[BATCH];
#pragma unroll
        for (int b = 0; b < BATCH; ++b) {
          ss[b] = 0.f;
#pragma unroll
          for (int j = 0; j < NJ; ++j) ss[b] += dot_four(v[b][j], v[b][j]);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1)
#pragma unroll
          for (int b = 0; b < BATCH; ++b) ss[b] += __shfl_xor_sync(0xffffffffu, ss[b], o);
#pragma unroll
        for (int b = 0; b < BATCH; ++b) {
          const float inv = rsqrtf(fmaf(ss[b], inv_d, a.eps));
#pragma unroll
          for (int j = 0; j < NJ; ++j) v[b][j] = mul_four(v[b][j], inv);
        }
      }
#pragma unroll
      for (int b = 0; b < BATCH; ++b) {
        if (!FULL && t0 + b >= toks) continue;
        const long long at = query ? static_cast<long long>(t0 + b) * a.H * a.P : place[t0 + b];
        if (at < 0) continue;
#pragma unroll
        for (int j = 0; j < NJ; ++j)
          if (4 * lane + 128 * j < a.P) store_four(dst0 + at, 4 * lane + 128 * j, v[b][j]);
      }
    };
    if constexpr (BATCH == 1) {
      batch(0, std::true_type{});
    } else {
#pragma unroll 1
      for (int t0 = 0; t0 < toks; t0 += BATCH) {
        if (t0 + BATCH <= toks) batch(t0, std::true_type{});
        else batch(t0, std::false_type{});
      }
    }
    // The last inputs become the state: by the tile with the segment's first tokens, the only reader of the old one.  A lane reads
    // and writes its own channels.  They are in the registers when the tile has the segment's last tokens too; else entry k takes
    // entry k + count, which is read before it is written.
    if (off == 0) {
      auto save = [&](int k, int j, float4 n) {
        const int c = 4 * lane + 128 * j;
        if (c >= d) return;
        T* dst = st + static_cast<size_t>(k) * p.ldw + wc;
        if (vec) {
          store_four(dst, c, n);
        } else {
          dst[c] = from_f<T>(n.x);
          if (c + 1 < d) dst[c + 1] = from_f<T>(n.y);
          if (c + 2 < d) dst[c + 2] = from_f<T>(n.z);
          if (c + 3 < d) dst[c + 3] = from_f<T>(n.w);
        }
      };
      if (TAPS > 0 && toks == count) {
#pragma unroll
        for (int k = 0; k < TAPS - 1; ++k)
#pragma unroll
          for (int j = 0; j < NJ; ++j) save(k, j, hist[k][j]);
      } else {
#pragma unroll 1
        for (int k = 0; k < hist_rows; ++k)
#pragma unroll
          for (int j = 0; j < NJ; ++j)
            if (4 * lane + 128 * j < d) save(k, j, input(count - hist_rows + k, j));
      }
    }
  }
}

template <typename T>
struct NormQkv {
  QkvPrep<T> a;
  const float* qw;            // [H d]
  const float* kw;            // [G d]
  const int* positions;
  float coef;                 // queries times 1 + coef ln(floor((position + 1) / every) + 1); every 0: no factor
  int every;
};

static constexpr int kNormWarps = 8;

// A block takes a token.
template <typename T>
__global__ void __launch_bounds__(32 * kNormWarps)
norm_qkv_kernel(const NormQkv<T> p) {
  __shared__ float part[2][kNormWarps];
  pdl_wait();
  pdl_launch_dependents();
  const QkvPrep<T>& a = p.a;
  const size_t t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* xr = a.x + t * a.ldx;
  const bool vec = a.vec;
  const int nq = a.H * a.d, nk = a.G * a.d;
  float ss[2] = {0.f, 0.f};
  for (int c = 4 * threadIdx.x; c < nq; c += 128 * kNormWarps) { const float4 v = load_four(xr + a.q_off, c, nq, vec); ss[0] += dot_four(v, v); }
  for (int c = 4 * threadIdx.x; c < nk; c += 128 * kNormWarps) { const float4 v = load_four(xr + a.k_off, c, nk, vec); ss[1] += dot_four(v, v); }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    ss[i] = warp_sum(ss[i]);
    if (lane == 0) part[i][warp] = ss[i];
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 2; ++i) ss[i] = warp_sum(lane < kNormWarps ? part[i][lane] : 0.f);
  float fq = 1.f / sqrtf(ss[0] / static_cast<float>(nq) + a.eps);
  const float fk = 1.f / sqrtf(ss[1] / static_cast<float>(nk) + a.eps);
  if (p.every > 0) fq *= fmaf(p.coef, logf(static_cast<float>((p.positions[t] + 1) / p.every + 1)), 1.f);
  const int slot = a.slots[t];
  for (int it = warp; it < a.H + 2 * a.G; it += kNormWarps) {
    T* dst = a.row(it, t, slot);
    if (!dst) continue;
    const int d = a.width(it);
    const T* src = xr + a.col(it);
    const float f = it < a.H ? fq : fk;
    const float* w = it < a.H ? p.qw + it * a.d : p.kw + (it - a.H) * a.d;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int c = 4 * lane + 128 * j;
      if (c >= a.P) continue;
      float4 v = load_four(src, c, d, vec);
      if (it < a.H + a.G) {
        const float4 g = load_four(w, c, d, vec);
        v = make_float4(v.x * f * g.x, v.y * f * g.y, v.z * f * g.z, v.w * f * g.w);
      }
      store_four(dst, c, v);
    }
  }
}

template <typename T>
struct HeadQkv {
  QkvPrep<T> a;
  const float* qw;            // [d]
  const float* kw;
  const float* freq;          // [2][pairs] radians per position, and what they were rounded by
  int pairs;
  const int* positions;
  int maps;                   // rows of d channels a head consists of; they share its P columns evenly
  int tokens;
};

static constexpr int kHeadBatch = 4;        // rows a group of lanes has in flight

// A block takes TOKS tokens and every gridDim.y-th of their rows; L lanes of four channels each take a row of 4 L columns (a query's
// or key's map) at a time.  Values are copied at the end.
template <typename T, int L, int TOKS>
__global__ void __launch_bounds__(32 * kQkvWarps)
head_qkv_kernel(const HeadQkv<T> p) {
  using Raw = typename RawFour<T>::type;
  extern __shared__ __align__(16) float lsm[];                         // cosines [TOKS][hp], sines
  constexpr int GROUPS = 32 * kQkvWarps / L, COLS = 4 * L;
  pdl_wait();
  pdl_launch_dependents();
  const QkvPrep<T>& a = p.a;
  const int t_first = blockIdx.x * TOKS, toks = min(TOKS, p.tokens - t_first);
  const int half = p.pairs, dims = 2 * half, hp = (half + 3) & ~3;
  float* cosine = lsm;
  float* sine = lsm + TOKS * hp;
  for (int i = threadIdx.x; i < toks * half; i += 32 * kQkvWarps) {
    const int t = TOKS == 1 ? 0 : i / half, j = i - t * half;
    // the rounding error of the product is put back: angles of far positions keep their fraction of a turn
    const float pos = static_cast<float>(p.positions[t_first + t]), f = p.freq[j];
    const float ang = pos * f, e = fmaf(pos, f, -ang) + pos * p.freq[half + j];
    float sn, cs;
    sincosf(ang, &sn, &cs);
    const float ce = fmaf(-0.5f * e, e, 1.f), se = e * fmaf(e * (-1.f / 6.f), e, 1.f);
    cosine[t * hp + j] = cs * ce - sn * se;
    sine[t * hp + j] = fmaf(sn, ce, cs * se);
  }
  __syncthreads();
  const int sub = threadIdx.x % L, group = threadIdx.x / L;
  const int lane0 = (threadIdx.x & 31) - sub;                          // first lane of the group
  const int c = 4 * sub;
  const bool vec = a.vec, vec_turn = (half & 3) == 0;
  const float inv_d = 1.f / static_cast<float>(a.d);
  const int nq = a.H * p.maps, rows = nq + a.G * p.maps;               // of a token
  const int stride = GROUPS * gridDim.y, first = blockIdx.y * GROUPS + group;
  // this lane's weights, and where its channels turn
  const float4 wq = load_four(p.qw, c, a.d, vec), wk = load_four(p.kw, c, a.d, vec);
  const bool hi = c >= half;
  const int low = hi ? c - half : c;
  // every group makes the same turns: its lanes exchange by shuffles
  const int units = toks * rows, turns = (units - static_cast<int>(blockIdx.y) * GROUPS + stride * kHeadBatch - 1) / (stride * kHeadBatch);
  for (int turn = 0; turn < turns; ++turn) {
    Raw raw[kHeadBatch];
    int tok[kHeadBatch], row[kHeadBatch];
#pragma unroll
    for (int b = 0; b < kHeadBatch; ++b) {
      const int u = first + (turn * kHeadBatch + b) * stride;
      const bool ok = u < units;
      tok[b] = ok ? (TOKS == 1 ? 0 : u / rows) : 0;
      row[b] = ok ? u - tok[b] * rows : -1;
      const int r = ok ? row[b] : 0;
      raw[b] = load_raw(a.x + static_cast<size_t>(t_first + tok[b]) * a.ldx + (r < nq ? a.q_off + r * a.d : a.k_off + (r - nq) * a.d), c, a.d, vec);
    }
#pragma unroll
    for (int b = 0; b < kHeadBatch; ++b) {
      float4 v = unpack_four(raw[b]);
      float ss = dot_four(v, v);
#pragma unroll
      for (int o = L / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const float inv = 1.f / sqrtf(fmaf(ss, inv_d, a.eps));
      const bool query = row[b] < nq;
      const float4 w = query ? wq : wk;
      v = make_float4(v.x * inv * w.x, v.y * inv * w.y, v.z * inv * w.z, v.w * inv * w.w);
      const float* cs = cosine + tok[b] * hp;
      const float* sn = sine + tok[b] * hp;
      if (vec_turn) {                                                  // four channels turn with four neighbours
        const int other = lane0 + (c < dims ? (hi ? c - half : c + half) >> 2 : sub);
        const float4 o = make_float4(__shfl_sync(0xffffffffu, v.x, other), __shfl_sync(0xffffffffu, v.y, other),
                                     __shfl_sync(0xffffffffu, v.z, other), __shfl_sync(0xffffffffu, v.w, other));
        if (c < dims) {
          const float sg = hi ? 1.f : -1.f;
          const float4 x = *reinterpret_cast<const float4*>(cs + low), y = *reinterpret_cast<const float4*>(sn + low);
          v = make_float4(fmaf(v.x, x.x, sg * o.x * y.x), fmaf(v.y, x.y, sg * o.y * y.y), fmaf(v.z, x.z, sg * o.z * y.z),
                          fmaf(v.w, x.w, sg * o.w * y.w));
        }
      } else {
        const float4 u = v;
        float* vp = &v.x;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int ch = c + i;
          const bool up = ch >= half;
          const int partner = ch < dims ? (up ? ch - half : ch + half) : ch, from = lane0 + (partner >> 2);
          const float o0 = __shfl_sync(0xffffffffu, u.x, from), o1 = __shfl_sync(0xffffffffu, u.y, from);
          const float o2 = __shfl_sync(0xffffffffu, u.z, from), o3 = __shfl_sync(0xffffffffu, u.w, from);
          if (ch >= dims) continue;
          const int e = partner & 3, j = up ? ch - half : ch;
          const float o = e == 0 ? o0 : e == 1 ? o1 : e == 2 ? o2 : o3;
          vp[i] = fmaf(vp[i], cs[j], (up ? o : -o) * sn[j]);
        }
      }
      if (row[b] < 0) continue;
      const int r = query ? row[b] : row[b] - nq, head = r / p.maps, map = r - head * p.maps;
      T* dst = a.row(query ? head : a.H + head, t_first + tok[b], a.slots[t_first + tok[b]]);
      if (dst) store_four(dst + map * COLS, c, v);
    }
  }
  const int quads = a.P >> 2;                                          // four columns of a value row at a time
  for (int i = blockIdx.y * 32 * kQkvWarps + threadIdx.x; i < toks * a.G * quads; i += 32 * kQkvWarps * gridDim.y) {
    const int qd = i % quads, tg = i / quads, g = tg % a.G, t = tg / a.G;
    T* dst = a.row(a.H + a.G + g, t_first + t, a.slots[t_first + t]);
    if (dst) store_four(dst, 4 * qd, load_four(a.x + static_cast<size_t>(t_first + t) * a.ldx + a.v_off + g * a.e, 4 * qd, a.e, vec));
  }
}

}  // namespace cb

extern "C" {

struct CbQkvPrep {
  const void* x; int ldx, q_off, k_off, v_off;
  void* q;
  void* cache;
  const void* slots;
  const void* positions;
  int H, G, d, e, P;
  float eps;
  int tokens, f32;
};

struct CbConvQkv {
  CbQkvPrep a;
  const void* w; int ldw, taps;
  void* state;
  const void* freq; int pairs;
};

struct CbNormQkv {
  CbQkvPrep a;
  const void* qw;
  const void* kw;
  float coef; int every;
};

struct CbHeadQkv {
  CbQkvPrep a;                // d: channels of a map
  const void* qw;
  const void* kw;
  const void* freq; int pairs;
  int maps;
};

}  // extern "C"

namespace cb {

static int qkv_check(const CbQkvPrep& a, int maps = 1) {
  if (a.H <= 0 || a.G <= 0 || a.d <= 0 || a.e <= 0 || a.P < maps * a.d || a.P < a.e || a.P > 256 || (a.P & 63)) return -10;
  if (a.q_off < 0 || a.k_off < a.q_off + a.H * maps * a.d || a.v_off < a.k_off + a.G * maps * a.d || a.ldx < a.v_off + a.G * a.e) return -11;
  return 0;
}

template <typename T>
static QkvPrep<T> qkv_fill(const CbQkvPrep& a) {
  QkvPrep<T> p;
  p.x = static_cast<const T*>(a.x); p.ldx = a.ldx; p.q_off = a.q_off; p.k_off = a.k_off; p.v_off = a.v_off;
  p.q = static_cast<T*>(a.q); p.cache = static_cast<T*>(a.cache); p.slots = static_cast<const int*>(a.slots);
  p.H = a.H; p.G = a.G; p.d = a.d; p.e = a.e; p.P = a.P; p.eps = a.eps;
  p.vec = ((a.d | a.e | a.ldx | a.q_off | a.k_off | a.v_off) & 3) == 0;
  return p;
}

}  // namespace cb

extern "C" {

int cb_conv_qkv(const CbConvQkv* c, const CbSegments* seg, void* stream) {
  using namespace cb;
  if (!c || !seg || seg->num <= 0 || c->a.tokens <= 0) return 0;
  if (const int rc = qkv_check(c->a)) return rc;
  if (c->taps < 1 || c->taps - 1 > kQkvTokens || c->pairs < 0 || 2 * c->pairs > c->a.d) return -12;
  if (c->ldw < c->a.v_off - c->a.q_off + c->a.G * c->a.e || (c->taps > 1 && !c->state) || !c->w || (c->pairs && !c->freq)) return -13;
  const int tiles = max_tiles(c->a.tokens, seg->num, kQkvTokens), items = c->a.H + 2 * c->a.G;
  // a head per warp where the tiles alone do not fill the device; the cosines are made once per block
  const int groups = (items + kQkvWarps - 1) / kQkvWarps;
  const bool one = c->a.P <= 128, single = c->a.tokens == seg->num;
  const int ny = min(groups, max(1, 148 * 24 / tiles));
  const int batch = c->taps > 4 ? 2 : single ? 1 : one ? 4 : 2, row = one && c->taps <= 4 ? 128 : 256;
  const size_t turns = static_cast<size_t>(batch == 1 ? 1 : kQkvTokens) * 2 * ((c->pairs + 3) & ~3);
  const size_t smem = (turns + static_cast<size_t>(kQkvWarps) * batch * row) * 4;
  auto go = [&](auto kernel, auto p) {
    using T = std::remove_pointer_t<decltype(p.a.q)>;
    p.a = qkv_fill<T>(c->a);
    p.a.vec = p.a.vec && (c->ldw & 3) == 0;
    p.w = static_cast<const float*>(c->w); p.ldw = c->ldw; p.taps = c->taps;
    p.state = static_cast<T*>(c->state);
    p.freq = static_cast<const float*>(c->freq); p.pairs = c->pairs;
    p.positions = static_cast<const int*>(c->a.positions);
    p.sg = make_segments(seg, c->a.tokens);
    return static_cast<int>(launch(kernel, dim3(tiles, ny), dim3(32 * kQkvWarps), smem, static_cast<cudaStream_t>(stream), p));
  };
  auto pick = [&](auto p) {
    using T = std::remove_pointer_t<decltype(p.a.q)>;
#define CB_TAPS(N)                                                                                            \
  case N:                                                                                                     \
    if (single) return one ? go(conv_qkv_kernel<T, N, 1, 1>, p) : go(conv_qkv_kernel<T, N, 2, 1>, p);         \
    return one ? go(conv_qkv_kernel<T, N, 1, 4>, p) : go(conv_qkv_kernel<T, N, 2, 2>, p);
    switch (c->taps) { CB_TAPS(1) CB_TAPS(2) CB_TAPS(3) CB_TAPS(4) }
#undef CB_TAPS
    return go(conv_qkv_kernel<T, 0, 2, 2>, p);
  };
  return c->a.f32 ? pick(ConvQkv<float>{}) : pick(ConvQkv<__nv_bfloat16>{});
}

int cb_norm_qkv(const CbNormQkv* c, void* stream) {
  using namespace cb;
  if (!c || c->a.tokens <= 0) return 0;
  if (const int rc = qkv_check(c->a)) return rc;
  if (!c->qw || !c->kw || c->every < 0) return -12;
  auto go = [&](auto kernel, auto p) {
    using T = std::remove_pointer_t<decltype(p.a.q)>;
    p.a = qkv_fill<T>(c->a);
    p.qw = static_cast<const float*>(c->qw); p.kw = static_cast<const float*>(c->kw);
    p.positions = static_cast<const int*>(c->a.positions);
    p.coef = c->coef; p.every = c->every;
    return static_cast<int>(launch(kernel, dim3(c->a.tokens), dim3(32 * kNormWarps), 0, static_cast<cudaStream_t>(stream), p));
  };
  return c->a.f32 ? go(norm_qkv_kernel<float>, NormQkv<float>{}) : go(norm_qkv_kernel<__nv_bfloat16>, NormQkv<__nv_bfloat16>{});
}

int cb_head_qkv(const CbHeadQkv* c, void* stream) {
  using namespace cb;
  if (!c || c->a.tokens <= 0) return 0;
  if (c->maps < 1 || c->maps > 2) return -12;
  if (const int rc = qkv_check(c->a, c->maps)) return rc;
  const int cols = c->a.P / c->maps;
  if (cols != 32 && cols != 64 && cols != 128) return -14;
  if (c->pairs < 0 || 2 * c->pairs > c->a.d || !c->qw || !c->kw || (c->pairs && !c->freq)) return -13;
  // few tokens: a token per block, and more blocks per token
  const bool single = c->a.tokens < 592;
  const int toks = single ? 1 : 8, tiles = (c->a.tokens + toks - 1) / toks;
  const int rows = (c->a.H + c->a.G) * c->maps * toks, groups = 32 * kQkvWarps / (cols / 4);
  const int ny = min((rows + groups * kHeadBatch - 1) / (groups * kHeadBatch), max(1, 148 * 8 / tiles));
  const size_t smem = static_cast<size_t>(toks) * 2 * ((c->pairs + 3) & ~3) * 4;
  auto go = [&](auto kernel, auto p) {
    using T = std::remove_pointer_t<decltype(p.a.q)>;
    p.a = qkv_fill<T>(c->a);
    p.qw = static_cast<const float*>(c->qw); p.kw = static_cast<const float*>(c->kw);
    p.freq = static_cast<const float*>(c->freq); p.pairs = c->pairs;
    p.positions = static_cast<const int*>(c->a.positions);
    p.maps = c->maps; p.tokens = c->a.tokens;
    return static_cast<int>(launch(kernel, dim3(tiles, ny), dim3(32 * kQkvWarps), smem, static_cast<cudaStream_t>(stream), p));
  };
  auto pick = [&](auto p) {
    using T = std::remove_pointer_t<decltype(p.a.q)>;
    if (cols == 32) return single ? go(head_qkv_kernel<T, 8, 1>, p) : go(head_qkv_kernel<T, 8, 8>, p);
    if (cols == 64) return single ? go(head_qkv_kernel<T, 16, 1>, p) : go(head_qkv_kernel<T, 16, 8>, p);
    return single ? go(head_qkv_kernel<T, 32, 1>, p) : go(head_qkv_kernel<T, 32, 8>, p);
  };
  return c->a.f32 ? pick(HeadQkv<float>{}) : pick(HeadQkv<__nv_bfloat16>{});
}

}  // extern "C"
