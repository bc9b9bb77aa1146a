// Grouped-query attention of the layered decoders over a paged cache in the activation type: a sliding window, first tokens that
// stay visible behind it, or chunks of positions; a bias per distance and head, a softmax entry without a value (sink), and the
// difference of two attention maps over the same values.
//
//   gqa_prepare_kernel    RMS norm of every query and key head, rotary positions on neighbouring channel pairs; keys and values
//                         to their page, where a value is the raw key of its token, as projected (qkv_prepare.cu has the others)
//   gqa_prefill_kernel    bf16: blocks of (token, head) rows of one key head on the tensor cores
//   gqa_decode_kernel,    bf16, one token per segment: the query heads of a key head are the rows, a warp walks whole pages;
//   gqa_merge_kernel      key splits are merged in split order
//   gqa_row_kernel        fp32 models: a warp per (token, head)
//
// The cache is [pages][key head][key, value][16][P], P the wider of the key and value widths rounded up to 64, zero columns behind
// the head.  With two maps (MAPS 2) a query or key row holds both, half of its columns each (P is 64, 128 or 256), and every (token,
// head) has a row of scores per map: rows of both maps share the keys and values a block has loaded, and the maps' outputs meet in
// the epilogue, where the difference is normed over the head and gated per channel.  Scores, softmax weights and sums are fp32; the weights are rounded to bf16 as the operand of the second product of the bf16 kernels.
#include <climits>
#include <type_traits>

#include "segments.cuh"
#include "launch.cuh"
#include "mma.cuh"

namespace cb {

static constexpr int kGqaPage = 16;
static constexpr float kLog2e = 1.4426950408889634f;

template <typename T>
struct GqaPrep {
  const T* x; int ldx;        // projections
  int q_off, k_off;           // columns of q [H d] and k [G d]
  const float* qw;            // [d]
  const float* kw;
  const float* freq;          // [pairs] radians per position
  float mult;                 // factor on cosine and sine
  const int* positions;       // [T]
  const int* slots;           // [T] cache row, < 0: none
  T* q;                       // [T, H, P]
  T* cache;
  int H, G, d, P, pairs;
  float eps;
};

template <typename T>
__global__ void __launch_bounds__(128)
gqa_prepare_kernel(const GqaPrep<T> p) {
  __shared__ float2 turn[128];
  pdl_wait();
  pdl_launch_dependents();
  const size_t t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (static_cast<int>(threadIdx.x) < p.pairs) {
    // the rounding error e of the product is put back (|e| < 0.04 up to a million radians): angles of far positions keep their
    // fraction of a turn
    const float pos = static_cast<float>(p.positions[t]), f = p.freq[threadIdx.x];
    const float a = pos * f, e = fmaf(pos, f, -a);
    float s, c;
    sincosf(a, &s, &c);
    const float ce = fmaf(-0.5f * e, e, 1.f), se = e * fmaf(e * (-1.f / 6.f), e, 1.f);
    turn[threadIdx.x] = make_float2((c * ce - s * se) * p.mult, fmaf(s, ce, c * se) * p.mult);
  }
  __syncthreads();
  const int slot = p.slots[t];
  const bool even = ((p.d | p.q_off | p.k_off | p.ldx) & 1) == 0;
  for (int hh = blockIdx.y * 4 + warp; hh < p.H + p.G; hh += 4 * gridDim.y) {
    const bool key = hh >= p.H;
    if (key && slot < 0) continue;
    const T* src = p.x + t * p.ldx + (key ? p.k_off + (hh - p.H) * p.d : p.q_off + hh * p.d);
    const float* w = key ? p.kw : p.qw;
    float2 v[4];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = 2 * (lane + 32 * i);
      v[i] = make_float2(0.f, 0.f);
      if (even) {
        if (c < p.d) {
          if constexpr (sizeof(T) == 2) v[i] = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(src + c));
          else v[i] = *reinterpret_cast<const float2*>(src + c);
        }
      } else {
        if (c < p.d) v[i].x = to_f(src[c]);
        if (c + 1 < p.d) v[i].y = to_f(src[c + 1]);
      }
      ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, ss));
    }
    const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(p.d) + p.eps);
    T* dst;
    if (key) {
      const size_t page = static_cast<size_t>(slot / kGqaPage), row = slot % kGqaPage;
      dst = p.cache + ((page * p.G + (hh - p.H)) * 2 * kGqaPage + row) * p.P;
    } else {
      dst = p.q + (t * p.H + hh) * p.P;
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int j = lane + 32 * i, c = 2 * j;
      if (c >= p.P) continue;
      float2 n = make_float2(c < p.d ? v[i].x * inv * w[c] : 0.f, c + 1 < p.d ? v[i].y * inv * w[c + 1] : 0.f);
      if (j < p.pairs) {
        const float2 r = turn[j];
        n = make_float2(n.x * r.x - n.y * r.y, fmaf(n.y, r.x, n.x * r.y));
      }
      T* val = dst + kGqaPage * p.P;
      if constexpr (sizeof(T) == 2) {
        *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16x2(n.x, n.y);
        if (key) *reinterpret_cast<uint32_t*>(val + c) = pack_bf16x2(v[i].x, v[i].y);
      } else {
        *reinterpret_cast<float2*>(dst + c) = n;
        if (key) *reinterpret_cast<float2*>(val + c) = v[i];
      }
    }
  }
}

template <typename T>
struct GqaAttn {
  const T* q;                 // [T, H, P]
  T* out; int ldo;            // [T, H d]
  const T* cache;
  const int* page_table;      // [slots, max_pages]
  int max_pages;
  int H, G, e, P, window;     // e: width of a value; window <= 0: every earlier token
  int keep;                   // the first tokens, visible whatever the window (0 without a window)
  int chunk;                  // > 0: a token sees its own chunk of positions only (no window then)
  float scale, out_scale;
  float sink;                 // score of the entry without a value, -inf: none
  const float* bias;          // [bias_far + 1, H] added to the scaled score by distance (the last row from bias_far on), null: none
  int bias_far;
  float less;                 // two maps: the second's output times this is taken from the first's, the difference o leaves as
  float eps;                  // o / sqrt(mean(o^2) + eps) * out_scale * sigmoid(gate)
  const T* gate; int ldg;     // [T, H e] logits
  Segments sg;

  // First key the token at `pos` sees (kept ones aside); it never decreases with the position
  __device__ __forceinline__ int first_key(int pos) const {
    return chunk > 0 ? pos - pos % chunk : window > 0 ? max(0, pos - window + 1) : 0;
  }
};

// Keys of a query tile from position pos0 on: the visible ones from `kmin` (a page's first key) on, and the kept ones below it, [0, kept)
struct GqaSpan {
  int kmin, kept;
  __device__ __forceinline__ GqaSpan(int first_key, int keep) {
    kmin = first_key & ~(kGqaPage - 1);
    kept = min(keep, kmin);
  }
};

__device__ __forceinline__ float sigmoid_of(float z) { return 1.f / (1.f + expf(-z)); }

// ------------------------------------------------------------------ fp32
template <int NR, int MAPS>
__global__ void __launch_bounds__(128)
gqa_row_kernel(const GqaAttn<float> p) {
  pdl_wait();
  pdl_launch_dependents();
  int s, off;
  if (!find_tile(p.sg, 1, blockIdx.x, s, off)) return;
  const int lane = threadIdx.x & 31;
  const int h = blockIdx.y * 4 + (threadIdx.x >> 5);
  if (h >= p.H) return;
  const int kh = h / (p.H / p.G);
  const size_t row = static_cast<size_t>(p.sg.row0[s]) + off;
  const int pos = p.sg.pos0[s] + off;
  const int lo = p.first_key(pos);
  const int* pages = p.page_table + static_cast<size_t>(p.sg.slot[s]) * p.max_pages;
  const float* qr = p.q + (row * p.H + h) * p.P;
  float q[NR], acc[MAPS][NR], m[MAPS], l[MAPS];
#pragma unroll
  for (int i = 0; i < NR; ++i) q[i] = qr[lane + 32 * i] * p.scale;
#pragma unroll
  for (int k = 0; k < MAPS; ++k) {
#pragma unroll
    for (int i = 0; i < NR; ++i) acc[k][i] = 0.f;
    m[k] = p.sink;
    l[k] = p.sink == -INFINITY ? 0.f : 1.f;
  }
  const int kept = min(p.keep, lo);
  for (int i = 0; i < kept + pos + 1 - lo; ++i) {
    const int j = i < kept ? i : lo + i - kept;
    const float* kr = p.cache + ((static_cast<size_t>(pages[j / kGqaPage]) * p.G + kh) * 2 * kGqaPage + j % kGqaPage) * p.P;
    const float* vr = kr + kGqaPage * p.P;
    float v[NR], sdot[MAPS] = {};
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      v[i] = vr[lane + 32 * i];
      sdot[i * MAPS / NR] = fmaf(q[i], kr[lane + 32 * i], sdot[i * MAPS / NR]);
    }
#pragma unroll
    for (int k = 0; k < MAPS; ++k) {
      sdot[k] = warp_sum(sdot[k]);
      if (p.bias) sdot[k] += __ldg(p.bias + static_cast<size_t>(min(pos - j, p.bias_far)) * p.H + h);
      const float mn = fmaxf(m[k], sdot[k]);
      const float f = expf(m[k] - mn), w = expf(sdot[k] - mn);
      m[k] = mn;
      l[k] = l[k] * f + w;
#pragma unroll
      for (int i = 0; i < NR; ++i) acc[k][i] = fmaf(w, v[i], acc[k][i] * f);
    }
  }
  float* orow = p.out + row * p.ldo + h * p.e;
  if constexpr (MAPS == 2) {
    const float i1 = 1.f / l[0], i2 = p.less / l[1];
    float ss = 0.f;                                     // columns behind the value are zero
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      acc[0][i] = acc[0][i] * i1 - acc[1][i] * i2;
      ss = fmaf(acc[0][i], acc[0][i], ss);
    }
    const float g = p.out_scale / sqrtf(warp_sum(ss) / static_cast<float>(p.e) + p.eps);
    const float* gr = p.gate + row * p.ldg + h * p.e;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int c = lane + 32 * i;
      if (c < p.e) orow[c] = acc[0][i] * g * sigmoid_of(gr[c]);
    }
  } else {
    const float g = p.out_scale / l[0];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int c = lane + 32 * i;
      if (c < p.e) orow[c] = acc[0][i] * g;
    }
  }
}

// ------------------------------------------------------------------ bf16, prompts and mixed steps
using bf16 = __nv_bfloat16;

__device__ __forceinline__ float ex2(float x) {       // 2^x, zero for -inf
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}

struct GqaMma {
  GqaAttn<bf16> a;
  int hb, qb;                 // heads and tokens of a block (hb * qb rows at most)
  int head_tiles;             // blocks of hb heads that share a key head
  int splits;
  int bias_rows;              // prompts: rows of the bias table kept in shared memory (bias_far + 1), 0: read in place
  float* partial;             // decode: [segment][key head tile][split][16][P + 2]
};
// Decode rows of a block are 16: the heads of a key head, with two maps eight heads' first maps and their second maps
template <int MAPS> constexpr int decode_heads() { return 16 / MAPS; }

__device__ __forceinline__ void store_pair(bf16* row, int c, int d, float x, float y) {
  if (c + 1 < d && (d & 1) == 0) {
    *reinterpret_cast<uint32_t*>(row + c) = pack_bf16x2(x, y);
  } else {
    if (c < d) row[c] = __float2bfloat16(x);
    if (c + 1 < d) row[c + 1] = __float2bfloat16(y);
  }
}

// Two channels of the normed and gated difference of two maps, written to a row of outputs (`gate`: the head's logits of the row)
__device__ __forceinline__ void store_gated_pair(bf16* row, const bf16* gate, int c, int e, float x, float y) {
  if (c + 1 < e && (e & 1) == 0) {
    const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gate + c));
    *reinterpret_cast<uint32_t*>(row + c) = pack_bf16x2(__fdividef(x, 1.f + __expf(-z.x)), __fdividef(y, 1.f + __expf(-z.y)));
  } else {
    if (c < e) row[c] = __float2bfloat16(__fdividef(x, 1.f + __expf(-to_f(gate[c]))));
    if (c + 1 < e) row[c + 1] = __float2bfloat16(__fdividef(y, 1.f + __expf(-to_f(gate[c + 1]))));
  }
}

// Four warps of 16 rows each, row = token * hb + head; key tiles of 64 keys in two buffers, 16-byte chunks XOR-swizzled by the
// row.  A warp keeps its rows' scores, weights and outputs in registers: no exchange between warps.  With two maps the first two
// warps have the first map's rows, the others the second's of the same (token, head); a warp's products run over its map's half of
// the columns, and the second map's outputs pass through shared memory once at the end.
static constexpr int kGqaWarps = 4;
static constexpr int kGqaBiasBytes = 11 << 10;      // three blocks of two column groups and their tables fit on an SM
template <int NCH, bool BIAS, int MAPS>
__global__ void __launch_bounds__(32 * kGqaWarps, NCH <= 2 ? 3 : 1)
gqa_prefill_kernel(const GqaMma p) {
  constexpr int P = NCH * 64, ROWB = P * 2, NW = kGqaWarps, MR = 16 * NW / MAPS, KT = 64, CH = P / 8, NT = P / 8;
  constexpr int KS = P / 16 / MAPS;                   // steps of a product over a map's columns
  static_assert(MAPS == 1 || (!BIAS && NCH != 3), "two maps take half of a row each");
  extern __shared__ __align__(128) uint8_t lsm[];
  constexpr bool QREG = NCH <= 2;                     // query fragments in registers; the rows pass through the second buffer
  uint8_t* kvs = lsm + (QREG ? 0 : MR * ROWB);        // [2 buffers][key, value][KT][ROWB]
  uint8_t* qs = QREG ? kvs + 2 * KT * ROWB : lsm;     // [MR][ROWB]
  float* table = reinterpret_cast<float*>(kvs + 4 * KT * ROWB);        // [bias_rows][hb], times log2 e
  pdl_wait();
  pdl_launch_dependents();
  const GqaAttn<bf16>& a = p.a;
  int s, off;
  if (!find_tile(a.sg, p.qb, blockIdx.x, s, off)) return;
  const int tid = threadIdx.x, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int warp = MAPS == 2 ? (tid >> 5) & 1 : tid >> 5, map = MAPS == 2 ? tid >> 6 : 0;     // warp: of the rows
  const int R = a.H / a.G, kh = blockIdx.y / p.head_tiles, hq0 = (blockIdx.y % p.head_tiles) * p.hb;
  const int heads = min(p.hb, R - hq0), h0 = kh * R + hq0;
  const int toks = min(p.qb, a.sg.count[s] - off);
  const size_t row0 = static_cast<size_t>(a.sg.row0[s]) + off;
  const int pos0 = a.sg.pos0[s] + off;
  const int* pages = a.page_table + static_cast<size_t>(a.sg.slot[s]) * a.max_pages;
  const GqaSpan span(a.first_key(pos0), a.keep);
  const int kmin = span.kmin, kept_tiles = (span.kept + KT - 1) / KT;
  const int kend = pos0 + toks;
  const int tiles = kept_tiles + (kend - kmin + KT - 1) / KT;
  // tiles of kept tokens come first; a tile's first key and the end of its keys
  auto tile_key = [&](int t) { return t < kept_tiles ? t * KT : kmin + (t - kept_tiles) * KT; };

  auto load_tile = [&](int t, int b) {
    const uint32_t dst0 = smem_u32(kvs + b * 2 * KT * ROWB);
#pragma unroll
    for (int i = 0; i < KT * CH / (32 * NW); ++i) {
      const int idx = tid + i * 32 * NW;
      const int r = idx / CH, c = idx % CH;
      const int key = tile_key(t) + r;
      const bool ok = key < (t < kept_tiles ? span.kept : kend);
      const int page = ok ? pages[key / kGqaPage] : 0;
      const bf16* src = a.cache + ((static_cast<size_t>(page) * a.G + kh) * 2 * kGqaPage + key % kGqaPage) * P + c * 8;
      const uint32_t at = dst0 + r * ROWB + ((c ^ (r & 7)) << 4);
      cp_async16(at, src, ok);
      cp_async16(at + KT * ROWB, src + kGqaPage * P, ok);
    }
  };
  if constexpr (BIAS) {
    for (int idx = tid; idx < p.bias_rows * p.hb; idx += 32 * NW) {
      const int n = idx / p.hb, h = idx - n * p.hb;
      table[idx] = h < heads ? __ldg(a.bias + static_cast<size_t>(n) * a.H + h0 + h) * kLog2e : 0.f;
    }
  }
  for (int idx = tid; idx < MR * CH; idx += 32 * NW) {
    const int r = idx / CH, c = idx % CH;
    const int tok = r / p.hb, h = r - tok * p.hb;
    const bool ok = tok < toks && h < heads;
    cp_async16(smem_u32(qs) + r * ROWB + ((c ^ (r & 7)) << 4),
               a.q + ((row0 + (ok ? tok : 0)) * a.H + h0 + (ok ? h : 0)) * P + c * 8, ok);
  }
  load_tile(0, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");

  // visible keys of the thread's two rows; rows without a query see none
  int lim_lo[2], lim_hi[2];
  // entries of the bias table (the one in shared memory, or the layer's): the rows' at distance 0 plus their position's, and the last
  const int bias_step = BIAS ? (p.bias_rows ? p.hb : a.H) : 0;
  int bias_at[2], bias_last[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = warp * 16 + g + 8 * i;
    const int tok = r / p.hb, h = r - tok * p.hb;
    lim_hi[i] = tok < toks && h < heads ? pos0 + tok : -1;
    lim_lo[i] = a.first_key(pos0 + tok);
    if constexpr (BIAS) {
      const int head = (h < heads ? h : 0) + (p.bias_rows ? 0 : h0);
      bias_at[i] = (pos0 + tok) * bias_step + head;
      bias_last[i] = a.bias_far * bias_step + head;
    }
  }
  // of the whole warp
  const int tok_a = min(warp * 16 / p.hb, toks - 1), tok_b = min((warp * 16 + 15) / p.hb, toks - 1);
  const bool idle = warp * 16 / p.hb >= toks;
  const int see_lo = a.first_key(pos0 + tok_a), see_hi = pos0 + tok_b;     // some row sees these
  const int all_lo = a.first_key(pos0 + tok_b), all_hi = pos0 + tok_a;     // every row sees these
  const float sc = a.scale * kLog2e;
  float m2[2] = {-INFINITY, -INFINITY}, l2[2] = {0.f, 0.f};
  float o[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int c = 0; c < 4; ++c) o[j][c] = 0.f;

  const uint32_t q_base = smem_u32(qs) + (warp * 16 + (lane & 15)) * ROWB;
  uint32_t q_at[4], k_at[4], v_at[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {                       // the swizzled chunk depends on the place inside a 128-byte group only
    q_at[i] = q_base + (((i * 2 + (lane >> 4)) ^ (lane & 7)) << 4);
    k_at[i] = ((lane & 7) + ((lane >> 4) << 3)) * ROWB + (((i * 2 + ((lane >> 3) & 1)) ^ (lane & 7)) << 4);
    v_at[i] = (lane & 15) * ROWB + (((i * 2 + (lane >> 4)) ^ (lane & 7)) << 4);
    if (MAPS == 2 && map) {                           // the second half of a row: four chunks, or whole 128-byte groups, on
      q_at[i] = NCH == 1 ? q_at[i] ^ 64 : q_at[i] + NCH * 64;
      k_at[i] = NCH == 1 ? k_at[i] ^ 64 : k_at[i] + NCH * 64;
    }
  }
  uint32_t qr[QREG ? KS : 1][4];
  if constexpr (QREG) {
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < KS; ++kk) ldsm4(qr[kk], q_at[kk & 3] + (kk >> 2) * 128);
    __syncthreads();
  }
  for (int t = 0; t < tiles; ++t) {
    const int b = t & 1;
    if (t + 1 < tiles) load_tile(t + 1, b ^ 1);       // its buffer was released by the barrier that ended the last turn
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    const int key_t = tile_key(t);
    const bool kept = t < kept_tiles;
    if (!idle && key_t <= see_hi && (key_t + KT > see_lo || key_t < a.keep)) {
      const uint32_t k_base = smem_u32(kvs + b * 2 * KT * ROWB), v_base = k_base + KT * ROWB;
      float sf[8][4];
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) sf[j][c] = 0.f;
#pragma unroll
      for (int kk = 0; kk < KS; ++kk) {
        uint32_t qa[4];
        if constexpr (QREG) { qa[0] = qr[kk][0]; qa[1] = qr[kk][1]; qa[2] = qr[kk][2]; qa[3] = qr[kk][3]; }
        else ldsm4(qa, q_at[kk & 3] + (kk >> 2) * 128);
#pragma unroll
        for (int j = 0; j < 8; j += 2) {
          uint32_t cb[4];
          ldsm4(cb, k_base + k_at[kk & 3] + (kk >> 2) * 128 + j * 8 * ROWB);
          mma_bf16(sf[j], qa, cb[0], cb[1]);
          mma_bf16(sf[j + 1], qa, cb[2], cb[3]);
        }
      }
      const bool whole = key_t >= all_lo && key_t + KT - 1 <= all_hi;
      float mx[2] = {m2[0], m2[1]};
      // a key is seen behind the window's start, or among the first tokens; a kept tile has no others
      const int seen_low = kept ? span.kept : a.keep;
      const int seen_from[2] = {kept ? INT_MAX : lim_lo[0], kept ? INT_MAX : lim_lo[1]};
      if constexpr (BIAS) {
        if (pos0 + tok_a - (key_t + KT - 1) >= a.bias_far) {             // the same for every distance of the tile
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const float far = p.bias_rows ? table[bias_last[i]] : __ldg(a.bias + bias_last[i]) * kLog2e;
#pragma unroll
            for (int j = 0; j < 8; ++j) {
              sf[j][2 * i] = fmaf(sf[j][2 * i], sc, far);
              sf[j][2 * i + 1] = fmaf(sf[j][2 * i + 1], sc, far);
            }
          }
        } else if (p.bias_rows && key_t + KT - 1 <= pos0 + tok_a && pos0 + (warp * 16 + 15) / p.hb - key_t <= a.bias_far) {
          // every distance has a row of its own: neighbouring keys are hb entries apart
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const float* row = table + bias_at[i] - (key_t + 2 * t4) * bias_step;
#pragma unroll
            for (int j = 0; j < 8; ++j) {
              sf[j][2 * i] = fmaf(sf[j][2 * i], sc, row[0]);
              sf[j][2 * i + 1] = fmaf(sf[j][2 * i + 1], sc, row[-bias_step]);
              row -= 8 * bias_step;
            }
          }
        } else {
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            int at = bias_at[i] - (key_t + 2 * t4) * bias_step;          // negative for keys that are not seen yet
#pragma unroll
            for (int j = 0; j < 8; ++j) {
              const int n0 = min(max(at, 0), bias_last[i]), n1 = min(max(at - bias_step, 0), bias_last[i]);
              const float b0 = p.bias_rows ? table[n0] : __ldg(a.bias + n0) * kLog2e;
              const float b1 = p.bias_rows ? table[n1] : __ldg(a.bias + n1) * kLog2e;
              sf[j][2 * i] = fmaf(sf[j][2 * i], sc, b0);
              sf[j][2 * i + 1] = fmaf(sf[j][2 * i + 1], sc, b1);
              at -= 8 * bias_step;
            }
          }
        }
      }
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const int key = key_t + j * 8 + 2 * t4 + (c & 1), i = c >> 1;
          const float v = BIAS ? sf[j][c] : sf[j][c] * sc;
          sf[j][c] = whole || ((key >= seen_from[i] || key < seen_low) && key <= lim_hi[i]) ? v : -INFINITY;
          mx[i] = fmaxf(mx[i], sf[j][c]);
        }
      float al[2], use[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
        mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
        use[i] = mx[i] == -INFINITY ? 0.f : mx[i];
        al[i] = ex2(m2[i] - use[i]);
        m2[i] = mx[i];
        l2[i] *= al[i];
      }
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          sf[j][c] = ex2(sf[j][c] - use[c >> 1]);
          l2[c >> 1] += sf[j][c];
        }
#pragma unroll
      for (int j = 0; j < NT; ++j) { o[j][0] *= al[0]; o[j][1] *= al[0]; o[j][2] *= al[1]; o[j][3] *= al[1]; }
#pragma unroll
      for (int ks = 0; ks < KT / 16; ++ks) {
        const uint32_t pa[4] = {pack_bf16x2(sf[2 * ks][0], sf[2 * ks][1]), pack_bf16x2(sf[2 * ks][2], sf[2 * ks][3]),
                                pack_bf16x2(sf[2 * ks + 1][0], sf[2 * ks + 1][1]), pack_bf16x2(sf[2 * ks + 1][2], sf[2 * ks + 1][3])};
#pragma unroll
        for (int j = 0; j < NT / 2; ++j) {
          uint32_t vb[4];
          ldsm4_t(vb, v_base + v_at[j & 3] + (j >> 2) * 128 + ks * 16 * ROWB);
          mma_bf16(o[2 * j], pa, vb[0], vb[1]);
          mma_bf16(o[2 * j + 1], pa, vb[2], vb[3]);
        }
      }
    }
    __syncthreads();                                  // the tile's buffer is free again
  }
  asm volatile("cp.async.wait_all;" ::: "memory");
  if constexpr (MAPS == 2) {
    constexpr int LD = P + 8;
    float* other = reinterpret_cast<float*>(kvs);      // [MR][LD]: what is taken away; nobody reads keys or values any more
    if (map) {
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        l2[i] += __shfl_xor_sync(0xffffffffu, l2[i], 1);
        l2[i] += __shfl_xor_sync(0xffffffffu, l2[i], 2);
        const float f = a.less / l2[i];
        float* row = other + (warp * 16 + g + 8 * i) * LD + 2 * t4;
#pragma unroll
        for (int j = 0; j < NT; ++j) *reinterpret_cast<float2*>(row + j * 8) = make_float2(o[j][2 * i] * f, o[j][2 * i + 1] * f);
      }
    }
    __syncthreads();
    if (map) return;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      l2[i] += __shfl_xor_sync(0xffffffffu, l2[i], 1);
      l2[i] += __shfl_xor_sync(0xffffffffu, l2[i], 2);
      const int r = warp * 16 + g + 8 * i;
      const int tok = r / p.hb, h = r - tok * p.hb;
      const float f = 1.f / l2[i];
      const float* sub = other + r * LD + 2 * t4;
      float ss = 0.f;                                  // columns behind the value are zero
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        const float2 u = *reinterpret_cast<const float2*>(sub + j * 8);
        o[j][2 * i] = o[j][2 * i] * f - u.x;
        o[j][2 * i + 1] = o[j][2 * i + 1] * f - u.y;
        ss = fmaf(o[j][2 * i], o[j][2 * i], fmaf(o[j][2 * i + 1], o[j][2 * i + 1], ss));
      }
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
      if (tok >= toks || h >= heads) continue;
      const float n = a.out_scale / sqrtf(ss / static_cast<float>(a.e) + a.eps);
      bf16* row = a.out + (row0 + tok) * a.ldo + (h0 + h) * a.e;
      const bf16* gate = a.gate + (row0 + tok) * a.ldg + (h0 + h) * a.e;
#pragma unroll
      for (int j = 0; j < NT; ++j) store_gated_pair(row, gate, j * 8 + 2 * t4, a.e, o[j][2 * i] * n, o[j][2 * i + 1] * n);
    }
    return;
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    l2[i] += __shfl_xor_sync(0xffffffffu, l2[i], 1);
    l2[i] += __shfl_xor_sync(0xffffffffu, l2[i], 2);
    const int r = warp * 16 + g + 8 * i;
    const int tok = r / p.hb, h = r - tok * p.hb;
    if (tok >= toks || h >= heads) continue;
    const float f = a.out_scale / (l2[i] + ex2(a.sink * kLog2e - m2[i]));
    bf16* row = a.out + (row0 + tok) * a.ldo + (h0 + h) * a.e;
#pragma unroll
    for (int j = 0; j < NT; ++j) store_pair(row, j * 8 + 2 * t4, a.e, o[j][2 * i] * f, o[j][2 * i + 1] * f);
  }
}

// ------------------------------------------------------------------ bf16, one token per segment
// Four warps deal the pages of a (segment, key head, split) among themselves; each has its own ring of kRing pages.  The rows of
// a product are the query heads of the key head (up to 16 of them); with two maps a query's row of the first map is zero in the
// second's columns and the other way round, so that one product makes both maps' scores.
static constexpr int kRing = 3;

// A head's output from its maps' outputs x1, x2 (columns 2 (lane + 32 i) of a warp) and their factors
template <int NCH>
__device__ __forceinline__ void store_difference(const GqaAttn<bf16>& a, size_t t, int h, int lane, const float2 (&x1)[NCH], float f1,
                                                 const float2 (&x2)[NCH], float f2) {
  float2 v[NCH];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NCH; ++i) {
    v[i] = make_float2(x1[i].x * f1 - x2[i].x * f2, x1[i].y * f1 - x2[i].y * f2);
    ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, ss));
  }
  const float n = a.out_scale / sqrtf(warp_sum(ss) / static_cast<float>(a.e) + a.eps);
#pragma unroll
  for (int i = 0; i < NCH; ++i)
    store_gated_pair(a.out + t * a.ldo + h * a.e, a.gate + t * a.ldg + h * a.e, 2 * (lane + 32 * i), a.e, v[i].x * n, v[i].y * n);
}

template <int NCH, bool BIAS, int MAPS>
__global__ void __launch_bounds__(128)
gqa_decode_kernel(const GqaMma p) {
  constexpr int P = NCH * 64, ROWB = P * 2, CH = P / 8, NT = P / 8, PAGEB = 2 * kGqaPage * ROWB;
  extern __shared__ __align__(128) uint8_t lsm[];     // [4 warps][kRing][key, value][16][ROWB], then the warps' results
  pdl_wait();
  pdl_launch_dependents();
  const GqaAttn<bf16>& a = p.a;
  const int s = blockIdx.x;
  if (a.sg.count[s] <= 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  constexpr int HB = decode_heads<MAPS>();
  const int R = a.H / a.G, kh = blockIdx.y / p.head_tiles, hq0 = (blockIdx.y % p.head_tiles) * HB;
  const int heads = min(HB, R - hq0), h0 = kh * R + hq0;
  const size_t row = a.sg.row0[s];
  const int pos = a.sg.pos0[s];
  const int* pages = a.page_table + static_cast<size_t>(a.sg.slot[s]) * a.max_pages;
  const int lo = a.first_key(pos);
  // the pages to walk: those with kept tokens below the window, then the window's
  const int pg_first = lo / kGqaPage, kept_pages = (min(a.keep, pg_first * kGqaPage) + kGqaPage - 1) / kGqaPage;
  const int skip = pg_first - kept_pages;             // pages between the two
  const int pg_all = pos / kGqaPage + 1 - skip, per = (pg_all + p.splits - 1) / p.splits;
  const int pg_lo = min(pg_all, static_cast<int>(blockIdx.z) * per), pg_hi = min(pg_all, pg_lo + per);
  uint8_t* ring = lsm + warp * kRing * PAGEB;

  auto load_page = [&](int at, int b) {               // nothing behind the last page
    if (at < pg_hi) {
      const bf16* src = a.cache + (static_cast<size_t>(pages[at < kept_pages ? at : at + skip]) * a.G + kh) * 2 * kGqaPage * P;
      const uint32_t dst0 = smem_u32(ring + b * PAGEB);
#pragma unroll
      for (int i = 0; i < 2 * kGqaPage * CH / 32; ++i) {
        const int idx = lane + i * 32;
        const int r = idx / CH, c = idx % CH;         // rows 0-15 keys, 16-31 values
        cp_async16(dst0 + r * ROWB + ((c ^ (r & 7)) << 4), src + r * P + c * 8, true);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int i = 0; i < kRing - 1; ++i) load_page(pg_lo + warp + 4 * i, i);
  uint32_t qa[P / 16][4];
#pragma unroll
  for (int kk = 0; kk < P / 16; ++kk)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int h = MAPS == 2 ? g : g + 8 * (i & 1), c = kk * 16 + 2 * t4 + 8 * (i >> 1);
      const bool in = MAPS == 1 || (kk >= P / 32) == ((i & 1) != 0);      // rows 8 .. 15 are the second maps
      qa[kk][i] = in && h < heads ? *reinterpret_cast<const uint32_t*>(a.q + (row * a.H + h0 + h) * P + c) : 0u;
    }
  const float sc = a.scale * kLog2e;
  float m2[2] = {-INFINITY, -INFINITY}, l2[2] = {0.f, 0.f};
  float o[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int c = 0; c < 4; ++c) o[j][c] = 0.f;
  uint32_t k_at[4], v_at[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    k_at[i] = ((lane & 7) + ((lane >> 4) << 3)) * ROWB + (((i * 2 + ((lane >> 3) & 1)) ^ (lane & 7)) << 4);
    v_at[i] = (lane & 15) * ROWB + (((i * 2 + (lane >> 4)) ^ (lane & 7)) << 4);
  }
  int b = 0;
  int bias_h[2] = {0, 0};
  float far[2] = {0.f, 0.f};
  if constexpr (BIAS) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      bias_h[i] = h0 + min(g + 8 * i, heads - 1);
      far[i] = __ldg(a.bias + static_cast<size_t>(a.bias_far) * a.H + bias_h[i]) * kLog2e;
    }
  }
  for (int at = pg_lo + warp; at < pg_hi; at += 4) {
    const int pg = at < kept_pages ? at : at + skip;
    load_page(at + 4 * (kRing - 1), (b + kRing - 1) % kRing);
    float bv[2][4];
    if constexpr (BIAS) {
      const bool near = pos - (pg * kGqaPage + kGqaPage - 1) < a.bias_far;
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          bv[j][c] = far[c >> 1];
          if (near) {
            const int n = min(max(pos - (pg * kGqaPage + j * 8 + 2 * t4 + (c & 1)), 0), a.bias_far);
            bv[j][c] = __ldg(a.bias + static_cast<size_t>(n) * a.H + bias_h[c >> 1]) * kLog2e;
          }
        }
    }
    asm volatile("cp.async.wait_group %0;" ::"n"(kRing - 1) : "memory");
    __syncwarp();
    const uint32_t k_base = smem_u32(ring + b * PAGEB), v_base = k_base + kGqaPage * ROWB;
    float sf[2][4] = {};
    float s2[2][4] = {};                              // two chains
#pragma unroll
    for (int kk = 0; kk < P / 16; ++kk) {
      uint32_t cb[4];
      ldsm4(cb, k_base + k_at[kk & 3] + (kk >> 2) * 128);
      mma_bf16(kk & 1 ? s2[0] : sf[0], qa[kk], cb[0], cb[1]);
      mma_bf16(kk & 1 ? s2[1] : sf[1], qa[kk], cb[2], cb[3]);
    }
    float mx[2] = {m2[0], m2[1]};
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int key = pg * kGqaPage + j * 8 + 2 * t4 + (c & 1);
        const float v = sf[j][c] + s2[j][c];
        sf[j][c] = (key >= lo || key < a.keep) && key <= pos ? (BIAS ? fmaf(v, sc, bv[j][c]) : v * sc) : -INFINITY;
        mx[c >> 1] = fmaxf(mx[c >> 1], sf[j][c]);
      }
    float use[2], al[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
      use[i] = mx[i] == -INFINITY ? 0.f : mx[i];
      al[i] = ex2(m2[i] - use[i]);
    }
    if (__any_sync(0xffffffffu, mx[0] > m2[0] || mx[1] > m2[1])) {
#pragma unroll
      for (int j = 0; j < NT; ++j) { o[j][0] *= al[0]; o[j][1] *= al[0]; o[j][2] *= al[1]; o[j][3] *= al[1]; }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      m2[i] = mx[i];
      l2[i] *= al[i];
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        sf[j][c] = ex2(sf[j][c] - use[c >> 1]);
        l2[c >> 1] += sf[j][c];
      }
    const uint32_t pa[4] = {pack_bf16x2(sf[0][0], sf[0][1]), pack_bf16x2(sf[0][2], sf[0][3]), pack_bf16x2(sf[1][0], sf[1][1]),
                            pack_bf16x2(sf[1][2], sf[1][3])};
#pragma unroll
    for (int j = 0; j < NT / 2; ++j) {
      uint32_t vb[4];
      ldsm4_t(vb, v_base + v_at[j & 3] + (j >> 2) * 128);
      mma_bf16(o[2 * j], pa, vb[0], vb[1]);
      mma_bf16(o[2 * j + 1], pa, vb[2], vb[3]);
    }
    __syncwarp();                                     // the page's buffer is free again
    b = b + 1 == kRing ? 0 : b + 1;
  }
  asm volatile("cp.async.wait_all;" ::: "memory");
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    l2[i] += __shfl_xor_sync(0xffffffffu, l2[i], 1);
    l2[i] += __shfl_xor_sync(0xffffffffu, l2[i], 2);
  }
  __syncthreads();                                    // all rings are done: their memory takes the warps' results
  constexpr int LD = P + 2;
  float* res = reinterpret_cast<float*>(lsm);         // [4][16][LD]: output columns, maximum, sum
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    float* dst = res + (warp * 16 + g + 8 * i) * LD;
#pragma unroll
    for (int j = 0; j < NT; ++j) *reinterpret_cast<float2*>(dst + j * 8 + 2 * t4) = make_float2(o[j][2 * i], o[j][2 * i + 1]);
    if (t4 == 0) *reinterpret_cast<float2*>(dst + P) = make_float2(m2[i], l2[i]);
  }
  __syncthreads();
  const size_t unit = static_cast<size_t>(s) * gridDim.y + blockIdx.y;
  // the warps' results of row r: maximum, sum and factors
  auto merge = [&](int r, float& mx, float& use, float& l, float (&f)[4]) {
    mx = -INFINITY;
    l = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) mx = fmaxf(mx, res[(w * 16 + r) * LD + P]);
    use = mx == -INFINITY ? 0.f : mx;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      f[w] = ex2(res[(w * 16 + r) * LD + P] - use);
      l += f[w] * res[(w * 16 + r) * LD + P + 1];
    }
  };
  if constexpr (MAPS == 2) {
    for (int r = warp; r < heads; r += 4) {
      float2 v[2][NCH];
      float l[2];
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        float mx, use, f[4];
        merge(r + 8 * k, mx, use, l[k], f);
#pragma unroll
        for (int i = 0; i < NCH; ++i) {
          v[k][i] = make_float2(0.f, 0.f);
#pragma unroll
          for (int w = 0; w < 4; ++w) {
            const float2 u = *reinterpret_cast<const float2*>(res + (w * 16 + r + 8 * k) * LD + 2 * (lane + 32 * i));
            v[k][i].x = fmaf(f[w], u.x, v[k][i].x);
            v[k][i].y = fmaf(f[w], u.y, v[k][i].y);
          }
        }
        if (p.splits > 1) {
          float* part = p.partial + ((unit * p.splits + blockIdx.z) * 16 + r + 8 * k) * LD;
#pragma unroll
          for (int i = 0; i < NCH; ++i) *reinterpret_cast<float2*>(part + 2 * (lane + 32 * i)) = v[k][i];
          if (lane == 0) *reinterpret_cast<float2*>(part + P) = make_float2(mx, l[k]);
        }
      }
      if (p.splits == 1) store_difference<NCH>(a, row, h0 + r, lane, v[0], 1.f / l[0], v[1], a.less / l[1]);
    }
    return;
  }
  for (int r = warp; r < heads; r += 4) {
    float mx, use, l, f[4];
    merge(r, mx, use, l, f);
    float* part = p.partial + ((unit * p.splits + blockIdx.z) * 16 + r) * LD;
    const float scale = p.splits > 1 ? 1.f : a.out_scale / (l + ex2(a.sink * kLog2e - use));
#pragma unroll
    for (int i = 0; i < P / 64; ++i) {
      const int c = 2 * (lane + 32 * i);
      float2 v = make_float2(0.f, 0.f);
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        const float2 u = *reinterpret_cast<const float2*>(res + (w * 16 + r) * LD + c);
        v.x = fmaf(f[w], u.x, v.x);
        v.y = fmaf(f[w], u.y, v.y);
      }
      if (p.splits > 1) *reinterpret_cast<float2*>(part + c) = v;
      else store_pair(a.out + row * a.ldo + (h0 + r) * a.e, c, a.e, v.x * scale, v.y * scale);
    }
    if (p.splits > 1 && lane == 0) *reinterpret_cast<float2*>(part + P) = make_float2(mx, l);
  }
}

// A warp per row of a unit.
template <int NCH, int MAPS>
__global__ void __launch_bounds__(128)
gqa_merge_kernel(const GqaMma p) {
  constexpr int P = NCH * 64, LD = P + 2;
  pdl_wait();
  pdl_launch_dependents();
  const GqaAttn<bf16>& a = p.a;
  const int s = blockIdx.x, lane = threadIdx.x & 31, r = blockIdx.z * 4 + (threadIdx.x >> 5);
  if (a.sg.count[s] <= 0) return;
  constexpr int HB = decode_heads<MAPS>();
  const int R = a.H / a.G, kh = blockIdx.y / p.head_tiles, hq0 = (blockIdx.y % p.head_tiles) * HB;
  if (r >= min(HB, R - hq0)) return;
  const size_t unit = static_cast<size_t>(s) * gridDim.y + blockIdx.y;
  constexpr int step = 16 * LD;
  // row `at` of the unit: sum over the splits, returns the sum of the weights
  auto merge = [&](int at, float2 (&v)[NCH]) {
    const float* part = p.partial + (unit * p.splits * 16 + at) * LD;
    float mx = a.sink * kLog2e;
    for (int z = 0; z < p.splits; ++z) mx = fmaxf(mx, part[z * step + P]);
    float l = ex2(a.sink * kLog2e - mx);
#pragma unroll
    for (int i = 0; i < NCH; ++i) v[i] = make_float2(0.f, 0.f);
    for (int z = 0; z < p.splits; ++z) {
      const float f = ex2(part[z * step + P] - mx);   // 0 for a split that saw no key
      l += f * part[z * step + P + 1];
#pragma unroll
      for (int i = 0; i < NCH; ++i) {
        const float2 u = *reinterpret_cast<const float2*>(part + z * step + 2 * (lane + 32 * i));
        v[i].x = fmaf(f, u.x, v[i].x);
        v[i].y = fmaf(f, u.y, v[i].y);
      }
    }
    return l;
  };
  const size_t t = static_cast<size_t>(a.sg.row0[s]);
  const int h = kh * R + hq0 + r;
  float2 v[NCH];
  const float l = merge(r, v);
  if constexpr (MAPS == 2) {
    float2 v2[NCH];
    const float l2 = merge(r + 8, v2);
    store_difference<NCH>(a, t, h, lane, v, 1.f / l, v2, a.less / l2);
  } else {
    const float f = a.out_scale / l;
    bf16* row = a.out + t * a.ldo + h * a.e;
#pragma unroll
    for (int i = 0; i < NCH; ++i) store_pair(row, 2 * (lane + 32 * i), a.e, v[i].x * f, v[i].y * f);
  }
}

// ------------------------------------------------------------------ host
// `most`: shared memory of the largest launch (0: of every launch)
template <typename K>
static int gqa_go(K kernel, dim3 grid, int threads, size_t smem, const GqaMma& p, bool (&configured)[64], cudaStream_t st, size_t most = 0) {
  int dev = 0;                                        // dynamic shared memory is configured once per device
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -18;
  if (!configured[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(most ? most : smem));
    if (e != cudaSuccess) return static_cast<int>(e);
    configured[dev] = true;
  }
  return static_cast<int>(launch(kernel, grid, dim3(threads), smem, st, p));
}

template <int NCH, bool BIAS, int MAPS>
static int gqa_prefill(const GqaMma& p, dim3 grid, cudaStream_t st) {
  static bool configured[64] = {};
  const size_t rows = static_cast<size_t>((NCH <= 2 ? 0 : 16 * kGqaWarps / MAPS) + 256) * NCH * 128;
  return gqa_go(gqa_prefill_kernel<NCH, BIAS, MAPS>, grid, 32 * kGqaWarps, rows + (BIAS ? static_cast<size_t>(p.bias_rows) * p.hb * 4 : 0), p,
                configured, st, rows + (BIAS ? kGqaBiasBytes : 0));
}

template <int NCH, bool BIAS, int MAPS>
static int gqa_decode(const GqaMma& p, dim3 grid, cudaStream_t st) {
  static bool configured[64] = {};
  const int rc = gqa_go(gqa_decode_kernel<NCH, BIAS, MAPS>, grid, 128, static_cast<size_t>(4) * kRing * 2 * kGqaPage * NCH * 128, p, configured, st);
  if (rc || p.splits == 1) return rc;
  return static_cast<int>(launch(gqa_merge_kernel<NCH, MAPS>, dim3(grid.x, grid.y, 4 / MAPS), dim3(128), 0, st, p));
}

template <bool BIAS, int MAPS>
static int gqa_mma(const GqaMma& p, int nch, bool decode, dim3 grid, cudaStream_t st) {
  switch (nch) {
    case 1: return decode ? gqa_decode<1, BIAS, MAPS>(p, grid, st) : gqa_prefill<1, BIAS, MAPS>(p, grid, st);
    case 2: return decode ? gqa_decode<2, BIAS, MAPS>(p, grid, st) : gqa_prefill<2, BIAS, MAPS>(p, grid, st);
    case 3:
      if constexpr (MAPS == 1) return decode ? gqa_decode<3, BIAS, 1>(p, grid, st) : gqa_prefill<3, BIAS, 1>(p, grid, st);
      return -15;
  }
  return decode ? gqa_decode<4, BIAS, MAPS>(p, grid, st) : gqa_prefill<4, BIAS, MAPS>(p, grid, st);
}
static int gqa_mma_any(const GqaMma& p, int nch, bool decode, dim3 grid, cudaStream_t st) {
  if (p.a.gate) return gqa_mma<false, 2>(p, nch, decode, grid, st);
  return p.a.bias ? gqa_mma<true, 1>(p, nch, decode, grid, st) : gqa_mma<false, 1>(p, nch, decode, grid, st);
}

}  // namespace cb

extern "C" {

struct CbGqaPrep {
  const void* x; int ldx, q_off, k_off;
  const void* qw;
  const void* kw;
  const void* freq;
  float mult;
  const void* positions;
  const void* slots;
  void* q;
  void* cache;
  int H, G, d, P, pairs;
  float eps;
  int tokens, f32;
};

struct CbGqaAttn {
  const void* q;
  void* out; int ldo;
  const void* cache;
  const void* page_table;
  int max_pages, H, G, e, P, window, keep, chunk;
  float scale, out_scale, sink;
  const void* bias;           // fp32 [bias_far + 1, H] or null
  int bias_far;
  const void* gate; int ldg;  // two maps: gate logits [T, H e] of their difference (null: one map), see GqaAttn
  float less, eps;
  int tokens, f32;
  int decode;                 // every segment has at most one row, row s belongs to segment s
  int splits;                 // key splits of the decode form (1 = none)
  void* partial;              // fp32 scratch of cb_gqa_attn_partial_floats elements (splits > 1)
};

// Scratch of a split decode launch; `units` receives the blocks of one split.
long long cb_gqa_attn_partial_floats(int tokens, int segs, int H, int G, int P, int maps, int decode, int splits, int* units) {
  if (!decode) return 0;
  const int hb = 16 / maps;
  const long long n = static_cast<long long>(segs) * G * ((H / G + hb - 1) / hb);
  if (units) *units = static_cast<int>(n);
  return splits > 1 ? n * splits * 16 * (P + 2) : 0;
}

int cb_gqa_prepare(const CbGqaPrep* a, void* stream) {
  using namespace cb;
  if (!a || a->tokens <= 0) return 0;
  if (a->H <= 0 || a->G <= 0 || a->d <= 0 || a->P < a->d || a->P > 256 || (a->P & 63) || a->pairs < 0 || 2 * a->pairs > a->d) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  // few tokens: more blocks per token
  const int ny = a->tokens >= 1024 ? 1 : min((a->H + a->G + 3) / 4, 8);
  auto go = [&](auto kernel, auto p) {
    using T = std::remove_pointer_t<decltype(p.q)>;
    p.x = static_cast<const T*>(a->x); p.ldx = a->ldx; p.q_off = a->q_off; p.k_off = a->k_off;
    p.qw = static_cast<const float*>(a->qw); p.kw = static_cast<const float*>(a->kw);
    p.freq = static_cast<const float*>(a->freq); p.mult = a->mult;
    p.positions = static_cast<const int*>(a->positions); p.slots = static_cast<const int*>(a->slots);
    p.q = static_cast<T*>(a->q); p.cache = static_cast<T*>(a->cache);
    p.H = a->H; p.G = a->G; p.d = a->d; p.P = a->P; p.pairs = a->pairs; p.eps = a->eps;
    return static_cast<int>(launch(kernel, dim3(a->tokens, ny), dim3(128), 0, st, p));
  };
  return a->f32 ? go(gqa_prepare_kernel<float>, GqaPrep<float>{}) : go(gqa_prepare_kernel<bf16>, GqaPrep<bf16>{});
}

int cb_gqa_attn(const CbGqaAttn* a, const CbSegments* seg, void* stream) {
  using namespace cb;
  if (!a || !seg || seg->num <= 0 || a->tokens <= 0) return 0;
  if (a->H <= 0 || a->G <= 0 || (a->H % a->G) || a->e <= 0 || a->P < a->e || a->P > 256 || (a->P & 63) || a->ldo < a->H * a->e) return -10;
  if (a->keep < 0 || (a->bias && a->bias_far < 0) || a->chunk < 0 || (a->chunk && (a->window > 0 || a->keep))) return -13;
  if (a->gate && (a->bias || a->P == 192 || a->ldg < a->H * a->e || a->sink != -INFINITY)) return -14;
  const int maps = a->gate ? 2 : 1;
  if (a->splits > 1 && (!a->decode || !a->partial || a->splits > 65535)) return -12;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  auto fill = [&](auto& p) {
    using T = std::remove_pointer_t<decltype(p.out)>;
    p.q = static_cast<const T*>(a->q);
    p.out = static_cast<T*>(a->out); p.ldo = a->ldo;
    p.cache = static_cast<const T*>(a->cache);
    p.page_table = static_cast<const int*>(a->page_table); p.max_pages = a->max_pages;
    p.H = a->H; p.G = a->G; p.e = a->e; p.P = a->P; p.window = a->window;
    p.keep = a->window > 0 ? a->keep : 0;
    p.chunk = a->chunk;
    p.gate = static_cast<const T*>(a->gate); p.ldg = a->ldg; p.less = a->less; p.eps = a->eps;
    p.bias = static_cast<const float*>(a->bias); p.bias_far = a->bias_far;
    p.scale = a->scale; p.out_scale = a->out_scale; p.sink = a->sink;
    p.sg = make_segments(seg, a->tokens);
  };
  if (a->f32) {
    GqaAttn<float> p;
    fill(p);
    const dim3 grid(a->tokens, (a->H + 3) / 4);
    auto row = [&](auto one, auto two) { return static_cast<int>(launch(maps == 2 ? two : one, grid, dim3(128), 0, st, p)); };
    switch (a->P / 64) {
      case 1: return row(gqa_row_kernel<2, 1>, gqa_row_kernel<2, 2>);
      case 2: return row(gqa_row_kernel<4, 1>, gqa_row_kernel<4, 2>);
      case 3: return static_cast<int>(launch(gqa_row_kernel<6, 1>, grid, dim3(128), 0, st, p));
    }
    return row(gqa_row_kernel<8, 1>, gqa_row_kernel<8, 2>);
  }
  GqaMma p;
  fill(p.a);
  p.splits = a->splits > 1 ? a->splits : 1;
  p.bias_rows = 0;
  p.partial = static_cast<float*>(a->partial);
  if (a->decode) {
    p.hb = 16 / maps; p.qb = 1;
    p.head_tiles = (a->H / a->G + p.hb - 1) / p.hb;
    const dim3 grid(seg->num, a->G * p.head_tiles, p.splits);
    if (grid.y > 65535) return -11;
    return gqa_mma_any(p, a->P / 64, true, grid, st);
  }
  const int R = a->H / a->G;
  p.hb = min(R, 16 * kGqaWarps / maps);
  p.qb = 16 * kGqaWarps / maps / p.hb;
  p.head_tiles = (R + p.hb - 1) / p.hb;
  const dim3 grid(max_tiles(a->tokens, seg->num, p.qb), a->G * p.head_tiles);
  if (grid.y > 65535) return -11;
  const long long rows = static_cast<long long>(a->bias_far) + 1;
  p.bias_rows = a->bias && rows * p.hb * 4 <= kGqaBiasBytes ? static_cast<int>(rows) : 0;
  return gqa_mma_any(p, a->P / 64, false, grid, st);
}

}  // extern "C"
