// Latent attention over a paged cache of latents, with a sliding window, a gate per head and a rotated key part, each of them optional.
//
// A token's cache row is its latent c (R channels, one row for all heads).  A head's key is W_uk c and its value W_uv c,
// so its scores are (W_uk^T q) . c: the runner multiplies the queries by W_uk^T once (a block-diagonal product), the
// attention below runs on latents for all heads at once, and W_uv is applied to its output.  A rotated key part that the heads share
// lies behind the latent in the same row, and the rotated part of a query behind its latent part: one product makes both scores.
// The output is taken over the latent's columns only.
//
//   latent_prepare_kernel   RMS norms of the query latent and of the cache latent, rotations; the cache row is written to its page
//   latent_attn_mma_kernel, latent_merge_kernel  bf16 rows on the tensor cores: 32 or 64 (token, head) rows share every latent they read
//   latent_attn_kernel      a warp per (token, head), fp32 arithmetic on rows of either type (32-bit models; wide latents)
//
// The cache is [pages][16][Rp], zero columns behind what a row holds.  (Rp, Rv): columns of a row and of the output, see
// cb_latent_attn_mma; other widths up to 1024 are served by the warp form.
#include <type_traits>

#include "segments.cuh"
#include "launch.cuh"
#include "mma.cuh"

namespace cb {

static constexpr int kLatentPage = 16;

template <typename T>
struct LatentPrep {
  const T* proj; int ldp;
  int q_off, q_rank;          // query latent (0: none)
  int c_off, R;               // cache latent
  const float* qw;
  const float* cw;
  T* cq; int ldq;
  T* cache; int Rp;
  const int* slots;           // [T] cache row, < 0: none
  int qr_off, r_off;          // rotated parts: the queries' [H, 2 pairs], the key's [2 pairs]
  int col, pairs;             // column of a row they go to; 0 pairs: none
  const float* freq;          // [2][pairs] radians per position, and what they were rounded by
  float mult;                 // factor on cosine and sine
  const int* positions;
  T* ql;                      // [T, H, Rp]
  int H;
  float eps;
};

static constexpr int kMaxRotPairs = 128;

template <typename T>
__global__ void __launch_bounds__(128)
latent_prepare_kernel(const LatentPrep<T> p) {
  __shared__ float red[2][4];
  __shared__ float2 turn[kMaxRotPairs];
  pdl_wait();
  pdl_launch_dependents();
  const size_t t = blockIdx.x;
  const T* pr = p.proj + t * p.ldp;
  const T* qr = pr + p.q_off;
  const T* cr = pr + p.c_off;
  if (static_cast<int>(threadIdx.x) < p.pairs) {
    // the rounding error of the product is put back: angles of far positions keep their fraction of a turn
    const float pos = static_cast<float>(p.positions[t]), f = p.freq[threadIdx.x];
    const float a = pos * f, e = fmaf(pos, f, -a) + pos * p.freq[p.pairs + threadIdx.x];
    float s, c;
    sincosf(a, &s, &c);
    const float ce = fmaf(-0.5f * e, e, 1.f), se = e * fmaf(e * (-1.f / 6.f), e, 1.f);
    turn[threadIdx.x] = make_float2((c * ce - s * se) * p.mult, fmaf(s, ce, c * se) * p.mult);
  }
  const int slot = p.slots[t];
  // blockIdx.y > 0 takes rotated queries only; the first block also has the norms and the key
  float sq = 0.f, sc = 0.f;
  if (blockIdx.y == 0) {
    for (int c = threadIdx.x; c < p.q_rank; c += 128) { const float v = to_f(qr[c]); sq = fmaf(v, v, sq); }
    for (int c = threadIdx.x; c < p.R; c += 128) { const float v = to_f(cr[c]); sc = fmaf(v, v, sc); }
    sq = warp_sum(sq);
    sc = warp_sum(sc);
    if ((threadIdx.x & 31) == 0) { red[0][threadIdx.x >> 5] = sq; red[1][threadIdx.x >> 5] = sc; }
  }
  __syncthreads();
  const int half = p.pairs;
  // two neighbouring channels; rows start at even elements
  auto rotate = [&](const T* src, T* dst, int i) {
    const float2 r = turn[i];
    float u, v;
    if constexpr (sizeof(T) == 2) {
      const float2 w = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(src + 2 * i));
      u = w.x; v = w.y;
    } else {
      const float2 w = *reinterpret_cast<const float2*>(src + 2 * i);
      u = w.x; v = w.y;
    }
    const float a = u * r.x - v * r.y, b = fmaf(v, r.x, u * r.y);
    if constexpr (sizeof(T) == 2) *reinterpret_cast<uint32_t*>(dst + 2 * i) = pack_bf16x2(a, b);
    else *reinterpret_cast<float2*>(dst + 2 * i) = make_float2(a, b);
  };
  for (int idx = blockIdx.y * 128 + threadIdx.x; idx < p.H * half; idx += 128 * gridDim.y) {
    const int h = idx / half, i = idx - h * half;
    rotate(pr + p.qr_off + h * 2 * half, p.ql + (t * p.H + h) * p.Rp + p.col, i);
  }
  if (blockIdx.y) return;
  sq = red[0][0] + red[0][1] + red[0][2] + red[0][3];
  sc = red[1][0] + red[1][1] + red[1][2] + red[1][3];
  if (p.q_rank) {
    const float iq = 1.f / sqrtf(sq / static_cast<float>(p.q_rank) + p.eps);
    for (int c = threadIdx.x; c < p.q_rank; c += 128) p.cq[t * p.ldq + c] = from_f<T>(to_f(qr[c]) * iq * p.qw[c]);
  }
  if (slot < 0) return;                                  // padding row
  const float ic = 1.f / sqrtf(sc / static_cast<float>(p.R) + p.eps);
  T* dst = p.cache + static_cast<size_t>(slot) * p.Rp;
  for (int c = threadIdx.x; c < p.R; c += 128) dst[c] = from_f<T>(to_f(cr[c]) * ic * p.cw[c]);
  if (static_cast<int>(threadIdx.x) < half) rotate(pr + p.r_off, dst + p.col, threadIdx.x);
}

template <typename T>
struct LatentAttn {
  const T* q;             // [T, H, Rp] queries in latent space
  T* out;                 // [T, H, Rv]
  const T* cache;         // [pages, 16, Rp]
  const T* gate; int ldg; // [T, H] gate logits: the output is multiplied by their sigmoid; null: none
  const int* page_table;  // [slots, max_pages]
  int max_pages;
  int H, Rp, Rv, window;  // window <= 0: every earlier token
  float scale;
  Segments sg;

  __device__ __forceinline__ float gate_at(size_t t, int h) const { return gate ? 1.f / (1.f + expf(-to_f(gate[t * ldg + h]))) : 1.f; }
};

template <typename T, int NR>
__global__ void __launch_bounds__(128)
latent_attn_kernel(const LatentAttn<T> p) {
  pdl_wait();
  pdl_launch_dependents();
  int s, off;
  if (!find_tile(p.sg, 1, blockIdx.x, s, off)) return;
  const int lane = threadIdx.x & 31;
  const int h = blockIdx.y * 4 + (threadIdx.x >> 5);
  if (h >= p.H) return;
  const size_t row = static_cast<size_t>(p.sg.row0[s]) + off;
  const int pos = p.sg.pos0[s] + off;
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int* pages = p.page_table + static_cast<size_t>(p.sg.slot[s]) * p.max_pages;
  const T* qr = p.q + (row * p.H + h) * p.Rp;
  float q[NR], acc[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int c = lane + 32 * i;
    q[i] = c < p.Rp ? to_f(qr[c]) * p.scale : 0.f;
    acc[i] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  for (int j = lo; j <= pos; ++j) {
    const T* cr = p.cache + (static_cast<size_t>(pages[j / kLatentPage]) * kLatentPage + (j % kLatentPage)) * p.Rp;
    float c[NR], sdot = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int col = lane + 32 * i;
      c[i] = col < p.Rp ? to_f(cr[col]) : 0.f;
      sdot = fmaf(q[i], c[i], sdot);
    }
    sdot = warp_sum(sdot);
    const float mn = fmaxf(m, sdot);
    const float f = expf(m - mn), w = expf(sdot - mn);
    m = mn;
    l = l * f + w;
#pragma unroll
    for (int i = 0; i < NR; ++i) acc[i] = fmaf(w, c[i], acc[i] * f);
  }
  const float g = p.gate_at(row, h) / l;
  T* orow = p.out + (row * p.H + h) * p.Rv;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int c = lane + 32 * i;
    if (c < p.Rv) orow[c] = from_f<T>(acc[i] * g);
  }
}

// ------------------------------------------------------------------ tensor-core form
// MR query rows per block: consecutive tokens of one segment x the heads of a head group, row = token * hb + head.  Key
// tiles of KT rows arrive by cp.async in two buffers (16-byte chunks XOR-swizzled by the row, so that ldmatrix reads
// both orientations without bank conflicts): the same tile is the key operand of S = Q C^T and the value operand of
// O += P C.  Eight warps: for S they form MR / 16 x 128 / MR (rows x keys); for O every warp owns Rv / 8 latent columns
// of all rows, so a value fragment is read once per block.  Scores, softmax weights and sums are fp32; the weights are
// rounded to bf16 as the operand of the second product.  With splits > 1 the key tiles are dealt to grid.z blocks and
// latent_merge_kernel adds their partial results in split order.  The 32-row form (decode) takes key tiles of 32, so that
// two blocks share an SM and one's loads overlap the other's products.

struct LatentMma {
  LatentAttn<__nv_bfloat16> a;
  int hb, qb;             // heads of a block, tokens of a block (hb * qb <= MR)
  int splits;
  float* partial;         // [tile][head group][split][MR][Rv + 2]
};

template <int MR> constexpr int key_tile() { return MR == 32 ? 32 : 64; }

template <int MR, int NCH, int NV>
__global__ void __launch_bounds__(256, MR == 32 ? 2 : 1)
latent_attn_mma_kernel(const LatentMma p) {
  constexpr int RP = NCH * 64, RV = NV * 64, ROWB = RP * 2;        // bytes of a cached row
  constexpr int PB = key_tile<MR>() * 2;             // bytes of a row of softmax weights
  constexpr int kKeyTile = key_tile<MR>();
  constexpr int MT = MR / 16, WN = 8 / MT;           // S: MT x WN warps
  constexpr int NS = kKeyTile / WN / 8;              // n8 key tiles of a warp in S
  constexpr int NT = NV;                             // n8 column tiles of a warp in O
  extern __shared__ __align__(128) uint8_t lsm[];
  uint8_t* qs = lsm;                                 // [MR][ROWB]
  uint8_t* cs = qs + MR * ROWB;                      // [2][key tile][ROWB]
  uint8_t* ps = cs + 2 * kKeyTile * ROWB;            // [MR][PB], 16-byte chunks XOR-swizzled over 128 bytes
  float* alpha = reinterpret_cast<float*>(ps + MR * PB);   // [MR]
  float* pmax = alpha + MR;                          // [WN][MR]
  float* lsum = pmax + WN * MR;                      // [WN][MR]
  float* mrow = lsum + WN * MR;                      // [MR]
  pdl_wait();
  pdl_launch_dependents();
  const LatentAttn<__nv_bfloat16>& a = p.a;
  int s, off;
  if (!find_tile(a.sg, p.qb, blockIdx.x, s, off)) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int h0 = blockIdx.y * p.hb;
  const int heads = min(p.hb, a.H - h0);
  const int toks = min(p.qb, a.sg.count[s] - off);
  const size_t row0 = static_cast<size_t>(a.sg.row0[s]) + off;
  const int pos0 = a.sg.pos0[s] + off;
  const int* pages = a.page_table + static_cast<size_t>(a.sg.slot[s]) * a.max_pages;
  // keys any row of the block sees, from a page boundary on
  const int kmin = a.window > 0 ? max(0, pos0 - a.window + 1) & ~(kLatentPage - 1) : 0;
  const int kend = pos0 + toks;                      // first key nobody sees
  const int tiles = (kend - kmin + kKeyTile - 1) / kKeyTile;
  const int per = (tiles + p.splits - 1) / p.splits;
  const int t_lo = min(tiles, static_cast<int>(blockIdx.z) * per), t_hi = min(tiles, t_lo + per);

  auto load_tile = [&](int t, int b) {
    const uint32_t dst0 = smem_u32(cs + b * kKeyTile * ROWB);
    constexpr int CH = RP / 8;                       // 16-byte chunks of a row
#pragma unroll
    for (int i = 0; i < kKeyTile * CH / 256; ++i) {
      const int idx = tid + i * 256;
      const int r = idx / CH, c = idx % CH;
      const int key = kmin + t * kKeyTile + r;
      const bool ok = key < kend;
      const int page = ok ? pages[key / kLatentPage] : 0;
      cp_async16(dst0 + r * ROWB + ((c ^ (r & 7)) << 4),
                 a.cache + (static_cast<size_t>(page) * kLatentPage + (key % kLatentPage)) * RP + c * 8, ok);
    }
  };
  {
    constexpr int CH = RP / 8;
    const uint32_t dst0 = smem_u32(qs);
    for (int idx = tid; idx < MR * CH; idx += 256) {
      const int r = idx / CH, c = idx % CH;
      const int tok = r / p.hb, h = r - tok * p.hb;
      const bool ok = tok < toks && h < heads;
      cp_async16(dst0 + r * ROWB + ((c ^ (r & 7)) << 4),
                 a.q + ((row0 + (ok ? tok : 0)) * a.H + h0 + (ok ? h : 0)) * RP + c * 8, ok);
    }
  }
  if (t_lo < t_hi) load_tile(t_lo, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");

  const int wm = warp % MT, wn = warp / MT;
  const int r_lo = wm * 16 + g, r_hi = r_lo + 8;     // this thread's rows in S
  // visible keys of the two rows: (first, last]; rows without a query see none
  int lim_lo[2], lim_hi[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = i ? r_hi : r_lo;
    const int tok = r / p.hb, h = r - tok * p.hb;
    const bool ok = tok < toks && h < heads;
    lim_hi[i] = ok ? pos0 + tok : -1;
    lim_lo[i] = a.window > 0 ? pos0 + tok - a.window + 1 : 0;
  }
  const float sc = a.scale * 1.4426950408889634f;
  float m2[2] = {-INFINITY, -INFINITY}, l2[2] = {0.f, 0.f};
  float o[MT][NT][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int c = 0; c < 4; ++c) o[i][j][c] = 0.f;

  // fragment addresses: the row of every fragment load is congruent to lane & 7 modulo 8, so the swizzled chunk depends on
  // the position inside a 128-byte group only and everything else is an immediate offset
  const uint32_t q_base = smem_u32(qs) + (wm * 16 + (lane & 15)) * ROWB;
  const int n_row = wn * (NS * 8) + (lane & 7) + (NS > 1 ? (lane >> 4) << 3 : 0);
  const uint32_t v_row = ((lane & 7) + ((lane >> 3) & 1) * 8) * ROWB;
  uint32_t q_at[4], c_at[4], v_at[NT > 1 ? NT / 2 : 1];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    q_at[i] = q_base + (((i * 2 + (lane >> 4)) ^ (lane & 7)) << 4);
    c_at[i] = n_row * ROWB + (((i * 2 + ((lane >> 3) & 1)) ^ (lane & 7)) << 4);
  }
#pragma unroll
  for (int j = 0; j < (NT > 1 ? NT / 2 : 1); ++j)
    v_at[j] = v_row + (((warp * NT + 2 * j + (NT > 1 ? lane >> 4 : 0)) ^ (lane & 7)) << 4);
  auto p_chunk = [](int r, int chunk) { return r * PB + ((chunk ^ (PB == 128 ? r & 7 : (r >> 1) & 3)) << 4); };
  uint32_t p_at[kKeyTile / 16];
#pragma unroll
  for (int ks = 0; ks < kKeyTile / 16; ++ks) p_at[ks] = smem_u32(ps) + p_chunk(lane & 15, ks * 2 + (lane >> 4));
  for (int t = t_lo; t < t_hi; ++t) {
    const int b = (t - t_lo) & 1;
    if (t + 1 < t_hi) load_tile(t + 1, b ^ 1);       // its buffer was released by the barrier that ended the last turn
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    const uint32_t c_base = smem_u32(cs + b * kKeyTile * ROWB);
    // ---- S = Q C^T
    float sfr[NS][4], sodd[NS][4];                   // even and odd k-steps: two accumulation chains per tile
#pragma unroll
    for (int j = 0; j < NS; ++j)
#pragma unroll
      for (int c = 0; c < 4; ++c) sfr[j][c] = sodd[j][c] = 0.f;
#pragma unroll
    for (int kk = 0; kk < RP / 16; ++kk) {
      uint32_t qa[4];
      ldsm4(qa, q_at[kk & 3] + (kk >> 2) * 128);
#pragma unroll
      for (int j = 0; j < NS; j += 2) {
        uint32_t cb[4];
        const uint32_t addr = c_base + c_at[kk & 3] + (kk >> 2) * 128 + j * 8 * ROWB;
        if constexpr (NS == 1) {
          ldsm2(cb, addr);
          mma_bf16(kk & 1 ? sodd[j] : sfr[j], qa, cb[0], cb[1]);
        } else {
          ldsm4(cb, addr);
          mma_bf16(kk & 1 ? sodd[j] : sfr[j], qa, cb[0], cb[1]);
          mma_bf16(kk & 1 ? sodd[j + 1] : sfr[j + 1], qa, cb[2], cb[3]);
        }
      }
    }
#pragma unroll
    for (int j = 0; j < NS; ++j)
#pragma unroll
      for (int c = 0; c < 4; ++c) sfr[j][c] += sodd[j][c];
    const int key0 = kmin + t * kKeyTile + wn * (NS * 8) + 2 * t4;
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int j = 0; j < NS; ++j)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int key = key0 + j * 8 + (c & 1), i = c >> 1;
        sfr[j][c] = (key >= lim_lo[i] && key <= lim_hi[i]) ? sfr[j][c] * sc : -INFINITY;
        mx[i] = fmaxf(mx[i], sfr[j][c]);
      }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
    }
    if (t4 == 0) {
      pmax[wn * MR + r_lo] = mx[0];
      pmax[wn * MR + r_hi] = mx[1];
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int r = i ? r_hi : r_lo;
      float mn = m2[i];
#pragma unroll
      for (int w = 0; w < WN; ++w) mn = fmaxf(mn, pmax[w * MR + r]);
      const float use = mn == -INFINITY ? 0.f : mn;
      const float al = exp2f(m2[i] - use);           // 0 on the first visible tile
      m2[i] = mn;
      if (wn == 0 && t4 == 0) alpha[r] = al;
      float sum = 0.f;
#pragma unroll
      for (int j = 0; j < NS; ++j) {
        const float e0 = exp2f(sfr[j][2 * i] - use), e1 = exp2f(sfr[j][2 * i + 1] - use);
        sum += e0 + e1;
        const int chunk = wn * NS + j;               // 8 keys per 16-byte chunk
        *reinterpret_cast<uint32_t*>(ps + p_chunk(r, chunk) + t4 * 4) = pack_bf16x2(e0, e1);
      }
      l2[i] = l2[i] * al + sum;
    }
    __syncthreads();
    // ---- O = alpha O + P C
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const float a0 = alpha[i * 16 + g], a1 = alpha[i * 16 + g + 8];
#pragma unroll
      for (int j = 0; j < NT; ++j) { o[i][j][0] *= a0; o[i][j][1] *= a0; o[i][j][2] *= a1; o[i][j][3] *= a1; }
    }
#pragma unroll
    for (int ks = 0; ks < kKeyTile / 16; ++ks) {
      uint32_t pa[MT][4];
#pragma unroll
      for (int i = 0; i < MT; ++i) ldsm4(pa[i], p_at[ks] + i * 16 * PB);
#pragma unroll
      for (int j = 0; j < NT; j += 2) {
        uint32_t vb[4];
        const uint32_t addr = c_base + v_at[j / 2] + ks * 16 * ROWB;
        if constexpr (NT == 1) ldsm2_t(vb, addr);
        else ldsm4_t(vb, addr);
#pragma unroll
        for (int i = 0; i < MT; ++i) {
          mma_bf16(o[i][j], pa[i], vb[0], vb[1]);
          if constexpr (NT > 1) mma_bf16(o[i][j + 1], pa[i], vb[2], vb[3]);
        }
      }
    }
    __syncthreads();                                 // tile buffer, P and the statistics are free again
  }
  asm volatile("cp.async.wait_all;" ::: "memory");
  // ---- row sums over the lanes and key warps of a row
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    l2[i] += __shfl_xor_sync(0xffffffffu, l2[i], 1);
    l2[i] += __shfl_xor_sync(0xffffffffu, l2[i], 2);
    const int r = i ? r_hi : r_lo;
    if (t4 == 0) {
      lsum[wn * MR + r] = l2[i];
      if (wn == 0) mrow[r] = m2[i];
    }
  }
  __syncthreads();
  auto row_total = [&](int r) {
    float l = 0.f;
#pragma unroll
    for (int w = 0; w < WN; ++w) l += lsum[w * MR + r];
    return l;
  };
  const int col0 = warp * (NT * 8) + 2 * t4;
  if (p.splits == 1) {
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int r = i * 16 + g + 8 * hf;
        const int tok = r / p.hb, h = r - tok * p.hb;
        if (tok >= toks || h >= heads) continue;
        const float f = a.gate_at(row0 + tok, h0 + h) / row_total(r);
        __nv_bfloat16* dst = a.out + ((row0 + tok) * a.H + h0 + h) * RV + col0;
#pragma unroll
        for (int j = 0; j < NT; ++j)
          *reinterpret_cast<uint32_t*>(dst + j * 8) = pack_bf16x2(o[i][j][2 * hf] * f, o[i][j][2 * hf + 1] * f);
      }
    return;
  }
  const size_t unit = static_cast<size_t>(blockIdx.x) * gridDim.y + blockIdx.y;
  float* base = p.partial + unit * p.splits * MR * (RV + 2);
  float* mine = base + static_cast<size_t>(blockIdx.z) * MR * (RV + 2);
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int r = i * 16 + g + 8 * hf;
#pragma unroll
      for (int j = 0; j < NT; ++j)
        *reinterpret_cast<float2*>(mine + static_cast<size_t>(r) * (RV + 2) + col0 + j * 8) =
            make_float2(o[i][j][2 * hf], o[i][j][2 * hf + 1]);
    }
  if (tid < MR) {
    mine[static_cast<size_t>(tid) * (RV + 2) + RV] = mrow[tid];
    mine[static_cast<size_t>(tid) * (RV + 2) + RV + 1] = row_total(tid);
  }
}

// Merge of the key splits: a warp per row, eight rows per block.
template <int NV>
__global__ void __launch_bounds__(256)
latent_merge_kernel(const LatentMma p, int mr) {
  constexpr int RV = NV * 64;
  pdl_wait();
  pdl_launch_dependents();
  const LatentAttn<__nv_bfloat16>& a = p.a;
  int s, off;
  if (!find_tile(a.sg, p.qb, blockIdx.x, s, off)) return;
  const int lane = threadIdx.x & 31, r = blockIdx.z * 8 + (threadIdx.x >> 5);
  const int h0 = blockIdx.y * p.hb;
  const int tok = r / p.hb, h = r - tok * p.hb;
  if (tok >= min(p.qb, a.sg.count[s] - off) || h >= min(p.hb, a.H - h0)) return;
  const size_t unit = static_cast<size_t>(blockIdx.x) * gridDim.y + blockIdx.y;
  const float* row = p.partial + unit * p.splits * mr * (RV + 2) + static_cast<size_t>(r) * (RV + 2);
  const size_t step = static_cast<size_t>(mr) * (RV + 2);
  float mx = -INFINITY;
  for (int z = 0; z < p.splits; ++z) mx = fmaxf(mx, row[z * step + RV]);
  float l = 0.f;
  float2 acc[NV];
#pragma unroll
  for (int c = 0; c < NV; ++c) acc[c] = make_float2(0.f, 0.f);
#pragma unroll 4
  for (int z = 0; z < p.splits; ++z) {
    const float mz = row[z * step + RV];
    const float f = mz == -INFINITY ? 0.f : exp2f(mz - mx);
    l += f * row[z * step + RV + 1];
#pragma unroll
    for (int c = 0; c < NV; ++c) {
      const float2 v = *reinterpret_cast<const float2*>(row + z * step + c * 64 + lane * 2);
      acc[c].x = fmaf(f, v.x, acc[c].x);
      acc[c].y = fmaf(f, v.y, acc[c].y);
    }
  }
  const size_t t = static_cast<size_t>(a.sg.row0[s]) + off + tok;
  const float f = a.gate_at(t, h0 + h) / l;
  __nv_bfloat16* dst = a.out + (t * a.H + h0 + h) * RV;
#pragma unroll
  for (int c = 0; c < NV; ++c)
    *reinterpret_cast<uint32_t*>(dst + c * 64 + lane * 2) = pack_bf16x2(acc[c].x * f, acc[c].y * f);
}

template <int MR, int NCH, int NV>
static int mma_go(const LatentMma& p, dim3 grid, cudaStream_t st) {
  constexpr int ROWB = NCH * 128, WN = 128 / MR;
  const size_t smem = static_cast<size_t>(MR) * ROWB + 2 * key_tile<MR>() * ROWB + MR * key_tile<MR>() * 2 + sizeof(float) * MR * (2 + 2 * WN);
  auto kernel = latent_attn_mma_kernel<MR, NCH, NV>;
  static bool configured[64] = {};     // per device
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -18;
  if (!configured[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
    configured[dev] = true;
  }
  const cudaError_t rc = launch(kernel, grid, dim3(256), smem, st, p);
  if (rc != cudaSuccess || p.splits == 1) return static_cast<int>(rc);
  return static_cast<int>(launch(latent_merge_kernel<NV>, dim3(grid.x, grid.y, MR / 8), dim3(256), 0, st, p, MR));
}
template <int MR>
static int mma_nch(const LatentMma& p, dim3 grid, cudaStream_t st) {
  switch (p.a.Rp) {
    case 64: return mma_go<MR, 1, 1>(p, grid, st);
    case 128: return mma_go<MR, 2, 2>(p, grid, st);
    case 192: return mma_go<MR, 3, 2>(p, grid, st);
    case 256: return mma_go<MR, 4, 4>(p, grid, st);
    case 320: return mma_go<MR, 5, 4>(p, grid, st);
    case 512: return mma_go<MR, 8, 8>(p, grid, st);
    case 576: return mma_go<MR, 9, 8>(p, grid, st);
  }
  return -14;
}

// Heads and tokens of a block: as many (token, head) rows as fit, 32 rows when a step has one token per segment.
static void mma_shape(int H, bool decode, int& mr, int& hb, int& qb) {
  mr = decode && H <= 32 ? 32 : 64;
  hb = H < mr ? H : mr;
  qb = decode ? 1 : mr / hb;
}

}  // namespace cb

extern "C" {

struct CbLatentAttn {
  const void* q;
  void* out;
  const void* cache;
  const void* gate; int ldg;
  const void* page_table;
  int max_pages, H, Rp, Rv, window;
  float scale;
  int tokens, f32;
  int decode;                 // every segment has at most one row
  int splits;                 // key splits of the tensor-core form (1 = none)
  void* partial;              // fp32 scratch of cb_latent_attn_partial_floats elements (splits > 1)
};

// Whether the tensor-core form has these columns of a cached row and of the output.
int cb_latent_attn_mma(int Rp, int Rv) {
  switch (Rp) {
    case 64: case 128: case 256: case 512: return Rv == Rp;
    case 192: case 320: case 576: return Rv == Rp - 64;
  }
  return 0;
}

// Scratch of a split launch; `units` receives the blocks of one split.
long long cb_latent_attn_partial_floats(int tokens, int segs, int H, int Rv, int decode, int splits, int* units) {
  int mr, hb, qb;
  cb::mma_shape(H, decode != 0, mr, hb, qb);
  const int n = cb::max_tiles(tokens, segs, qb) * ((H + hb - 1) / hb);
  if (units) *units = n;
  return splits > 1 ? static_cast<long long>(n) * splits * mr * (Rv + 2) : 0;
}

}  // extern "C"

namespace cb {
template <typename T>
static int latent_attn_typed(const CbLatentAttn* a, const CbSegments* seg, cudaStream_t st) {
  LatentAttn<T> p;
  p.q = static_cast<const T*>(a->q);
  p.out = static_cast<T*>(a->out);
  p.cache = static_cast<const T*>(a->cache);
  p.gate = static_cast<const T*>(a->gate); p.ldg = a->ldg;
  p.page_table = static_cast<const int*>(a->page_table);
  p.max_pages = a->max_pages; p.H = a->H; p.Rp = a->Rp; p.Rv = a->Rv; p.window = a->window; p.scale = a->scale;
  p.sg = make_segments(seg, a->tokens);
  const dim3 grid(a->tokens, (a->H + 3) / 4);
  if (a->Rp <= 64) return static_cast<int>(launch(latent_attn_kernel<T, 2>, grid, dim3(128), 0, st, p));
  if (a->Rp <= 128) return static_cast<int>(launch(latent_attn_kernel<T, 4>, grid, dim3(128), 0, st, p));
  if (a->Rp <= 256) return static_cast<int>(launch(latent_attn_kernel<T, 8>, grid, dim3(128), 0, st, p));
  if (a->Rp <= 512) return static_cast<int>(launch(latent_attn_kernel<T, 16>, grid, dim3(128), 0, st, p));
  return static_cast<int>(launch(latent_attn_kernel<T, 32>, grid, dim3(128), 0, st, p));
}
}  // namespace cb

extern "C" {

struct CbLatentPrep {
  const void* proj; int ldp, q_off, q_rank, c_off, R;
  const void* qw;
  const void* cw;
  void* cq; int ldq;
  void* cache; int Rp;
  const void* slots;
  int qr_off, r_off, col, pairs;
  const void* freq;
  float mult;
  const void* positions;
  void* ql; int H;
  int tokens;
  float eps;
  int f32;
};

int cb_latent_prepare(const CbLatentPrep* a, void* stream) {
  using namespace cb;
  if (!a || a->tokens <= 0) return 0;
  if (a->q_rank < 0 || a->R <= 0 || a->R > a->Rp || a->q_rank > a->ldq || (a->q_rank && !a->cq)) return -10;
  if (a->pairs < 0 || a->pairs > kMaxRotPairs || (a->pairs && (a->col < a->R || a->col + 2 * a->pairs > a->Rp || !a->freq || !a->positions || !a->ql)))
    return -11;
  if (a->pairs && ((a->ldp | a->qr_off | a->r_off | a->col | a->Rp) & 1)) return -12;
  auto go = [&](auto kernel, auto p) {
    using T = std::remove_pointer_t<decltype(p.cache)>;
    p.proj = static_cast<const T*>(a->proj); p.ldp = a->ldp;
    p.q_off = a->q_off; p.q_rank = a->q_rank; p.c_off = a->c_off; p.R = a->R;
    p.qw = static_cast<const float*>(a->qw); p.cw = static_cast<const float*>(a->cw);
    p.cq = static_cast<T*>(a->cq); p.ldq = a->ldq;
    p.cache = static_cast<T*>(a->cache); p.Rp = a->Rp;
    p.slots = static_cast<const int*>(a->slots);
    p.qr_off = a->qr_off; p.r_off = a->r_off; p.col = a->col; p.pairs = a->pairs;
    p.freq = static_cast<const float*>(a->freq); p.mult = a->mult;
    p.positions = static_cast<const int*>(a->positions);
    p.ql = static_cast<T*>(a->ql); p.H = a->pairs ? a->H : 0;
    p.eps = a->eps;
    // few tokens: more blocks share a token's queries
    const int ny = a->tokens >= 512 ? 1 : min(4, 1 + p.H * p.pairs / 512);
    return static_cast<int>(launch(kernel, dim3(a->tokens, ny), dim3(128), 0, static_cast<cudaStream_t>(stream), p));
  };
  return a->f32 ? go(latent_prepare_kernel<float>, LatentPrep<float>{}) : go(latent_prepare_kernel<__nv_bfloat16>, LatentPrep<__nv_bfloat16>{});
}

int cb_latent_attn(const CbLatentAttn* a, const CbSegments* seg, void* stream) {
  if (!a || !seg || seg->num <= 0 || a->tokens <= 0) return 0;
  if (a->H <= 0 || a->Rp <= 0 || a->Rp > 1024 || a->Rv <= 0 || a->Rv > a->Rp || (a->H + 3) / 4 > 65535) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (!a->f32 && cb_latent_attn_mma(a->Rp, a->Rv)) {
    using namespace cb;
    if (a->splits > 1 && (!a->partial || a->splits > 65535)) return -12;
    LatentMma p;
    p.a.q = static_cast<const __nv_bfloat16*>(a->q);
    p.a.out = static_cast<__nv_bfloat16*>(a->out);
    p.a.cache = static_cast<const __nv_bfloat16*>(a->cache);
    p.a.gate = static_cast<const __nv_bfloat16*>(a->gate); p.a.ldg = a->ldg;
    p.a.page_table = static_cast<const int*>(a->page_table);
    p.a.max_pages = a->max_pages; p.a.H = a->H; p.a.Rp = a->Rp; p.a.Rv = a->Rv; p.a.window = a->window; p.a.scale = a->scale;
    p.a.sg = make_segments(seg, a->tokens);
    int mr;
    mma_shape(a->H, a->decode != 0, mr, p.hb, p.qb);
    p.splits = a->splits > 1 ? a->splits : 1;
    p.partial = static_cast<float*>(a->partial);
    const dim3 grid(max_tiles(a->tokens, seg->num, p.qb), (a->H + p.hb - 1) / p.hb, p.splits);
    return mr == 32 ? mma_nch<32>(p, grid, st) : mma_nch<64>(p, grid, st);
  }
  return a->f32 ? cb::latent_attn_typed<float>(a, seg, st) : cb::latent_attn_typed<__nv_bfloat16>(a, seg, st);
}

}  // extern "C"
