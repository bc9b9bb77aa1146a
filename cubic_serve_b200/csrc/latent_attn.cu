// Latent attention without positions over a paged cache of latents, with a sliding window and a gate per head.
//
// A token's cache row is its latent c (R channels, one row for all heads).  A head's key is W_uk c and its value W_uv c,
// so its scores are (W_uk^T q) . c: the runner multiplies the queries by W_uk^T once (a block-diagonal product), the
// attention below runs on latents for all heads at once, and W_uv is applied to its output.
//
//   latent_prepare_kernel   RMS norms of the query latent and of the cache latent; the latter is written to its page
//   latent_attn_mma_kernel, latent_merge_kernel  bf16 rows on the tensor cores: 32 or 64 (token, head) rows share every latent they read
//   latent_attn_kernel      a warp per (token, head), fp32 arithmetic on rows of either type (32-bit models; wide latents)
//
// The cache is [pages][16][Rp] with Rp >= R (64, 128, 256, 512 or 1024) and zero columns behind R.
#include "segments.cuh"
#include "launch.cuh"
#include "mma.cuh"

namespace cb {

static constexpr int kLatentPage = 16;

template <typename T>
__global__ void __launch_bounds__(128)
latent_prepare_kernel(const T* __restrict__ proj, int ldp, int q_off, int q_rank, int c_off, int R, const float* __restrict__ qw,
                      const float* __restrict__ cw, T* __restrict__ cq, int ldq, T* __restrict__ cache, int Rp,
                      const int* __restrict__ slots, float eps) {
  __shared__ float red[2][4];
  pdl_wait();
  pdl_launch_dependents();
  const size_t t = blockIdx.x;
  const T* qr = proj + t * ldp + q_off;
  const T* cr = proj + t * ldp + c_off;
  float sq = 0.f, sc = 0.f;
  for (int c = threadIdx.x; c < q_rank; c += 128) { const float v = to_f(qr[c]); sq = fmaf(v, v, sq); }
  for (int c = threadIdx.x; c < R; c += 128) { const float v = to_f(cr[c]); sc = fmaf(v, v, sc); }
  sq = warp_sum(sq);
  sc = warp_sum(sc);
  if ((threadIdx.x & 31) == 0) { red[0][threadIdx.x >> 5] = sq; red[1][threadIdx.x >> 5] = sc; }
  __syncthreads();
  sq = red[0][0] + red[0][1] + red[0][2] + red[0][3];
  sc = red[1][0] + red[1][1] + red[1][2] + red[1][3];
  const float iq = 1.f / sqrtf(sq / static_cast<float>(q_rank) + eps);
  for (int c = threadIdx.x; c < q_rank; c += 128) cq[t * ldq + c] = from_f<T>(to_f(qr[c]) * iq * qw[c]);
  const int slot = slots[t];
  if (slot < 0) return;                                  // padding row
  const float ic = 1.f / sqrtf(sc / static_cast<float>(R) + eps);
  T* dst = cache + static_cast<size_t>(slot) * Rp;
  for (int c = threadIdx.x; c < R; c += 128) dst[c] = from_f<T>(to_f(cr[c]) * ic * cw[c]);
}

template <typename T>
struct LatentAttn {
  const T* q;             // [T, H, Rp] queries in latent space
  T* out;                 // [T, H, Rp]
  const T* cache;         // [pages, 16, Rp]
  const T* gate; int ldg; // [T, H] gate logits: the output is multiplied by their sigmoid
  const int* page_table;  // [slots, max_pages]
  int max_pages;
  int H, Rp, window;      // window <= 0: every earlier token
  float scale;
  Segments sg;
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
  const float g = 1.f / (1.f + expf(-to_f(p.gate[row * p.ldg + h]))) / l;
  T* orow = p.out + (row * p.H + h) * p.Rp;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int c = lane + 32 * i;
    if (c < p.Rp) orow[c] = from_f<T>(acc[i] * g);
  }
}

// ------------------------------------------------------------------ tensor-core form
// MR query rows per block: consecutive tokens of one segment x the heads of a head group, row = token * hb + head.  Key
// tiles of KT latents arrive by cp.async in two buffers (16-byte chunks XOR-swizzled by the row, so that ldmatrix reads
// both orientations without bank conflicts): the same tile is the key operand of S = Q C^T and the value operand of
// O += P C.  Eight warps: for S they form MR / 16 x 128 / MR (rows x keys); for O every warp owns Rp / 8 latent columns
// of all rows, so a value fragment is read once per block.  Scores, softmax weights and sums are fp32; the weights are
// rounded to bf16 as the operand of the second product.  With splits > 1 the key tiles are dealt to grid.z blocks and
// latent_merge_kernel adds their partial results in split order.  The 32-row form (decode) takes key tiles of 32, so that
// two blocks share an SM and one's loads overlap the other's products.

struct LatentMma {
  LatentAttn<__nv_bfloat16> a;
  int hb, qb;             // heads of a block, tokens of a block (hb * qb <= MR)
  int splits;
  float* partial;         // [tile][head group][split][MR][Rp + 2]
};

template <int MR> constexpr int key_tile() { return MR == 32 ? 32 : 64; }

template <int MR, int NCH>
__global__ void __launch_bounds__(256, MR == 32 ? 2 : 1)
latent_attn_mma_kernel(const LatentMma p) {
  constexpr int RP = NCH * 64, ROWB = RP * 2;        // bytes of a latent row
  constexpr int kKeyTile = key_tile<MR>();
  constexpr int MT = MR / 16, WN = 8 / MT;           // S: MT x WN warps
  constexpr int NS = kKeyTile / WN / 8;              // n8 key tiles of a warp in S
  constexpr int NT = NCH;                            // n8 column tiles of a warp in O
  extern __shared__ __align__(128) uint8_t lsm[];
  uint8_t* qs = lsm;                                 // [MR][ROWB]
  uint8_t* cs = qs + MR * ROWB;                      // [2][64][ROWB]
  uint8_t* ps = cs + 2 * kKeyTile * ROWB;            // [MR][128]
  float* alpha = reinterpret_cast<float*>(ps + MR * 128);   // [MR]
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
  const uint32_t p_at0 = smem_u32(ps) + (lane & 15) * 128;
  uint32_t p_at[kKeyTile / 16];
#pragma unroll
  for (int ks = 0; ks < kKeyTile / 16; ++ks) p_at[ks] = p_at0 + (((ks * 2 + (lane >> 4)) ^ (lane & 7)) << 4);
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
        *reinterpret_cast<uint32_t*>(ps + r * 128 + ((chunk ^ (r & 7)) << 4) + t4 * 4) = pack_bf16x2(e0, e1);
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
      for (int i = 0; i < MT; ++i) ldsm4(pa[i], p_at[ks] + i * 16 * 128);
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
  auto gate_at = [&](int tok, int h) {
    return 1.f / (1.f + expf(-__bfloat162float(a.gate[(row0 + tok) * a.ldg + h0 + h])));
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
        const float f = gate_at(tok, h) / row_total(r);
        __nv_bfloat16* dst = a.out + ((row0 + tok) * a.H + h0 + h) * RP + col0;
#pragma unroll
        for (int j = 0; j < NT; ++j)
          *reinterpret_cast<uint32_t*>(dst + j * 8) = pack_bf16x2(o[i][j][2 * hf] * f, o[i][j][2 * hf + 1] * f);
      }
    return;
  }
  const size_t unit = static_cast<size_t>(blockIdx.x) * gridDim.y + blockIdx.y;
  float* base = p.partial + unit * p.splits * MR * (RP + 2);
  float* mine = base + static_cast<size_t>(blockIdx.z) * MR * (RP + 2);
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int r = i * 16 + g + 8 * hf;
#pragma unroll
      for (int j = 0; j < NT; ++j)
        *reinterpret_cast<float2*>(mine + static_cast<size_t>(r) * (RP + 2) + col0 + j * 8) =
            make_float2(o[i][j][2 * hf], o[i][j][2 * hf + 1]);
    }
  if (tid < MR) {
    mine[static_cast<size_t>(tid) * (RP + 2) + RP] = mrow[tid];
    mine[static_cast<size_t>(tid) * (RP + 2) + RP + 1] = row_total(tid);
  }
}

// Merge of the key splits: a warp per row, eight rows per block.
template <int NCH>
__global__ void __launch_bounds__(256)
latent_merge_kernel(const LatentMma p, int mr) {
  constexpr int RP = NCH * 64;
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
  const float* row = p.partial + unit * p.splits * mr * (RP + 2) + static_cast<size_t>(r) * (RP + 2);
  const size_t step = static_cast<size_t>(mr) * (RP + 2);
  float mx = -INFINITY;
  for (int z = 0; z < p.splits; ++z) mx = fmaxf(mx, row[z * step + RP]);
  float l = 0.f;
  float2 acc[NCH];
#pragma unroll
  for (int c = 0; c < NCH; ++c) acc[c] = make_float2(0.f, 0.f);
#pragma unroll 4
  for (int z = 0; z < p.splits; ++z) {
    const float mz = row[z * step + RP];
    const float f = mz == -INFINITY ? 0.f : exp2f(mz - mx);
    l += f * row[z * step + RP + 1];
#pragma unroll
    for (int c = 0; c < NCH; ++c) {
      const float2 v = *reinterpret_cast<const float2*>(row + z * step + c * 64 + lane * 2);
      acc[c].x = fmaf(f, v.x, acc[c].x);
      acc[c].y = fmaf(f, v.y, acc[c].y);
    }
  }
  const size_t t = static_cast<size_t>(a.sg.row0[s]) + off + tok;
  const float f = 1.f / (1.f + expf(-__bfloat162float(a.gate[t * a.ldg + h0 + h]))) / l;
  __nv_bfloat16* dst = a.out + (t * a.H + h0 + h) * RP;
#pragma unroll
  for (int c = 0; c < NCH; ++c)
    *reinterpret_cast<uint32_t*>(dst + c * 64 + lane * 2) = pack_bf16x2(acc[c].x * f, acc[c].y * f);
}

template <int MR, int NCH>
static int mma_go(const LatentMma& p, dim3 grid, cudaStream_t st) {
  constexpr int ROWB = NCH * 128, WN = 128 / MR;
  const size_t smem = static_cast<size_t>(MR) * ROWB + 2 * key_tile<MR>() * ROWB + MR * 128 + sizeof(float) * MR * (2 + 2 * WN);
  auto kernel = latent_attn_mma_kernel<MR, NCH>;
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
  return static_cast<int>(launch(latent_merge_kernel<NCH>, dim3(grid.x, grid.y, MR / 8), dim3(256), 0, st, p, MR));
}
template <int MR>
static int mma_nch(const LatentMma& p, dim3 grid, cudaStream_t st) {
  switch (p.a.Rp) {
    case 64: return mma_go<MR, 1>(p, grid, st);
    case 128: return mma_go<MR, 2>(p, grid, st);
    case 256: return mma_go<MR, 4>(p, grid, st);
    case 512: return mma_go<MR, 8>(p, grid, st);
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
  int max_pages, H, Rp, window;
  float scale;
  int tokens, f32;
  int decode;                 // every segment has at most one row
  int splits;                 // key splits of the tensor-core form (1 = none)
  void* partial;              // fp32 scratch of cb_latent_attn_partial_floats elements (splits > 1)
};

// Scratch of a split launch; `units` receives the blocks of one split.
long long cb_latent_attn_partial_floats(int tokens, int segs, int H, int Rp, int decode, int splits, int* units) {
  int mr, hb, qb;
  cb::mma_shape(H, decode != 0, mr, hb, qb);
  const int n = cb::max_tiles(tokens, segs, qb) * ((H + hb - 1) / hb);
  if (units) *units = n;
  return splits > 1 ? static_cast<long long>(n) * splits * mr * (Rp + 2) : 0;
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
  p.max_pages = a->max_pages; p.H = a->H; p.Rp = a->Rp; p.window = a->window; p.scale = a->scale;
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

int cb_latent_prepare(const void* proj, int ldp, int q_off, int q_rank, int c_off, int R, const void* qw, const void* cw,
                      void* cq, int ldq, void* cache, int Rp, const void* slots, int tokens, float eps, int f32, void* stream) {
  using namespace cb;
  if (tokens <= 0) return 0;
  if (q_rank <= 0 || R <= 0 || R > Rp || q_rank > ldq) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32)
    return static_cast<int>(launch(latent_prepare_kernel<float>, dim3(tokens), dim3(128), 0, st, static_cast<const float*>(proj),
                                   ldp, q_off, q_rank, c_off, R, static_cast<const float*>(qw), static_cast<const float*>(cw),
                                   static_cast<float*>(cq), ldq, static_cast<float*>(cache), Rp, static_cast<const int*>(slots), eps));
  return static_cast<int>(launch(latent_prepare_kernel<__nv_bfloat16>, dim3(tokens), dim3(128), 0, st,
                                 static_cast<const __nv_bfloat16*>(proj), ldp, q_off, q_rank, c_off, R,
                                 static_cast<const float*>(qw), static_cast<const float*>(cw), static_cast<__nv_bfloat16*>(cq), ldq,
                                 static_cast<__nv_bfloat16*>(cache), Rp, static_cast<const int*>(slots), eps));
}

int cb_latent_attn(const CbLatentAttn* a, const CbSegments* seg, void* stream) {
  if (!a || !seg || seg->num <= 0 || a->tokens <= 0) return 0;
  if (a->H <= 0 || a->Rp <= 0 || a->Rp > 1024 || (a->H + 3) / 4 > 65535) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (!a->f32 && a->Rp <= 512) {
    using namespace cb;
    if (a->splits > 1 && (!a->partial || a->splits > 65535)) return -12;
    LatentMma p;
    p.a.q = static_cast<const __nv_bfloat16*>(a->q);
    p.a.out = static_cast<__nv_bfloat16*>(a->out);
    p.a.cache = static_cast<const __nv_bfloat16*>(a->cache);
    p.a.gate = static_cast<const __nv_bfloat16*>(a->gate); p.a.ldg = a->ldg;
    p.a.page_table = static_cast<const int*>(a->page_table);
    p.a.max_pages = a->max_pages; p.a.H = a->H; p.a.Rp = a->Rp; p.a.window = a->window; p.a.scale = a->scale;
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
