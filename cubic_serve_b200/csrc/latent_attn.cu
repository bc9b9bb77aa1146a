// Latent attention without positions over a paged cache of latents, with a sliding window and a gate per head.
//
// A token's cache row is its latent c (R channels, one row for all heads).  A head's key is W_uk c and its value W_uv c,
// so its scores are (W_uk^T q) . c: the runner multiplies the queries by W_uk^T once (a block-diagonal product), the
// attention below runs on latents for all heads at once, and W_uv is applied to its output.
//
//   latent_prepare_kernel   RMS norms of the query latent and of the cache latent; the latter is written to its page
//   latent_attn_kernel      a warp per (token, head), fp32 arithmetic on rows of either activation type
//
// The cache is [pages][16][Rp] with Rp = R rounded up to 64 and zero columns behind R.
#include "segments.cuh"
#include "launch.cuh"

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
};

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
  p.sg = make_segments(seg);
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
  return a->f32 ? cb::latent_attn_typed<float>(a, seg, st) : cb::latent_attn_typed<__nv_bfloat16>(a, seg, st);
}

}  // extern "C"
