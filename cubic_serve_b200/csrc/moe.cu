// Mixture-of-experts routing: stable top-k, per-expert counts, permutation, gather, weighted combine.
//
// Counterparts in the reference: ops/cuda/moe/fused.py (_stable_topk_logits :44,
// _sort_and_normalize_topk :71, _count/_prefix/_scatter_local_routes :159-222,
// _route_combine :444).  Semantics kept: top-k over router logits with the
// lowest expert id winning ties, softmax over the SELECTED logits only
// (= softmax over all experts renormalised to the top-k), routes of one expert
// contiguous for the grouped GEMM (wq_gemm.cu, grouped mode), combine in fixed
// route order per token so the result does not depend on the permutation.
//
// Expert parallelism: `expert_lo / expert_count` select the experts THIS rank
// owns; routes to other experts get position -1 and contribute +0 (the
// reference's replicated-token EP, runtime/README.md:140-160 there), so the same
// kernels serve EP = 1 and the EP shards whose partial outputs are then reduced
// like any row-parallel partial sum.
#include "ptx.cuh"
#include "launch.cuh"

namespace cb {

static constexpr int kMaxTopK = 8;

// One warp per token: E <= 256 experts, lane l holds experts l, l+32, ...
__global__ void __launch_bounds__(128)
moe_route_kernel(const __nv_bfloat16* __restrict__ logits, int ld, int T, int E, int k, int normalize,
                 int expert_lo, int expert_count, int* __restrict__ topk_ids, float* __restrict__ topk_w,
                 int* __restrict__ counts) {
  const int t = blockIdx.x * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (t >= T) return;
  float v[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int e = lane + 32 * j;
    v[j] = e < E ? __bfloat162float(logits[static_cast<size_t>(t) * ld + e]) : -INFINITY;
    if (!(v[j] == v[j])) v[j] = -INFINITY;
  }
  float sel_v[kMaxTopK];
  int sel_e[kMaxTopK];
  for (int r = 0; r < k; ++r) {
    float bv = -INFINITY;
    int be = 0x7fffffff;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int e = lane + 32 * j;
      if (v[j] > bv || (v[j] == bv && e < be)) { bv = v[j]; be = e; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      if (ov > bv || (ov == bv && oe < be)) { bv = ov; be = oe; }
    }
    sel_v[r] = bv;
    sel_e[r] = be;
    if ((be & 31) == lane) v[be >> 5] = -INFINITY;   // remove the winner
  }
  if (lane == 0) {
    float w[kMaxTopK], sum = 0.f;
    for (int r = 0; r < k; ++r) { w[r] = __expf(sel_v[r] - sel_v[0]); sum += w[r]; }
    // normalize = 1: softmax over the selected logits.  normalize = 0: softmax over ALL experts, not
    // renormalised: needs the full denominator
    float denom = sum;
    if (!normalize) {
      denom = 0.f;
      for (int e = 0; e < E; ++e) denom += __expf(__bfloat162float(logits[static_cast<size_t>(t) * ld + e]) - sel_v[0]);
    }
    for (int r = 0; r < k; ++r) {
      topk_ids[t * k + r] = sel_e[r];
      topk_w[t * k + r] = w[r] / denom;
      const int local = sel_e[r] - expert_lo;
      if (local >= 0 && local < expert_count) atomicAdd(&counts[local], 1);
    }
  }
}

// Single CTA: exclusive scan of the counts -> offsets (cursors start there), and the work list of the grouped
// GEMM: one item per (expert, block of `mb` rows) = {expert, first row, rows}; at most ceil(routes / mb) + E items.
__global__ void __launch_bounds__(256)
moe_scan_kernel(const int* __restrict__ counts, int* __restrict__ offsets, int* __restrict__ cursors, int E, int mb,
                int* __restrict__ total, int* __restrict__ tiles /* [0] = count, then {expert,row0,rows} triples */) {
  __shared__ int sm[256];
  __shared__ int st[256];
  const int e = threadIdx.x;
  const int cnt = e < E ? counts[e] : 0;
  const int nt = (cnt + mb - 1) / mb;
  sm[e] = cnt;
  st[e] = nt;
  __syncthreads();
  for (int o = 1; o < 256; o <<= 1) {
    const int a = e >= o ? sm[e - o] : 0;
    const int b = e >= o ? st[e - o] : 0;
    __syncthreads();
    sm[e] += a;
    st[e] += b;
    __syncthreads();
  }
  if (e < E) {
    const int off = sm[e] - cnt;
    offsets[e] = off;
    cursors[e] = off;
    const int t0 = st[e] - nt;
    for (int i = 0; i < nt; ++i) {
      tiles[1 + 3 * (t0 + i)] = e;
      tiles[2 + 3 * (t0 + i)] = off + i * mb;
      tiles[3 + 3 * (t0 + i)] = min(mb, cnt - i * mb);
    }
  }
  if (e == 255) {
    *total = sm[255];
    tiles[0] = st[255];
  }
}

// One warp per route: claim a slot in the expert's range and copy the token's row there.
__global__ void __launch_bounds__(128)
moe_scatter_kernel(const __nv_bfloat16* __restrict__ x, const int* __restrict__ topk_ids, int T, int k, int H,
                   int expert_lo, int expert_count, int* __restrict__ cursors, int* __restrict__ route_pos,
                   __nv_bfloat16* __restrict__ xs) {
  const int route = blockIdx.x * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (route >= T * k) return;
  const int local = topk_ids[route] - expert_lo;
  int pos = -1;
  if (local >= 0 && local < expert_count) {
    if (lane == 0) pos = atomicAdd(&cursors[local], 1);
    pos = __shfl_sync(0xffffffffu, pos, 0);
    const int t = route / k;
    const uint4* src = reinterpret_cast<const uint4*>(x + static_cast<size_t>(t) * H);
    uint4* dst = reinterpret_cast<uint4*>(xs + static_cast<size_t>(pos) * H);
    for (int i = lane; i < (H >> 3); i += 32) dst[i] = src[i];
  }
  if (lane == 0) route_pos[route] = pos;
}

// out[t] (+)= sum_r w[t, r] * y[route_pos[t, r]]   (fixed r order; absent routes contribute +0)
__global__ void __launch_bounds__(256)
moe_combine_kernel(const __nv_bfloat16* __restrict__ y, const int* __restrict__ route_pos,
                   const float* __restrict__ topk_w, int k, int H, const __nv_bfloat16* residual,
                   __nv_bfloat16* __restrict__ out) {
  const int t = blockIdx.x;
  for (int v = threadIdx.x; v < (H >> 3); v += blockDim.x) {
    float acc[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j] = 0.f;
    for (int r = 0; r < k; ++r) {
      const int pos = route_pos[t * k + r];
      if (pos < 0) continue;
      const float w = topk_w[t * k + r];
      const uint4 yv = reinterpret_cast<const uint4*>(y + static_cast<size_t>(pos) * H)[v];
      const __nv_bfloat162* yp = reinterpret_cast<const __nv_bfloat162*>(&yv);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 f = __bfloat1622float2(yp[j]);
        acc[2 * j] = fmaf(w, f.x, acc[2 * j]);
        acc[2 * j + 1] = fmaf(w, f.y, acc[2 * j + 1]);
      }
    }
    if (residual) {
      const uint4 rv = reinterpret_cast<const uint4*>(residual + static_cast<size_t>(t) * H)[v];
      const __nv_bfloat162* rp = reinterpret_cast<const __nv_bfloat162*>(&rv);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 f = __bfloat1622float2(rp[j]);
        acc[2 * j] += f.x;
        acc[2 * j + 1] += f.y;
      }
    }
    uint4 ov;
    __nv_bfloat162* op = reinterpret_cast<__nv_bfloat162*>(&ov);
#pragma unroll
    for (int j = 0; j < 4; ++j) op[j] = __floats2bfloat162_rn(acc[2 * j], acc[2 * j + 1]);
    reinterpret_cast<uint4*>(out + static_cast<size_t>(t) * H)[v] = ov;
  }
}

// ------------------------------------------------------------------ scored routing (layered decoders)
// Router logits and everything up to the weights are fp32: s = softmax(z) over all `outputs` (more than `experts`: the rest return
// the token itself), the `top` largest s + correction are chosen (lowest id on ties), their weights are s over the sum of the
// chosen.  A route's rank among its expert's comes from the expert's counter.
struct ScoredRoute {
  const float* z; int ldz;    // [T, ldz]
  const float* correction;    // [outputs]
  int T, experts, outputs, top;
  int* ids;                   // [T, top] expert, -1: none (the token itself)
  int* rank;                  // [T, top] in: nothing, out: rank among the expert's routes
  float* weight;              // [T, top]
  float* self;                // [T] summed weight of the token itself
  int* counts;                // [experts], zero on entry
};

static constexpr int kMaxScoredTop = 32;

__global__ void __launch_bounds__(128)
scored_route_kernel(const ScoredRoute p) {
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (t >= p.T) return;
  float s[8], c[8], mx = -INFINITY;
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int e = lane + 32 * j;
    s[j] = e < p.outputs ? p.z[static_cast<size_t>(t) * p.ldz + e] : -INFINITY;
    if (!(s[j] == s[j])) s[j] = -INFINITY;
    mx = fmaxf(mx, s[j]);
  }
  mx = warp_max(mx);
  if (mx == -INFINITY) mx = 0.f;
  float sum = 0.f;
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    s[j] = expf(s[j] - mx);
    sum += s[j];
  }
  sum = warp_sum(sum);
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int e = lane + 32 * j;
    s[j] /= sum;
    c[j] = e < p.outputs ? s[j] + __ldg(p.correction + e) : -INFINITY;
    if (e < p.outputs && !(c[j] > -INFINITY)) c[j] = -3.0e38f;           // never chosen before a real score, always a valid id
  }
  float mine = 0.f;                                                      // lane r holds the r-th choice
  int expert = -1;
  for (int r = 0; r < p.top; ++r) {
    float bv = -INFINITY, bs = 0.f;
    int be = 0x7fffffff;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int e = lane + 32 * j;
      if (e < p.outputs && (c[j] > bv || (c[j] == bv && c[j] > -INFINITY && e < be))) { bv = c[j]; be = e; bs = s[j]; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o), os = __shfl_xor_sync(0xffffffffu, bs, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      if (ov > bv || (ov == bv && oe < be)) { bv = ov; be = oe; bs = os; }
    }
    if (lane == r) { mine = bs; expert = be; }
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (lane + 32 * j == be) c[j] = -INFINITY;
  }
  const float w = mine / (warp_sum(mine) + 1e-20f);
  const bool routed = lane < p.top && expert >= 0 && expert < p.experts;
  const float own = warp_sum(lane < p.top && !routed ? w : 0.f);
  if (lane == 0) p.self[t] = own;
  if (lane < p.top) {
    const size_t i = static_cast<size_t>(t) * p.top + lane;
    p.ids[i] = routed ? expert : -1;
    p.weight[i] = w;
    p.rank[i] = routed ? atomicAdd(p.counts + expert, 1) : -1;
  }
}

struct RouteScatter {
  const void* x; int ldx;     // [T, ldx] elements of `elem` bytes, W of them are copied
  void* xs; int ldxs;         // [routes, ldxs] rows by expert
  int T, W, elem, top, experts, mb;
  const int* ids;
  int* pos;                   // in: rank, out: place in xs (-1: none)
  int* counts;                // zero again on exit
  int* done;                  // blocks that are through, zero on entry and exit
  int* tiles;                 // work list of the grouped products: {count, then {expert, first row, rows}}
};

// Every block derives the experts' first rows from the counts; block 0 writes the work list.  A warp copies a route's row.
__global__ void __launch_bounds__(256)
route_scatter_kernel(const RouteScatter p) {
  __shared__ int rows[256], sums[2][8];
  __shared__ int last;
  pdl_wait();
  pdl_launch_dependents();
  const int e = threadIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int cnt = e < p.experts ? p.counts[e] : 0, nt = (cnt + p.mb - 1) / p.mb;
  int first = cnt, t0 = nt;                                              // sums up to here, then without this one
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int a = __shfl_up_sync(0xffffffffu, first, o), b = __shfl_up_sync(0xffffffffu, t0, o);
    if (lane >= o) { first += a; t0 += b; }
  }
  if (lane == 31) { sums[0][warp] = first; sums[1][warp] = t0; }
  __syncthreads();
  for (int w = 0; w < warp; ++w) { first += sums[0][w]; t0 += sums[1][w]; }
  first -= cnt;
  t0 -= nt;
  rows[e] = first;
  if (blockIdx.x == 0) {
    for (int i = 0; i < nt; ++i) {
      p.tiles[1 + 3 * (t0 + i)] = e;
      p.tiles[2 + 3 * (t0 + i)] = first + i * p.mb;
      p.tiles[3 + 3 * (t0 + i)] = min(p.mb, cnt - i * p.mb);
    }
    if (e == p.experts - 1) p.tiles[0] = t0 + nt;
  }
  __syncthreads();
  const size_t bytes = static_cast<size_t>(p.W) * p.elem;
  const bool vec = (bytes & 15) == 0 && ((static_cast<size_t>(p.ldx) * p.elem) & 15) == 0 && ((static_cast<size_t>(p.ldxs) * p.elem) & 15) == 0;
  for (int route = blockIdx.x * 8 + warp; route < p.T * p.top; route += 8 * gridDim.x) {
    const int ex = p.ids[route];
    if (ex < 0) continue;                                                // its place is -1 already
    const int at = rows[ex] + p.pos[route];
    const char* src = static_cast<const char*>(p.x) + static_cast<size_t>(route / p.top) * p.ldx * p.elem;
    char* dst = static_cast<char*>(p.xs) + static_cast<size_t>(at) * p.ldxs * p.elem;
    if (vec) {
      for (size_t i = lane; i < (bytes >> 4); i += 32) reinterpret_cast<uint4*>(dst)[i] = reinterpret_cast<const uint4*>(src)[i];
    } else if (p.elem == 2) {
      for (int i = lane; i < p.W; i += 32) reinterpret_cast<uint16_t*>(dst)[i] = reinterpret_cast<const uint16_t*>(src)[i];
    } else {
      for (int i = lane; i < p.W; i += 32) reinterpret_cast<uint32_t*>(dst)[i] = reinterpret_cast<const uint32_t*>(src)[i];
    }
    __syncwarp();
    if (lane == 0) p.pos[route] = at;
  }
  // the last block through leaves the counters as it found them: every block has read them by then
  __syncthreads();
  if (threadIdx.x == 0) {
    __threadfence();
    last = atomicAdd(p.done, 1) == static_cast<int>(gridDim.x) - 1;
  }
  __syncthreads();
  if (last) {
    if (e < p.experts) p.counts[e] = 0;
    if (e == 0) *p.done = 0;
  }
}

}  // namespace cb

extern "C" {

struct CbScoredMoe {
  const void* z; int ldz;
  const void* correction;
  const void* x; int ldx;
  void* xs; int ldxs;
  int T, W, elem, experts, outputs, top, mb;
  void* ids;
  void* pos;
  void* weight;
  void* self;
  void* counts;               // int [experts + 1], zero between launches
  void* tiles;                // int [1 + 3 (ceil(T top / mb) + experts)]
};

// Routing from fp32 logits and permutation of the rows to their experts (see ScoredRoute and RouteScatter).
int cb_scored_moe_route(const CbScoredMoe* a, void* stream) {
  using namespace cb;
  if (!a || a->T <= 0) return 0;
  if (a->experts < 1 || a->outputs < a->experts || a->outputs > 256 || a->top < 1 || a->top > kMaxScoredTop || a->top > a->outputs) return -10;
  if (a->W <= 0 || (a->elem != 2 && a->elem != 4) || a->ldx < a->W || a->ldxs < a->W || a->mb <= 0 || a->ldz < a->outputs) return -11;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  ScoredRoute r;
  r.z = static_cast<const float*>(a->z); r.ldz = a->ldz; r.correction = static_cast<const float*>(a->correction);
  r.T = a->T; r.experts = a->experts; r.outputs = a->outputs; r.top = a->top;
  r.ids = static_cast<int*>(a->ids); r.rank = static_cast<int*>(a->pos); r.weight = static_cast<float*>(a->weight);
  r.self = static_cast<float*>(a->self); r.counts = static_cast<int*>(a->counts);
  cudaError_t e = launch(scored_route_kernel, dim3((a->T + 3) / 4), dim3(128), 0, st, r);
  if (e != cudaSuccess) return static_cast<int>(e);
  RouteScatter s;
  s.x = a->x; s.ldx = a->ldx; s.xs = a->xs; s.ldxs = a->ldxs;
  s.T = a->T; s.W = a->W; s.elem = a->elem; s.top = a->top; s.experts = a->experts; s.mb = a->mb;
  s.ids = r.ids; s.pos = r.rank; s.counts = r.counts; s.done = r.counts + a->experts; s.tiles = static_cast<int*>(a->tiles);
  const long long routes = static_cast<long long>(a->T) * a->top;
  const int blocks = static_cast<int>(routes / 8 + 1 < 148 * 8 ? (routes + 7) / 8 : 148 * 8);
  return static_cast<int>(launch(route_scatter_kernel, dim3(blocks), dim3(256), 0, st, s));
}

// Routing + permutation in one call: zeroes the counts, selects the top-k, scans, scatters the rows.
// Buffers: topk_ids [T,k] i32, topk_w [T,k] f32, counts/offsets/cursors [expert_count] i32, total [1] i32,
// tiles [1 + 3 * (ceil(T*k / mb) + expert_count)] i32 (work list of the grouped GEMM with `mb` rows per item),
// route_pos [T,k] i32, xs [T*k, H] bf16 (rows of owned routes, expert-major).
int cb_moe_route(const void* logits, int ld, const void* x, int T, int E, int k, int H, int normalize, int expert_lo,
                 int expert_count, int mb, void* topk_ids, void* topk_w, void* counts, void* offsets, void* cursors,
                 void* total, void* tiles, void* route_pos, void* xs, void* stream) {
  using namespace cb;
  if (T <= 0) return 0;
  if (E > 256 || k > kMaxTopK || k < 1 || H % 8 != 0 || expert_count > 256) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaError_t e = cudaMemsetAsync(counts, 0, sizeof(int) * expert_count, st);
  if (e != cudaSuccess) return static_cast<int>(e);
  moe_route_kernel<<<(T + 3) / 4, 128, 0, st>>>(static_cast<const __nv_bfloat16*>(logits), ld, T, E, k, normalize,
                                                 expert_lo, expert_count, static_cast<int*>(topk_ids),
                                                 static_cast<float*>(topk_w), static_cast<int*>(counts));
  moe_scan_kernel<<<1, 256, 0, st>>>(static_cast<const int*>(counts), static_cast<int*>(offsets),
                                     static_cast<int*>(cursors), expert_count, mb, static_cast<int*>(total),
                                     static_cast<int*>(tiles));
  moe_scatter_kernel<<<(T * k + 3) / 4, 128, 0, st>>>(static_cast<const __nv_bfloat16*>(x),
                                                       static_cast<const int*>(topk_ids), T, k, H, expert_lo,
                                                       expert_count, static_cast<int*>(cursors),
                                                       static_cast<int*>(route_pos), static_cast<__nv_bfloat16*>(xs));
  return static_cast<int>(cudaGetLastError());
}

// Scan + permutation only, for callers that have already filled topk_ids ([T,k], -1 = no route) and counts
// (expert-parallel receive side: the "tokens" are the records received from the other ranks).
int cb_moe_permute(const void* x, const void* topk_ids, int T, int k, int H, int expert_lo, int expert_count, int mb,
                   const void* counts, void* offsets, void* cursors, void* total, void* tiles, void* route_pos,
                   void* xs, void* stream) {
  using namespace cb;
  if (T <= 0) return 0;
  if (k > kMaxTopK || k < 1 || H % 8 != 0 || expert_count > 256) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  moe_scan_kernel<<<1, 256, 0, st>>>(static_cast<const int*>(counts), static_cast<int*>(offsets),
                                     static_cast<int*>(cursors), expert_count, mb, static_cast<int*>(total),
                                     static_cast<int*>(tiles));
  moe_scatter_kernel<<<(T * k + 3) / 4, 128, 0, st>>>(static_cast<const __nv_bfloat16*>(x),
                                                       static_cast<const int*>(topk_ids), T, k, H, expert_lo,
                                                       expert_count, static_cast<int*>(cursors),
                                                       static_cast<int*>(route_pos), static_cast<__nv_bfloat16*>(xs));
  return static_cast<int>(cudaGetLastError());
}

int cb_moe_combine(const void* y, const void* route_pos, const void* topk_w, int T, int k, int H, const void* residual,
                   void* out, void* stream) {
  using namespace cb;
  if (T <= 0) return 0;
  if (H % 8 != 0) return -10;
  moe_combine_kernel<<<T, 256, 0, static_cast<cudaStream_t>(stream)>>>(
      static_cast<const __nv_bfloat16*>(y), static_cast<const int*>(route_pos), static_cast<const float*>(topk_w), k, H,
      static_cast<const __nv_bfloat16*>(residual), static_cast<__nv_bfloat16*>(out));
  return static_cast<int>(cudaGetLastError());
}

}  // extern "C"
