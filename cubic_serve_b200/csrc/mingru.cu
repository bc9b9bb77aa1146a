// Element-wise gated recurrence of the layered decoders: per channel S_t = (1 - z_t) S_(t-1) + z_t c_t, where gate z and candidate c read
// the current token only, so that a run of tokens is an affine map of the state before it: S -> A S + B with A the product of (1 - z).
//
//   mingru_walk_kernel   prompts and mixed steps: a block takes the channels of a warp's lanes of a segment, its warps consecutive runs of
//                        tokens at the same time.  A warp reads its run once, keeps gates and candidates in registers and leaves the
//                        run's map; every warp then composes the maps before its own (in token order) and walks its run from the
//                        state it got.  With a cluster the blocks share a segment's tokens the same way, maps of whole blocks pass
//                        through distributed shared memory.
//   mingru_step_kernel   steps of one token per segment: a thread per two channels.
//
// Projections are activations; gates, candidates, maps and the state are fp32.
#include <type_traits>

#include "segments.cuh"
#include "launch.cuh"

namespace cb {

template <typename T>
struct MinGru {
  const T* x; int ldx;        // projections
  int z_off, x_off, g_off;    // columns of gate, candidate and output gate
  const float* bias;          // [2][width] of gate and candidate
  float* state; int lds;      // [slots][lds]
  T* out; int ldo;            // [T, width]
  int width;
  Segments sg;
};

// Sigmoids: as exact as fp32 goes for fp32 models, the device's fast exponential and quotient for bf16 models
template <typename T>
__device__ __forceinline__ float gru_sigmoid(float v) {
  if constexpr (sizeof(T) == 2) return __fdividef(1.f, 1.f + __expf(-v));
  else return 1.f / (1.f + expf(-v));
}
template <typename T> __device__ __forceinline__ float gru_candidate(float u) { return u >= 0.f ? u + 0.5f : gru_sigmoid<T>(u); }
template <typename T> __device__ __forceinline__ float gru_silu(float v) { return v * gru_sigmoid<T>(v); }

// N neighbouring channels as they are stored, and as numbers
template <typename T, int N> struct GruRaw { using type = T; };
template <> struct GruRaw<__nv_bfloat16, 2> { using type = __nv_bfloat162; };
template <> struct GruRaw<float, 2> { using type = float2; };
template <int N>
__device__ __forceinline__ void gru_unpack(float raw, float (&v)[N]) { v[0] = raw; }
template <int N>
__device__ __forceinline__ void gru_unpack(__nv_bfloat16 raw, float (&v)[N]) { v[0] = __bfloat162float(raw); }
__device__ __forceinline__ void gru_unpack(float2 raw, float (&v)[2]) { v[0] = raw.x; v[1] = raw.y; }
__device__ __forceinline__ void gru_unpack(__nv_bfloat162 raw, float (&v)[2]) {
  const float2 f = __bfloat1622float2(raw);
  v[0] = f.x; v[1] = f.y;
}
template <int N>
__device__ __forceinline__ void gru_store(float* dst, const float (&v)[N]) {
  if constexpr (N == 2) *reinterpret_cast<float2*>(dst) = make_float2(v[0], v[1]);
  else dst[0] = v[0];
}
template <int N>
__device__ __forceinline__ void gru_store(__nv_bfloat16* dst, const float (&v)[N]) {
  if constexpr (N == 2) *reinterpret_cast<uint32_t*>(dst) = pack_bf16x2(v[0], v[1]);
  else dst[0] = __float2bfloat16(v[0]);
}

static constexpr int kGruWarps = 16;
static constexpr int kGruRun = 8;           // tokens of a warp's run
static constexpr int kGruCluster = 8;       // most blocks that share a segment

// N: channels of a lane.  CLUSTER: the blocks of a cluster (along x) take consecutive turns of a segment's tokens.
template <typename T, int N, bool CLUSTER>
__global__ void __launch_bounds__(32 * kGruWarps)
mingru_walk_kernel(const MinGru<T> p) {
  using Raw = typename GruRaw<T, N>::type;
  __shared__ float2 maps[2][kGruWarps][N][32];
  __shared__ float2 whole[2][N][32];        // map of this block's tokens of a turn, read by the other blocks of its cluster
  pdl_wait();
  pdl_launch_dependents();
  const int s = blockIdx.y;
  const int count = p.sg.count[s];
  const int blocks = CLUSTER ? static_cast<int>(cluster_nctarank()) : 1, rank = CLUSTER ? static_cast<int>(cluster_ctarank()) : 0;
  if (count <= 0) return;                   // the same for all blocks of a cluster
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, ch = (blockIdx.x / blocks * 32 + lane) * N;
  const bool live = ch < p.width;           // N 2: the width is even
  const int c = live ? ch : 0;
  const size_t row0 = p.sg.row0[s];
  float* st = p.state + static_cast<size_t>(p.sg.slot[s]) * p.lds + c;
  float bz[N], bx[N], S[N];
#pragma unroll
  for (int k = 0; k < N; ++k) {
    bz[k] = p.bias[c + k];
    bx[k] = p.bias[p.width + c + k];
    S[k] = p.sg.pos0[s] > 0 ? st[k] : 0.f;  // the same in every warp
  }
  if constexpr (CLUSTER) cluster_sync_all();        // every block has read the old state
  Raw zr[kGruRun] = {}, xr[kGruRun] = {}, gr[kGruRun] = {};
  auto load = [&](int t0) {
    const T* row = p.x + (row0 + t0) * p.ldx + c;
#pragma unroll
    for (int i = 0; i < kGruRun; ++i)
      if (t0 + i < count) {
        zr[i] = *reinterpret_cast<const Raw*>(row + static_cast<size_t>(i) * p.ldx + p.z_off);
        xr[i] = *reinterpret_cast<const Raw*>(row + static_cast<size_t>(i) * p.ldx + p.x_off);
        gr[i] = *reinterpret_cast<const Raw*>(row + static_cast<size_t>(i) * p.ldx + p.g_off);
      }
  };
  const int turn = kGruWarps * kGruRun;     // tokens of a block's turn
  load(rank * turn + warp * kGruRun);
  int b = 0;
  for (int base = 0; base < count; base += blocks * turn, b ^= 1) {
    const int t0 = base + rank * turn + warp * kGruRun;
    float keep[kGruRun][N], in[kGruRun][N], gate[kGruRun][N], A[N], B[N];
#pragma unroll
    for (int k = 0; k < N; ++k) { A[k] = 1.f; B[k] = 0.f; }
#pragma unroll
    for (int i = 0; i < kGruRun; ++i) {
      float z[N], u[N], g[N];
      gru_unpack(zr[i], z);
      gru_unpack(xr[i], u);
      gru_unpack(gr[i], g);
      const bool ok = t0 + i < count;
#pragma unroll
      for (int k = 0; k < N; ++k) {
        const float zk = gru_sigmoid<T>(z[k] + bz[k]);
        keep[i][k] = ok ? 1.f - zk : 1.f;
        in[i][k] = ok ? zk * gru_candidate<T>(u[k] + bx[k]) : 0.f;
        gate[i][k] = gru_silu<T>(g[k]);
        A[k] *= keep[i][k];
        B[k] = fmaf(keep[i][k], B[k], in[i][k]);
      }
    }
#pragma unroll
    for (int k = 0; k < N; ++k) maps[b][warp][k][lane] = make_float2(A[k], B[k]);
    load(t0 + blocks * turn);               // the next run's projections are on their way (nothing behind the segment)
    __syncthreads();                        // two buffers: the next turn's maps are written behind this turn's barrier only
    float first[N];                         // state before the block's tokens
#pragma unroll
    for (int k = 0; k < N; ++k) first[k] = S[k];
    if constexpr (CLUSTER) {
      if (warp < N) {                       // a warp composes a channel of the block
        float2 m = make_float2(1.f, 0.f);
#pragma unroll
        for (int w = 0; w < kGruWarps; ++w) {
          const float2 o = maps[b][w][warp][lane];
          m = make_float2(o.x * m.x, fmaf(o.x, m.y, o.y));
        }
        whole[b][warp][lane] = m;
      }
      cluster_sync_all();
#pragma unroll
      for (int k = 0; k < N; ++k) {
        const uint32_t at = smem_u32(&whole[b][k][lane]);
        for (int r = 0; r < blocks; ++r) {
          if (r == rank) first[k] = S[k];
          const uint32_t peer = cluster_map(at, static_cast<uint32_t>(r));
          S[k] = fmaf(ld_cluster_f32(peer), S[k], ld_cluster_f32(peer + 4));
        }
      }
    }
    float mine[N];
#pragma unroll
    for (int k = 0; k < N; ++k) {
      float at = first[k];
      mine[k] = at;
#pragma unroll
      for (int w = 0; w < kGruWarps; ++w) {
        if (w == warp) mine[k] = at;
        const float2 m = maps[b][w][k][lane];
        at = fmaf(m.x, at, m.y);
      }
      if constexpr (!CLUSTER) S[k] = at;
    }
    T* orow = p.out + (row0 + t0) * p.ldo + c;
#pragma unroll
    for (int i = 0; i < kGruRun; ++i) {
      float v[N];
#pragma unroll
      for (int k = 0; k < N; ++k) {
        mine[k] = fmaf(keep[i][k], mine[k], in[i][k]);
        v[k] = mine[k] * gate[i][k];
      }
      if (live && t0 + i < count) gru_store<N>(orow + static_cast<size_t>(i) * p.ldo, v);
    }
  }
  // every warp has read the old state before the first barrier
  if (rank == 0 && warp == 0 && live) {
#pragma unroll
    for (int k = 0; k < N; ++k) st[k] = S[k];
  }
  if constexpr (CLUSTER) cluster_sync_all();        // nobody leaves while others read its maps
}

static constexpr int kGruStepThreads = 128;

// Two channels (column pairs are aligned, and the width is even) or one.
template <typename T, int N>
__global__ void __launch_bounds__(kGruStepThreads)
mingru_step_kernel(const MinGru<T> p) {
  pdl_wait();
  pdl_launch_dependents();
  const int s = blockIdx.y, c = N * (blockIdx.x * kGruStepThreads + threadIdx.x);
  if (p.sg.count[s] <= 0 || c >= p.width) return;
  const size_t row = p.sg.row0[s];
  const T* xr = p.x + row * p.ldx + c;
  float* st = p.state + static_cast<size_t>(p.sg.slot[s]) * p.lds + c;
  const bool fresh = p.sg.pos0[s] == 0;
  using Raw = typename GruRaw<T, N>::type;
  float z[N], u[N], g[N], S[N];
  gru_unpack(*reinterpret_cast<const Raw*>(xr + p.z_off), z);
  gru_unpack(*reinterpret_cast<const Raw*>(xr + p.x_off), u);
  gru_unpack(*reinterpret_cast<const Raw*>(xr + p.g_off), g);
#pragma unroll
  for (int i = 0; i < N; ++i) S[i] = fresh ? 0.f : st[i];
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const float zi = gru_sigmoid<T>(z[i] + p.bias[c + i]);
    S[i] = fmaf(1.f - zi, S[i], zi * gru_candidate<T>(u[i] + p.bias[p.width + c + i]));
    st[i] = S[i];
    S[i] *= gru_silu<T>(g[i]);
  }
  gru_store<N>(p.out + row * p.ldo + c, S);
}

}  // namespace cb

extern "C" {

struct CbMinGru {
  const void* x; int ldx, z_off, x_off, g_off;
  const void* bias;
  void* state; int lds;
  void* out; int ldo;
  int width, tokens, f32;
};

int cb_mingru(const CbMinGru* a, const CbSegments* seg, void* stream) {
  using namespace cb;
  if (!a || !seg || seg->num <= 0 || a->tokens <= 0) return 0;
  if (a->width <= 0 || a->lds < a->width || a->ldo < a->width || a->z_off < 0 || a->x_off < 0 || a->g_off < 0) return -10;
  if (a->ldx < a->width + max(a->z_off, max(a->x_off, a->g_off)) || seg->num > 65535) return -11;
  const bool step = a->tokens == seg->num;
  const bool pair = ((a->width | a->ldx | a->ldo | a->z_off | a->x_off | a->g_off) & 1) == 0;
  auto go = [&](auto p) {
    using T = std::remove_pointer_t<decltype(p.out)>;
    p.x = static_cast<const T*>(a->x); p.ldx = a->ldx; p.z_off = a->z_off; p.x_off = a->x_off; p.g_off = a->g_off;
    p.bias = static_cast<const float*>(a->bias);
    p.state = static_cast<float*>(a->state); p.lds = a->lds;
    p.out = static_cast<T*>(a->out); p.ldo = a->ldo;
    p.width = a->width;
    p.sg = make_segments(seg, a->tokens);
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (!step) {
      // few blocks: clusters share the segments, as long as the longest has a turn for every block
      const int n = pair ? 2 : 1, tiles = (a->width + 32 * n - 1) / (32 * n);
      const int longest = a->tokens - (seg->num - 1), turns = (longest + kGruWarps * kGruRun - 1) / (kGruWarps * kGruRun);
      int cluster = 1;
      while (cluster < kGruCluster && 2 * cluster <= turns && tiles * seg->num * cluster < 148) cluster *= 2;
      const dim3 grid(tiles * cluster, seg->num), block(32 * kGruWarps), shape(cluster, 1, 1);
      if (cluster > 1)
        return static_cast<int>(pair ? launch(mingru_walk_kernel<T, 2, true>, grid, block, 0, st, shape, p)
                                     : launch(mingru_walk_kernel<T, 1, true>, grid, block, 0, st, shape, p));
      return static_cast<int>(pair ? launch(mingru_walk_kernel<T, 2, false>, grid, block, 0, st, p)
                                   : launch(mingru_walk_kernel<T, 1, false>, grid, block, 0, st, p));
    }
    const int per = (pair ? 2 : 1) * kGruStepThreads;
    const dim3 grid((a->width + per - 1) / per, seg->num);
    return static_cast<int>(pair ? launch(mingru_step_kernel<T, 2>, grid, dim3(kGruStepThreads), 0, st, p)
                                 : launch(mingru_step_kernel<T, 1>, grid, dim3(kGruStepThreads), 0, st, p));
  };
  return a->f32 ? go(MinGru<float>{}) : go(MinGru<__nv_bfloat16>{});
}

}  // extern "C"
