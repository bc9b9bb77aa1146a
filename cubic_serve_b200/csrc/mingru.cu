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

// 1 / (1 + e^-(v + bias)): as exact as fp32 goes for fp32 models; for bf16 models the device's approximate exponential and reciprocal
// without their handling of ranges that cannot occur (a power that is too large makes the sigmoid zero).  `scaled` is the bias as
// gru_bias makes it.
__device__ __forceinline__ float gru_exp2(float x) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
__device__ __forceinline__ float gru_reciprocal(float x) {
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
static constexpr float kGruLog2e = 1.4426950408889634f;
template <typename T> __device__ __forceinline__ float gru_bias(float bias) { return sizeof(T) == 2 ? -kGruLog2e * bias : bias; }
template <typename T>
__device__ __forceinline__ float gru_sigmoid(float v, float scaled) {
  if constexpr (sizeof(T) == 2) return gru_reciprocal(1.f + gru_exp2(fmaf(v, -kGruLog2e, scaled)));
  else return 1.f / (1.f + expf(-(v + scaled)));
}
template <typename T>
__device__ __forceinline__ float gru_candidate(float u, float bias, float scaled) {
  const float v = u + bias;
  return v >= 0.f ? v + 0.5f : gru_sigmoid<T>(u, scaled);
}
template <typename T> __device__ __forceinline__ float gru_silu(float v) { return v * gru_sigmoid<T>(v, 0.f); }

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
  __shared__ __align__(16) float2 maps[2][kGruWarps][32][N];
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
  float bz[N], bx[N], sx[N], S[N];
#pragma unroll
  for (int k = 0; k < N; ++k) {
    bz[k] = gru_bias<T>(p.bias[c + k]);
    bx[k] = p.bias[p.width + c + k];
    sx[k] = gru_bias<T>(bx[k]);
    S[k] = p.sg.pos0[s] > 0 ? st[k] : 0.f;  // the same in every warp
  }
  if constexpr (CLUSTER) cluster_sync_all();        // every block has read the old state
  Raw zr[kGruRun] = {}, xr[kGruRun] = {}, gr[kGruRun] = {};
  auto load = [&](int t0) {
    const T* row = p.x + (row0 + t0) * p.ldx + c;
    const T* z = row + p.z_off;
    const T* x = row + p.x_off;
    const T* g = row + p.g_off;
    auto all = [&](auto full) {
#pragma unroll
      for (int i = 0; i < kGruRun; ++i)
        if (decltype(full)::value || t0 + i < count) {
          zr[i] = *reinterpret_cast<const Raw*>(z + i * p.ldx);
          xr[i] = *reinterpret_cast<const Raw*>(x + i * p.ldx);
          gr[i] = *reinterpret_cast<const Raw*>(g + i * p.ldx);
        }
    };
    if (t0 + kGruRun <= count) all(std::true_type{});
    else all(std::false_type{});
  };
  const int turn = kGruWarps * kGruRun;     // tokens of a block's turn
  load(rank * turn + warp * kGruRun);
  int b = 0;
  for (int base = 0; base < count; base += blocks * turn, b ^= 1) {
    const int t0 = base + rank * turn + warp * kGruRun;
    float keep[kGruRun][N], in[kGruRun][N], gate[kGruRun][N], A[N], B[N];
    auto make = [&](auto full) {
#pragma unroll
      for (int k = 0; k < N; ++k) { A[k] = 1.f; B[k] = 0.f; }
#pragma unroll
      for (int i = 0; i < kGruRun; ++i) {
        float z[N], u[N], g[N];
        gru_unpack(zr[i], z);
        gru_unpack(xr[i], u);
        gru_unpack(gr[i], g);
        const bool ok = decltype(full)::value || t0 + i < count;      // a token behind the segment changes nothing
#pragma unroll
        for (int k = 0; k < N; ++k) {
          const float zk = gru_sigmoid<T>(z[k], bz[k]);
          keep[i][k] = ok ? 1.f - zk : 1.f;
          in[i][k] = ok ? zk * gru_candidate<T>(u[k], bx[k], sx[k]) : 0.f;
          gate[i][k] = gru_silu<T>(g[k]);
          A[k] *= keep[i][k];
          B[k] = fmaf(keep[i][k], B[k], in[i][k]);
        }
      }
    };
    if (t0 + kGruRun <= count) make(std::true_type{});
    else make(std::false_type{});
#pragma unroll
    for (int k = 0; k < N; ++k) maps[b][warp][lane][k] = make_float2(A[k], B[k]);
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
          const float2 o = maps[b][w][lane][warp];
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
    float mine[N], at[N];
#pragma unroll
    for (int k = 0; k < N; ++k) mine[k] = at[k] = first[k];
#pragma unroll
    for (int w = 0; w < kGruWarps; ++w) {
      float2 m[N];
      if constexpr (N == 2) *reinterpret_cast<float4*>(m) = *reinterpret_cast<const float4*>(maps[b][w][lane]);
      else m[0] = maps[b][w][lane][0];
#pragma unroll
      for (int k = 0; k < N; ++k) {
        if (w == warp) mine[k] = at[k];
        at[k] = fmaf(m[k].x, at[k], m[k].y);
      }
    }
    if constexpr (!CLUSTER) {
#pragma unroll
      for (int k = 0; k < N; ++k) S[k] = at[k];
    }
    T* orow = p.out + (row0 + t0) * p.ldo + c;
    const int most = live ? count - t0 : 0;
#pragma unroll
    for (int i = 0; i < kGruRun; ++i) {
      float v[N];
#pragma unroll
      for (int k = 0; k < N; ++k) {
        mine[k] = fmaf(keep[i][k], mine[k], in[i][k]);
        v[k] = mine[k] * gate[i][k];
      }
      if (i < most) gru_store<N>(orow + i * p.ldo, v);
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
    const float bx = p.bias[p.width + c + i], zi = gru_sigmoid<T>(z[i], gru_bias<T>(p.bias[c + i]));
    S[i] = fmaf(1.f - zi, S[i], zi * gru_candidate<T>(u[i], bx, gru_bias<T>(bx)));
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
      // clusters share the segments where that shortens the run of waves (a block per SM) and of turns a block makes; a block's start
      // costs about a turn, meeting in a cluster a third of one
      const int n = pair ? 2 : 1, tiles = (a->width + 32 * n - 1) / (32 * n);
      const int longest = a->tokens - (seg->num - 1), turns = (longest + kGruWarps * kGruRun - 1) / (kGruWarps * kGruRun);
      auto cost = [&](int c) {
        const long long waves = (static_cast<long long>(tiles) * seg->num * c + 147) / 148, each = (turns + c - 1) / c;
        return waves * (3 * each + 3 + (c > 1 ? each : 0));
      };
      int cluster = 1;
      for (int c = 2; c <= kGruCluster && c <= turns; c *= 2)
        if (cost(c) < cost(cluster)) cluster = c;
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
