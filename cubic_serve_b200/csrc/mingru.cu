// Element-wise gated recurrence of the layered decoders: per channel S_t = (1 - z_t) S_(t-1) + z_t c_t, where gate z and candidate c read
// the current token only, so that a run of tokens is an affine map of the state before it: S -> A S + B with A the product of (1 - z).
//
//   mingru_walk_kernel   prompts and mixed steps: a block takes 32 channels of a segment, its warps consecutive runs of tokens at the same
//                        time.  A warp reads its run once, keeps gates and candidates in registers and leaves the run's map; every warp
//                        then composes the maps before its own (in token order) and walks its run from the state it got.
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

__device__ __forceinline__ float gru_sigmoid(float v) { return 1.f / (1.f + expf(-v)); }
__device__ __forceinline__ float gru_candidate(float u) { return u >= 0.f ? u + 0.5f : gru_sigmoid(u); }
__device__ __forceinline__ float gru_silu(float v) { return v / (1.f + expf(-v)); }

static constexpr int kGruWarps = 16;
static constexpr int kGruRun = 8;           // tokens of a warp's run

template <typename T>
__global__ void __launch_bounds__(32 * kGruWarps)
mingru_walk_kernel(const MinGru<T> p) {
  __shared__ float2 maps[2][kGruWarps][32];
  pdl_wait();
  pdl_launch_dependents();
  const int s = blockIdx.y;
  const int count = p.sg.count[s];
  if (count <= 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, ch = blockIdx.x * 32 + lane;
  const bool live = ch < p.width;
  const int c = live ? ch : 0;
  const size_t row0 = p.sg.row0[s];
  float* st = p.state + static_cast<size_t>(p.sg.slot[s]) * p.lds + c;
  const float bz = p.bias[c], bx = p.bias[p.width + c];
  float S = p.sg.pos0[s] > 0 ? *st : 0.f;   // the same in every warp
  T zr[kGruRun], xr[kGruRun], gr[kGruRun];
  auto load = [&](int t0) {
    const T* row = p.x + (row0 + t0) * p.ldx + c;
#pragma unroll
    for (int i = 0; i < kGruRun; ++i)
      if (t0 + i < count) {
        zr[i] = row[static_cast<size_t>(i) * p.ldx + p.z_off];
        xr[i] = row[static_cast<size_t>(i) * p.ldx + p.x_off];
        gr[i] = row[static_cast<size_t>(i) * p.ldx + p.g_off];
      }
  };
  load(warp * kGruRun);
  int b = 0;
  for (int base = 0; base < count; base += kGruWarps * kGruRun, b ^= 1) {
    const int t0 = base + warp * kGruRun;
    float keep[kGruRun], in[kGruRun], gate[kGruRun];
    float A = 1.f, B = 0.f;
#pragma unroll
    for (int i = 0; i < kGruRun; ++i) {
      keep[i] = 1.f; in[i] = 0.f; gate[i] = 0.f;
      if (t0 + i < count) {
        const float z = gru_sigmoid(to_f(zr[i]) + bz);
        keep[i] = 1.f - z;
        in[i] = z * gru_candidate(to_f(xr[i]) + bx);
        gate[i] = gru_silu(to_f(gr[i]));
      }
      A *= keep[i];
      B = fmaf(keep[i], B, in[i]);
    }
    maps[b][warp][lane] = make_float2(A, B);
    load(t0 + kGruWarps * kGruRun);         // the next run's projections are on their way (nothing behind the segment)
    __syncthreads();                        // two buffers: the next turn's maps are written behind this turn's barrier only
    float mine = S;
#pragma unroll
    for (int w = 0; w < kGruWarps; ++w) {
      if (w == warp) mine = S;
      const float2 m = maps[b][w][lane];
      S = fmaf(m.x, S, m.y);
    }
    T* orow = p.out + (row0 + t0) * p.ldo + c;
#pragma unroll
    for (int i = 0; i < kGruRun; ++i) {
      mine = fmaf(keep[i], mine, in[i]);
      if (live && t0 + i < count) orow[static_cast<size_t>(i) * p.ldo] = from_f<T>(mine * gate[i]);
    }
  }
  // every warp has read the old state before the first barrier
  if (warp == 0 && live) *st = S;
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
  float z[N], u[N], g[N], S[N];
  auto two = [](const T* src, float (&v)[N]) {
    if constexpr (N == 1) {
      v[0] = to_f(src[0]);
    } else if constexpr (sizeof(T) == 2) {
      const float2 w = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(src));
      v[0] = w.x; v[1] = w.y;
    } else {
      const float2 w = *reinterpret_cast<const float2*>(src);
      v[0] = w.x; v[1] = w.y;
    }
  };
  two(xr + p.z_off, z);
  two(xr + p.x_off, u);
  two(xr + p.g_off, g);
#pragma unroll
  for (int i = 0; i < N; ++i) S[i] = fresh ? 0.f : st[i];
  T* orow = p.out + row * p.ldo + c;
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const float zi = gru_sigmoid(z[i] + p.bias[c + i]);
    S[i] = fmaf(1.f - zi, S[i], zi * gru_candidate(u[i] + p.bias[p.width + c + i]));
    st[i] = S[i];
    S[i] *= gru_silu(g[i]);
  }
  if constexpr (N == 2 && sizeof(T) == 2) {
    *reinterpret_cast<uint32_t*>(orow) = pack_bf16x2(S[0], S[1]);
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) orow[i] = from_f<T>(S[i]);
  }
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
    if (!step)
      return static_cast<int>(launch(mingru_walk_kernel<T>, dim3((a->width + 31) / 32, seg->num), dim3(32 * kGruWarps), 0, st, p));
    const int per = (pair ? 2 : 1) * kGruStepThreads;
    const dim3 grid((a->width + per - 1) / per, seg->num);
    return static_cast<int>(pair ? launch(mingru_step_kernel<T, 2>, grid, dim3(kGruStepThreads), 0, st, p)
                                 : launch(mingru_step_kernel<T, 1>, grid, dim3(kGruStepThreads), 0, st, p));
  };
  return a->f32 ? go(MinGru<float>{}) : go(MinGru<__nv_bfloat16>{});
}

}  // extern "C"
