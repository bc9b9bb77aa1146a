// Several fp32 residual streams beside one another (hyper-connections): a sublayer reads a weighted sum of a token's streams, and
// its result is added to all of them while they are mixed.  The rows are [T, S, W]; a step between two sublayers passes over them
// once:
//
//   stream_embed_kernel   all streams = scale * table[id];  h = norm(sum_s in[s] x_s)
//   stream_step_kernel    x_t <- sum_s mix[s, t] x_s + out[t] y for all t at once;  h = norm(sum_s in[s] x_s) of the next sublayer.
//                         y is the sublayer's result as stored, or put together here from what a token's experts left
//   stream_norm_kernel    h = norm(sum_s in[s] x_s) of selected rows
#include <type_traits>

#include "segments.cuh"
#include "launch.cuh"

namespace cb {

static constexpr int kStreamThreads = 256;
static constexpr int kStreamMax = 8;        // streams
static constexpr int kStreamRow = 32 * kStreamThreads;     // columns of a row that a block keeps in registers

__device__ __forceinline__ float stream_row_sum(float v, float* red) {
  v = warp_sum(v);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
  if (l == 0) red[w] = v;
  __syncthreads();
  return warp_sum(l < (kStreamThreads >> 5) ? red[l] : 0.f);
}

// N neighbouring columns: 4 (rows start at multiples of four elements) or 1
template <int N> struct Cols { float v[N]; };
template <int N, typename T> __device__ __forceinline__ Cols<N> load_cols(const T* p) {
  Cols<N> r;
  if constexpr (N == 1) {
    r.v[0] = to_f(p[0]);
  } else if constexpr (sizeof(T) == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w;
  } else {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    r.v[0] = a.x; r.v[1] = a.y; r.v[2] = b.x; r.v[3] = b.y;
  }
  return r;
}
template <int N, typename T> __device__ __forceinline__ void store_cols(T* p, const Cols<N>& c) {
  if constexpr (N == 1) p[0] = from_f<T>(c.v[0]);
  else if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>(p) = make_float4(c.v[0], c.v[1], c.v[2], c.v[3]);
  else *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(c.v[0], c.v[1]), pack_bf16x2(c.v[2], c.v[3]));
}

// What a sublayer with experts left for its tokens, beside the shared expert's rows (the plain result `y`)
template <typename T>
struct StreamRoutes {
  const T* rows; int ld;      // results by place
  const int* pos;             // [T, top] place of a token's route, < 0: none
  const float* weight;        // [T, top]
  const float* self;          // [T] factor of the sublayer's input (experts that return it), null: none
  int top;                    // 0: no routes
  const float* gate; int ldg; // [T] logit of the sigmoid that scales `y`, null: 1
};

template <typename T>
struct StreamStep {
  float* x;                   // [T, S, W]
  const T* y; int ldy;        // may be null with routes
  StreamRoutes<T> r;
  const float* mix;           // [S, S] from, to
  const float* out;           // [S]
  const float* in;            // [S] of the next sublayer
  const float* w;             // [W] its norm's factor, null: no h
  T* h; int ldh;              // the sublayer's input; replaced by the next one's
  int W;
  float eps;
};

// VEC: four columns at a time, the row in registers; else column by column, any width.
template <typename T, int S, bool VEC>
__global__ void __launch_bounds__(kStreamThreads)
stream_step_kernel(const StreamStep<T> p) {
  constexpr int N = VEC ? 4 : 1, KEEP = VEC ? 8 : 1;
  __shared__ float red[kStreamThreads >> 5];
  __shared__ float rw[32];
  __shared__ int rp[32];
  float mix[S][S], out[S], in[S];
#pragma unroll
  for (int s = 0; s < S; ++s) {                       // the weights are written by no kernel
    out[s] = __ldg(p.out + s);
    in[s] = p.w ? __ldg(p.in + s) : 0.f;
#pragma unroll
    for (int t = 0; t < S; ++t) mix[s][t] = __ldg(p.mix + s * S + t);
  }
  pdl_wait();
  pdl_launch_dependents();
  const size_t tok = blockIdx.x;
  float gate = 1.f, self = 0.f;
  if (p.r.top) {
    if (static_cast<int>(threadIdx.x) < p.r.top) {
      rw[threadIdx.x] = p.r.weight[tok * p.r.top + threadIdx.x];
      rp[threadIdx.x] = p.r.pos[tok * p.r.top + threadIdx.x];
    }
    if (p.r.gate) gate = 1.f / (1.f + expf(-p.r.gate[tok * p.r.ldg]));
    if (p.r.self) self = p.r.self[tok];
    __syncthreads();
  }
  float* xr = p.x + tok * S * p.W;
  T* hr = p.h + tok * p.ldh;
  float ss = 0.f;
  Cols<N> keep[KEEP];
  auto column = [&](int c) {                          // columns c .. c + N - 1 of the new streams; returns the next input's
    Cols<N> x[S], y;
#pragma unroll
    for (int s = 0; s < S; ++s) x[s] = load_cols<N>(xr + static_cast<size_t>(s) * p.W + c);
    if (p.y) y = load_cols<N>(p.y + tok * p.ldy + c);
    else
#pragma unroll
      for (int i = 0; i < N; ++i) y.v[i] = 0.f;
    if (p.r.top) {
#pragma unroll
      for (int i = 0; i < N; ++i) y.v[i] *= gate;
      if (self != 0.f) {
        const Cols<N> h = load_cols<N>(hr + c);
#pragma unroll
        for (int i = 0; i < N; ++i) y.v[i] = fmaf(self, h.v[i], y.v[i]);
      }
      for (int k = 0; k < p.r.top; ++k) {
        if (rp[k] < 0) continue;
        const Cols<N> e = load_cols<N>(p.r.rows + static_cast<size_t>(rp[k]) * p.r.ld + c);
#pragma unroll
        for (int i = 0; i < N; ++i) y.v[i] = fmaf(rw[k], e.v[i], y.v[i]);
      }
    }
    Cols<N> u;
#pragma unroll
    for (int i = 0; i < N; ++i) u.v[i] = 0.f;
#pragma unroll
    for (int t = 0; t < S; ++t) {
      Cols<N> n;
#pragma unroll
      for (int i = 0; i < N; ++i) {
        float v = out[t] * y.v[i];
#pragma unroll
        for (int s = 0; s < S; ++s) v = fmaf(mix[s][t], x[s].v[i], v);
        n.v[i] = v;
        u.v[i] = fmaf(in[t], v, u.v[i]);
      }
      store_cols<N>(xr + static_cast<size_t>(t) * p.W + c, n);
    }
#pragma unroll
    for (int i = 0; i < N; ++i) ss = fmaf(u.v[i], u.v[i], ss);
    return u;
  };
  if constexpr (VEC) {
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int c = 4 * (threadIdx.x + i * kStreamThreads);
      if (c < p.W) keep[i] = column(c);
    }
  } else {
    for (int c = threadIdx.x; c < p.W; c += kStreamThreads) column(c);
  }
  if (!p.w) return;
  const float inv = 1.f / sqrtf(stream_row_sum(ss, red) / static_cast<float>(p.W) + p.eps);
  if constexpr (VEC) {
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int c = 4 * (threadIdx.x + i * kStreamThreads);
      if (c >= p.W) continue;
      const Cols<N> g = load_cols<N>(p.w + c);
#pragma unroll
      for (int k = 0; k < N; ++k) keep[i].v[k] *= inv * g.v[k];
      store_cols<N>(hr + c, keep[i]);
    }
  } else {
    for (int c = threadIdx.x; c < p.W; c += kStreamThreads) {          // a thread's own columns
      float u = 0.f;
#pragma unroll
      for (int s = 0; s < S; ++s) u = fmaf(in[s], xr[static_cast<size_t>(s) * p.W + c], u);
      hr[c] = from_f<T>(u * inv * p.w[c]);
    }
  }
}

template <typename T>
struct StreamNorm {
  const int* ids;             // embedding: x is written from the table
  const __nv_bfloat16* table; int vocab;
  float scale;
  float* x;
  const long long* rows;      // selected rows of x, null: all
  const float* in;            // [S], null: ones
  const float* w;
  T* h; int ldh;
  int S, W;
  float eps;
};

template <typename T, bool EMBED>
__global__ void __launch_bounds__(kStreamThreads)
stream_norm_kernel(const StreamNorm<T> p) {
  __shared__ float red[kStreamThreads >> 5];
  pdl_wait();
  pdl_launch_dependents();
  float in[kStreamMax], all = 0.f;
  for (int s = 0; s < kStreamMax; ++s) {
    in[s] = s < p.S ? (p.in ? __ldg(p.in + s) : 1.f) : 0.f;
    all += in[s];
  }
  const size_t row = !EMBED && p.rows ? static_cast<size_t>(p.rows[blockIdx.x]) : blockIdx.x;
  float* xr = p.x + row * p.S * p.W;
  T* hr = p.h + static_cast<size_t>(blockIdx.x) * p.ldh;
  const __nv_bfloat16* e = nullptr;
  if (EMBED) e = p.table + static_cast<size_t>(min(max(p.ids[row], 0), p.vocab - 1)) * p.W;
  float ss = 0.f;
  auto value = [&](int c) {
    if (EMBED) return __bfloat162float(e[c]) * p.scale * all;
    float u = 0.f;
#pragma unroll
    for (int s = 0; s < kStreamMax; ++s)
      if (s < p.S) u = fmaf(in[s], xr[static_cast<size_t>(s) * p.W + c], u);
    return u;
  };
  if ((p.W & 3) == 0) {
    auto four = [&](int c) {
      Cols<4> u;
      if (EMBED) {
        u = load_cols<4>(e + c);
#pragma unroll
        for (int i = 0; i < 4; ++i) u.v[i] *= p.scale;
      } else {
#pragma unroll
        for (int i = 0; i < 4; ++i) u.v[i] = 0.f;
#pragma unroll
        for (int s = 0; s < kStreamMax; ++s)
          if (s < p.S) {
            const Cols<4> x = load_cols<4>(xr + static_cast<size_t>(s) * p.W + c);
#pragma unroll
            for (int i = 0; i < 4; ++i) u.v[i] = fmaf(in[s], x.v[i], u.v[i]);
          }
      }
      return u;
    };
    for (int c = 4 * threadIdx.x; c < p.W; c += 4 * kStreamThreads) {
      Cols<4> u = four(c);
      if (EMBED) {
        for (int s = 0; s < p.S; ++s) store_cols<4>(xr + static_cast<size_t>(s) * p.W + c, u);
#pragma unroll
        for (int i = 0; i < 4; ++i) u.v[i] *= all;
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) ss = fmaf(u.v[i], u.v[i], ss);
    }
    const float inv = 1.f / sqrtf(stream_row_sum(ss, red) / static_cast<float>(p.W) + p.eps);
    for (int c = 4 * threadIdx.x; c < p.W; c += 4 * kStreamThreads) {
      Cols<4> u = four(c);
      const Cols<4> g = load_cols<4>(p.w + c);
#pragma unroll
      for (int i = 0; i < 4; ++i) u.v[i] *= (EMBED ? all : 1.f) * inv * g.v[i];
      store_cols<4>(hr + c, u);
    }
    return;
  }
  for (int c = threadIdx.x; c < p.W; c += kStreamThreads) {
    const float u = value(c);
    if (EMBED)
      for (int s = 0; s < p.S; ++s) xr[static_cast<size_t>(s) * p.W + c] = __bfloat162float(e[c]) * p.scale;
    ss = fmaf(u, u, ss);
  }
  const float inv = 1.f / sqrtf(stream_row_sum(ss, red) / static_cast<float>(p.W) + p.eps);
  for (int c = threadIdx.x; c < p.W; c += kStreamThreads) hr[c] = from_f<T>(value(c) * inv * p.w[c]);
}

}  // namespace cb

extern "C" {

struct CbStreamStep {
  void* x;
  const void* y; int ldy;
  const void* rows; int ld_rows;
  const void* pos;
  const void* weight;
  const void* self;
  int top;
  const void* gate; int ldg;
  const void* mix;
  const void* out;
  const void* in;
  const void* w;
  void* h; int ldh;
  int n, S, W;
  float eps;
  int f32;
};

int cb_stream_step(const CbStreamStep* a, void* stream) {
  using namespace cb;
  if (!a || a->n <= 0) return 0;
  if (a->S < 1 || a->S > kStreamMax || a->W <= 0 || !a->h || a->ldh < a->W || (a->w && !a->in) || (!a->y && a->top <= 0)) return -10;
  if (a->top < 0 || a->top > 32 || (a->top && (!a->rows || !a->pos || !a->weight || a->ld_rows < a->W)) || (a->y && a->ldy < a->W)) return -11;
  const bool vec = (a->W & 3) == 0 && (a->ldh & 3) == 0 && (a->ldy & 3) == 0 && (a->ld_rows & 3) == 0 && a->W <= kStreamRow;
  auto go = [&](auto kernel, auto* act) {
    using T = std::remove_pointer_t<decltype(act)>;
    StreamStep<T> p;
    p.x = static_cast<float*>(a->x);
    p.y = static_cast<const T*>(a->y); p.ldy = a->ldy;
    p.r.rows = static_cast<const T*>(a->rows); p.r.ld = a->ld_rows;
    p.r.pos = static_cast<const int*>(a->pos); p.r.weight = static_cast<const float*>(a->weight);
    p.r.self = static_cast<const float*>(a->self); p.r.top = a->top;
    p.r.gate = static_cast<const float*>(a->gate); p.r.ldg = a->ldg;
    p.mix = static_cast<const float*>(a->mix); p.out = static_cast<const float*>(a->out); p.in = static_cast<const float*>(a->in);
    p.w = static_cast<const float*>(a->w);
    p.h = static_cast<T*>(a->h); p.ldh = a->ldh; p.W = a->W; p.eps = a->eps;
    return static_cast<int>(launch(kernel, dim3(a->n), dim3(kStreamThreads), 0, static_cast<cudaStream_t>(stream), p));
  };
#define CB_STREAMS(N)                                                                                     \
  case N:                                                                                                 \
    if (a->f32) return vec ? go(stream_step_kernel<float, N, true>, static_cast<float*>(nullptr))         \
                           : go(stream_step_kernel<float, N, false>, static_cast<float*>(nullptr));       \
    return vec ? go(stream_step_kernel<__nv_bfloat16, N, true>, static_cast<__nv_bfloat16*>(nullptr))     \
               : go(stream_step_kernel<__nv_bfloat16, N, false>, static_cast<__nv_bfloat16*>(nullptr));
  switch (a->S) {
    CB_STREAMS(1) CB_STREAMS(2) CB_STREAMS(3) CB_STREAMS(4) CB_STREAMS(5) CB_STREAMS(6) CB_STREAMS(7) CB_STREAMS(8)
  }
#undef CB_STREAMS
  return -10;
}

struct CbStreamNorm {
  const void* ids;            // with a table: the embedding is written to x first
  const void* table; int vocab;
  float scale;
  void* x;
  const void* rows;
  const void* in;
  const void* w;
  void* h; int ldh;
  int n, S, W;
  float eps;
  int f32;
};

int cb_stream_norm(const CbStreamNorm* a, void* stream) {
  using namespace cb;
  if (!a || a->n <= 0) return 0;
  if (a->S < 1 || a->S > kStreamMax || a->W <= 0 || !a->w || a->ldh < a->W || (a->ldh & 3) || (a->table && (!a->ids || a->vocab <= 0))) return -10;
  auto go = [&](auto kernel, auto* act) {
    using T = std::remove_pointer_t<decltype(act)>;
    StreamNorm<T> p;
    p.ids = static_cast<const int*>(a->ids); p.table = static_cast<const __nv_bfloat16*>(a->table); p.vocab = a->vocab; p.scale = a->scale;
    p.x = static_cast<float*>(a->x); p.rows = static_cast<const long long*>(a->rows);
    p.in = static_cast<const float*>(a->in); p.w = static_cast<const float*>(a->w);
    p.h = static_cast<T*>(a->h); p.ldh = a->ldh; p.S = a->S; p.W = a->W; p.eps = a->eps;
    return static_cast<int>(launch(kernel, dim3(a->n), dim3(kStreamThreads), 0, static_cast<cudaStream_t>(stream), p));
  };
  if (a->f32)
    return a->table ? go(stream_norm_kernel<float, true>, static_cast<float*>(nullptr)) : go(stream_norm_kernel<float, false>, static_cast<float*>(nullptr));
  return a->table ? go(stream_norm_kernel<__nv_bfloat16, true>, static_cast<__nv_bfloat16*>(nullptr))
                  : go(stream_norm_kernel<__nv_bfloat16, false>, static_cast<__nv_bfloat16*>(nullptr));
}

}  // extern "C"
