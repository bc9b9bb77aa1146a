// Row kernels and the fp32 matrix product of the layered decoders (models/layered.py): the residual stream is fp32, a
// layer's norm writes the activation type T (bf16, or fp32 when the model runs in 32-bit).
#include "segments.cuh"
#include "launch.cuh"
#include "mma.cuh"

namespace cb {

static constexpr int kRowThreads = 256;

__device__ __forceinline__ float row_sum(float v, float* red) {
  v = warp_sum(v);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
  if (l == 0) red[w] = v;
  __syncthreads();
  float t = (l < (blockDim.x >> 5)) ? red[l] : 0.f;
  return warp_sum(t);
}

// out[i] = x[row] * w / rms(x[row]) with row = rows ? rows[i] : i; w is the whole factor (1 + stored weight).
template <typename T>
__global__ void __launch_bounds__(kRowThreads)
row_norm_kernel(const float* __restrict__ x, const long long* __restrict__ rows, const float* __restrict__ w,
                T* __restrict__ out, int ldo, int W, float eps) {
  __shared__ float red[8];
  pdl_wait();
  pdl_launch_dependents();
  const size_t row = rows ? static_cast<size_t>(rows[blockIdx.x]) : blockIdx.x;
  const float* xr = x + row * W;
  T* orow = out + static_cast<size_t>(blockIdx.x) * ldo;
  float ss = 0.f;
  if ((W & 3) == 0) {
    // up to eight float4 per thread stay in registers (8192 columns); wider rows are read again
    float4 v[8];
    const int nv = W >> 2;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int c = threadIdx.x + i * kRowThreads;
      if (c < nv) {
        v[i] = reinterpret_cast<const float4*>(xr)[c];
        ss = fmaf(v[i].x, v[i].x, ss); ss = fmaf(v[i].y, v[i].y, ss);
        ss = fmaf(v[i].z, v[i].z, ss); ss = fmaf(v[i].w, v[i].w, ss);
      }
    }
    for (int c = threadIdx.x + 8 * kRowThreads; c < nv; c += kRowThreads) {
      const float4 t = reinterpret_cast<const float4*>(xr)[c];
      ss += t.x * t.x + t.y * t.y + t.z * t.z + t.w * t.w;
    }
    const float inv = 1.f / sqrtf(row_sum(ss, red) / static_cast<float>(W) + eps);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int c = threadIdx.x + i * kRowThreads;
      if (c < nv) {
        const float4 wv = reinterpret_cast<const float4*>(w)[c];
        const float a = v[i].x * inv * wv.x, b = v[i].y * inv * wv.y, d = v[i].z * inv * wv.z, e = v[i].w * inv * wv.w;
        if constexpr (sizeof(T) == 2)
          reinterpret_cast<uint2*>(orow)[c] = make_uint2(pack_bf16x2(a, b), pack_bf16x2(d, e));
        else
          reinterpret_cast<float4*>(orow)[c] = make_float4(a, b, d, e);
      }
    }
    for (int c = 4 * (threadIdx.x + 8 * kRowThreads); c < W; c += 4 * kRowThreads)
      for (int j = 0; j < 4; ++j) orow[c + j] = from_f<T>(xr[c + j] * inv * w[c + j]);
  } else {
    for (int c = threadIdx.x; c < W; c += kRowThreads) ss = fmaf(xr[c], xr[c], ss);
    const float inv = 1.f / sqrtf(row_sum(ss, red) / static_cast<float>(W) + eps);
    for (int c = threadIdx.x; c < W; c += kRowThreads) orow[c] = from_f<T>(xr[c] * inv * w[c]);
  }
}

// x[t] = x0[t] = norm(table[ids[t]]); x0 may be null.
__global__ void __launch_bounds__(kRowThreads)
embed_norm_kernel(const int* __restrict__ ids, const __nv_bfloat16* __restrict__ table, const float* __restrict__ w,
                  float* __restrict__ x, float* __restrict__ x0, int W, int vocab, float eps) {
  __shared__ float red[8];
  pdl_wait();
  pdl_launch_dependents();
  const size_t t = blockIdx.x;
  const int id = min(max(ids[t], 0), vocab - 1);       // admission checks the range; a stray id never reads outside
  const __nv_bfloat16* e = table + static_cast<size_t>(id) * W;
  float ss = 0.f;
  for (int c = threadIdx.x; c < W; c += kRowThreads) {
    const float v = __bfloat162float(e[c]);
    ss = fmaf(v, v, ss);
  }
  const float inv = 1.f / sqrtf(row_sum(ss, red) / static_cast<float>(W) + eps);
  for (int c = threadIdx.x; c < W; c += kRowThreads) {
    const float v = __bfloat162float(e[c]) * inv * w[c];
    x[t * W + c] = v;
    if (x0) x0[t * W + c] = v;
  }
}

// out[t] = [x[t] ; x0[t]] in the activation type (input of a loop pass's entry projection)
template <typename T>
__global__ void __launch_bounds__(kRowThreads)
concat_rows_kernel(const float* __restrict__ x, const float* __restrict__ x0, T* __restrict__ out, int ldo, int W) {
  pdl_wait();
  pdl_launch_dependents();
  const size_t t = blockIdx.x;
  for (int c = threadIdx.x; c < W; c += kRowThreads) {
    out[t * ldo + c] = from_f<T>(x[t * W + c]);
    out[t * ldo + W + c] = from_f<T>(x0[t * W + c]);
  }
}

// A row of up to 8192 columns (a multiple of 4) over the block's threads in registers, four columns at a time.
struct Row8 {
  float4 v[8];
  template <typename F> __device__ __forceinline__ void each(int W, F f) {
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int c = threadIdx.x + i * kRowThreads;
      if (c < (W >> 2)) f(c, v[i]);
    }
  }
};
__device__ __forceinline__ float dot4(float4 a, float4 b) { return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, a.w * b.w))); }
__device__ __forceinline__ float4 load4(const float* p, int c) { return reinterpret_cast<const float4*>(p)[c]; }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p, int c) {
  const uint2 u = reinterpret_cast<const uint2*>(p)[c];
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, int c, float4 v) { reinterpret_cast<float4*>(p)[c] = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, int c, float4 v) {
  reinterpret_cast<uint2*>(p)[c] = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}

// x[t] = scale * table[ids[t]] (fp32), added to what x[t] holds with `add`, and h[t] = x[t] * w / rms(x[t])
template <typename T>
__global__ void __launch_bounds__(kRowThreads)
embed_rows_kernel(const int* __restrict__ ids, const __nv_bfloat16* __restrict__ table, const float* __restrict__ w,
                  float* __restrict__ x, T* __restrict__ h, int ldh, int W, int vocab, float eps, float scale, int add) {
  __shared__ float red[8];
  pdl_wait();
  pdl_launch_dependents();
  const size_t t = blockIdx.x;
  const int id = min(max(ids[t], 0), vocab - 1);
  const __nv_bfloat16* e = table + static_cast<size_t>(id) * W;
  float* xr = x + t * W;
  T* hr = h + t * ldh;
  float ss = 0.f;
  if ((W & 3) == 0 && W <= 32 * kRowThreads) {
    Row8 r;
    r.each(W, [&](int c, float4& v) {
      v = load4(e, c);
      v = make_float4(v.x * scale, v.y * scale, v.z * scale, v.w * scale);
      if (add) {
        const float4 u = load4(xr, c);
        v = make_float4(v.x + u.x, v.y + u.y, v.z + u.z, v.w + u.w);
      }
      ss += dot4(v, v);
      store4(xr, c, v);
    });
    const float inv = 1.f / sqrtf(row_sum(ss, red) / static_cast<float>(W) + eps);
    r.each(W, [&](int c, float4& v) {
      const float4 g = load4(w, c);
      store4(hr, c, make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w));
    });
    return;
  }
  for (int c = threadIdx.x; c < W; c += kRowThreads) {
    const float v = fmaf(__bfloat162float(e[c]), scale, add ? xr[c] : 0.f);
    ss = fmaf(v, v, ss);
    xr[c] = v;
  }
  const float inv = 1.f / sqrtf(row_sum(ss, red) / static_cast<float>(W) + eps);
  for (int c = threadIdx.x; c < W; c += kRowThreads) hr[c] = from_f<T>(xr[c] * inv * w[c]);
}

// x[t] += y[t] * w / rms(y[t]); then, with h, h[t] = x[t] * w2 / rms(x[t]): a normed addition to the residual and the norm that
// reads it next
template <typename T>
__global__ void __launch_bounds__(kRowThreads)
add_norm_rows_kernel(const T* __restrict__ y, int ldy, const float* __restrict__ w, float* __restrict__ x,
                     const float* __restrict__ w2, T* __restrict__ h, int ldh, int W, float eps) {
  __shared__ float red[8], red2[8];
  pdl_wait();
  pdl_launch_dependents();
  const size_t t = blockIdx.x;
  const T* yr = y + t * ldy;
  float* xr = x + t * W;
  float ss = 0.f, s2 = 0.f;
  if ((W & 3) == 0 && (ldy & 3) == 0 && W <= 32 * kRowThreads) {
    Row8 r, o;
    r.each(W, [&](int c, float4& v) { v = load4(yr, c); ss += dot4(v, v); });
    o.each(W, [&](int c, float4& v) { v = load4(xr, c); });
    const float inv = 1.f / sqrtf(row_sum(ss, red) / static_cast<float>(W) + eps);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int c = threadIdx.x + i * kRowThreads;
      if (c >= (W >> 2)) continue;
      const float4 g = load4(w, c), v = r.v[i];
      float4& u = o.v[i];
      u.x = fmaf(v.x * inv, g.x, u.x); u.y = fmaf(v.y * inv, g.y, u.y);
      u.z = fmaf(v.z * inv, g.z, u.z); u.w = fmaf(v.w * inv, g.w, u.w);
      store4(xr, c, u);
      s2 += dot4(u, u);
    }
    if (!h) return;
    const float in2 = 1.f / sqrtf(row_sum(s2, red2) / static_cast<float>(W) + eps);
    T* hr = h + t * ldh;
    o.each(W, [&](int c, float4& u) {
      const float4 g = load4(w2, c);
      store4(hr, c, make_float4(u.x * in2 * g.x, u.y * in2 * g.y, u.z * in2 * g.z, u.w * in2 * g.w));
    });
    return;
  }
  for (int c = threadIdx.x; c < W; c += kRowThreads) { const float v = to_f(yr[c]); ss = fmaf(v, v, ss); }
  const float inv = 1.f / sqrtf(row_sum(ss, red) / static_cast<float>(W) + eps);
  for (int c = threadIdx.x; c < W; c += kRowThreads) {
    const float u = fmaf(to_f(yr[c]) * inv, w[c], xr[c]);
    xr[c] = u;
    s2 = fmaf(u, u, s2);
  }
  if (!h) return;
  const float in2 = 1.f / sqrtf(row_sum(s2, red2) / static_cast<float>(W) + eps);
  for (int c = threadIdx.x; c < W; c += kRowThreads) h[t * ldh + c] = from_f<T>(xr[c] * in2 * w2[c]);
}

// ------------------------------------------------------------------ gate of a token's side input
// out[t, n] = gelu_tanh(x[t] . w[n]) * table[ids[t], col + n] with few outputs n: the fp32 residual is read once and rounded on
// its way into the product (bf16 models).
struct SideGate {
  const float* x; int W;
  const __nv_bfloat16* w; int ldw;        // [dim, ldw], zero columns behind W
  const int* ids;
  const __nv_bfloat16* table; int ldt, col, vocab;
  void* out; int ldo;
  int T, dim;
};

static constexpr int kSideWarps = 8;

// A block takes 16 tokens and 8 NB outputs; its warps and the blocks of its cluster (grid.z) deal the columns of x in chunks of
// 32.  Lane (g, t4) feeds the columns 8 t4 .. + 7 of a chunk to two tensor-core steps: which column goes to which place of a step
// is the same for both operands, so 16-byte loads make the fragments.
template <int NB>
__global__ void __launch_bounds__(32 * kSideWarps)
side_gate_mma_kernel(const SideGate p) {
  __shared__ float part[kSideWarps][16][NB * 8 + 1];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  const int t0 = blockIdx.x * 16, n0 = blockIdx.y * NB * 8;
  pdl_wait();
  pdl_launch_dependents();
  float acc[NB][4] = {};
  const int chunks = (p.W + 31) / 32, step = kSideWarps * gridDim.z;
  const bool vec = (p.W & 3) == 0;
  for (int ch = blockIdx.z * kSideWarps + warp; ch < chunks; ch += step) {
    const int k = ch * 32 + 8 * t4;
    float a[2][8];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int t = t0 + g + 8 * i;
      const float* xr = p.x + static_cast<size_t>(t) * p.W + k;
#pragma unroll
      for (int j = 0; j < 8; j += 4) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (t < p.T) {
          if (vec) {
            if (k + j < p.W) v = *reinterpret_cast<const float4*>(xr + j);
          } else {
            if (k + j < p.W) v.x = xr[j];
            if (k + j + 1 < p.W) v.y = xr[j + 1];
            if (k + j + 2 < p.W) v.z = xr[j + 2];
            if (k + j + 3 < p.W) v.w = xr[j + 3];
          }
        }
        a[i][j] = v.x; a[i][j + 1] = v.y; a[i][j + 2] = v.z; a[i][j + 3] = v.w;
      }
    }
    uint4 b[NB];
#pragma unroll
    for (int n = 0; n < NB; ++n) {
      const int row = n0 + n * 8 + g;
      b[n] = row < p.dim ? *reinterpret_cast<const uint4*>(p.w + static_cast<size_t>(row) * p.ldw + k) : make_uint4(0, 0, 0, 0);
    }
    const uint32_t a0[4] = {pack_bf16x2(a[0][0], a[0][1]), pack_bf16x2(a[1][0], a[1][1]), pack_bf16x2(a[0][2], a[0][3]), pack_bf16x2(a[1][2], a[1][3])};
    const uint32_t a1[4] = {pack_bf16x2(a[0][4], a[0][5]), pack_bf16x2(a[1][4], a[1][5]), pack_bf16x2(a[0][6], a[0][7]), pack_bf16x2(a[1][6], a[1][7])};
#pragma unroll
    for (int n = 0; n < NB; ++n) {
      mma_bf16(acc[n], a0, b[n].x, b[n].y);
      mma_bf16(acc[n], a1, b[n].z, b[n].w);
    }
  }
#pragma unroll
  for (int n = 0; n < NB; ++n)
#pragma unroll
    for (int c = 0; c < 4; ++c) part[warp][g + 8 * (c >> 1)][n * 8 + 2 * t4 + (c & 1)] = acc[n][c];
  __syncthreads();
  const int cluster = gridDim.z;
  if (cluster > 1) {
    for (int i = threadIdx.x; i < 16 * NB * 8; i += blockDim.x) {
      const int r = i / (NB * 8), n = i % (NB * 8);
      float z = 0.f;
#pragma unroll
      for (int w = 0; w < kSideWarps; ++w) z += part[w][r][n];
      part[0][r][n] = z;
    }
    __syncwarp();
    cluster_sync_all();
  }
  // the blocks of a cluster share the rows
  for (int i = threadIdx.x + blockIdx.z * blockDim.x; i < 16 * NB * 8; i += blockDim.x * cluster) {
    const int r = i / (NB * 8), n = i % (NB * 8), t = t0 + r;
    if (t >= p.T || n0 + n >= p.dim) continue;
    float z = 0.f;
    if (cluster > 1) {
      const uint32_t at = smem_u32(&part[0][r][n]);
      float v[8];
#pragma unroll
      for (int c = 0; c < 8; ++c) v[c] = c < cluster ? ld_cluster_f32(cluster_map(at, c)) : 0.f;
      z = ((v[0] + v[1]) + (v[2] + v[3])) + ((v[4] + v[5]) + (v[6] + v[7]));
    } else {
#pragma unroll
      for (int w = 0; w < kSideWarps; ++w) z += part[w][r][n];
    }
    const int id = min(max(p.ids[t], 0), p.vocab - 1);
    const float e = __bfloat162float(p.table[static_cast<size_t>(id) * p.ldt + p.col + n0 + n]);
    static_cast<__nv_bfloat16*>(p.out)[static_cast<size_t>(t) * p.ldo + n0 + n] = __float2bfloat16(gelu_tanh_fast(z) * e);
  }
  __syncwarp();
  if (cluster > 1) cluster_sync_all();                   // nobody leaves while others read its sums
}

// The same in 32-bit, a block per token and a warp per output.
__global__ void __launch_bounds__(32 * kSideWarps)
side_gate_f32_kernel(const SideGate p) {
  pdl_wait();
  pdl_launch_dependents();
  const size_t t = blockIdx.x;
  const int lane = threadIdx.x & 31;
  const float* xr = p.x + t * p.W;
  const int id = min(max(p.ids[t], 0), p.vocab - 1);
  for (int n = threadIdx.x >> 5; n < p.dim; n += kSideWarps) {
    const __nv_bfloat16* wr = p.w + static_cast<size_t>(n) * p.ldw;
    float z = 0.f;
    for (int c = lane; c < p.W; c += 32) z = fmaf(xr[c], __bfloat162float(wr[c]), z);
    z = warp_sum(z);
    if (lane == 0)
      static_cast<float*>(p.out)[t * p.ldo + n] =
          gelu_tanh(z) * __bfloat162float(p.table[static_cast<size_t>(id) * p.ldt + p.col + n]);
  }
}

// ------------------------------------------------------------------ a layer's whole side input in one kernel
// g = gelu_tanh(x Wg) e;  y = g Wp;  x += y * norm_w / rms(y);  h = x * next_w / rms(x)   (bf16 models, up to 64 side channels)
// A cluster takes 16 tokens, each of its blocks a slice of 64 NTW columns of x: the slices' partial gates and the two row sums of
// squares meet through distributed shared memory, everything else stays in registers and x passes through once.
struct SideInput {
  SideGate s;
  float* x;                               // the gate's input, written back
  const __nv_bfloat16* proj; int ldp;     // [W, ldp], zero columns behind dim
  const float* norm_w;
  const float* next_w;                    // null: no h
  __nv_bfloat16* h; int ldh;
  float eps;
};

template <int NB, int NTW>
__global__ void __launch_bounds__(32 * kSideWarps, 2)
side_input_kernel(const SideInput p) {
  constexpr int KC = (NB * 8 + 31) / 32, LDG = 32 * KC + 8;
  __shared__ float part[kSideWarps][16][NB * 8 + 1];
  __shared__ __align__(16) __nv_bfloat16 gs[16][LDG];
  __shared__ float red[kSideWarps][16], sums[2][16], total[16];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  const int t0 = blockIdx.x * 16, W = p.s.W, T = p.s.T, cluster = gridDim.z;
  const int c_lo = blockIdx.z * 64 * NTW;
  // the slice's weights on their way into L2 while the kernel before this one ends
  for (int i = threadIdx.x; i < 64 * NTW * KC / 2; i += 32 * kSideWarps) {        // a row of the projection is 64 KC bytes
    const int n = c_lo + (KC == 1 ? 2 * i : i);
    if (n < W) asm volatile("prefetch.global.L2 [%0];" ::"l"(p.proj + static_cast<size_t>(n) * p.ldp));
  }
  pdl_wait();
  pdl_launch_dependents();
  // a thread's share of the gates, two neighbouring ones at a time, and their factors from the side embedding
  constexpr int PAIRS = 16 * NB * 4, ITER = (PAIRS + 32 * kSideWarps - 1) / (32 * kSideWarps);
  const int share = PAIRS / cluster;                       // PAIRS and the cluster are powers of two
  float e[ITER][2];
#pragma unroll
  for (int it = 0; it < ITER; ++it) {
    const int i = threadIdx.x + it * 32 * kSideWarps, idx = blockIdx.z * share + i, t = t0 + idx / (NB * 4), n = 2 * (idx % (NB * 4));
    e[it][0] = e[it][1] = 0.f;
    if (i < share && t < T) {
      const __nv_bfloat16* er = p.s.table + static_cast<size_t>(min(max(p.s.ids[t], 0), p.s.vocab - 1)) * p.s.ldt + p.s.col;
      if (n < p.s.dim) e[it][0] = __bfloat162float(er[n]);
      if (n + 1 < p.s.dim) e[it][1] = __bfloat162float(er[n + 1]);
    }
  }
  auto meet = [&]() {                     // barrier of everybody who works on the tokens
    __syncwarp();
    if (cluster > 1) cluster_sync_all();
    else __syncthreads();
  };
  // ---- partial gates of this slice
  {
    float acc[NB][4] = {};
#pragma unroll
    for (int j = 0; j < 2 * NTW / kSideWarps; ++j) {
      const int ch = warp + j * kSideWarps;
      const int k = c_lo + ch * 32 + 8 * t4;               // W is a multiple of 8: all of a lane's columns exist, or none
      float a[2][8];
      uint4 b[NB];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        float4 u = make_float4(0.f, 0.f, 0.f, 0.f), v = u;
        if (t0 + g + 8 * i < T && k < W) {
          const float* xr = p.x + static_cast<size_t>(t0 + g + 8 * i) * W + k;
          u = *reinterpret_cast<const float4*>(xr);
          v = *reinterpret_cast<const float4*>(xr + 4);
        }
        a[i][0] = u.x; a[i][1] = u.y; a[i][2] = u.z; a[i][3] = u.w;
        a[i][4] = v.x; a[i][5] = v.y; a[i][6] = v.z; a[i][7] = v.w;
      }
#pragma unroll
      for (int n = 0; n < NB; ++n)
        b[n] = n * 8 + g < p.s.dim && k < W ? *reinterpret_cast<const uint4*>(p.s.w + static_cast<size_t>(n * 8 + g) * p.s.ldw + k)
                                            : make_uint4(0, 0, 0, 0);
      const uint32_t a0[4] = {pack_bf16x2(a[0][0], a[0][1]), pack_bf16x2(a[1][0], a[1][1]), pack_bf16x2(a[0][2], a[0][3]), pack_bf16x2(a[1][2], a[1][3])};
      const uint32_t a1[4] = {pack_bf16x2(a[0][4], a[0][5]), pack_bf16x2(a[1][4], a[1][5]), pack_bf16x2(a[0][6], a[0][7]), pack_bf16x2(a[1][6], a[1][7])};
#pragma unroll
      for (int n = 0; n < NB; ++n) {
        mma_bf16(acc[n], a0, b[n].x, b[n].y);
        mma_bf16(acc[n], a1, b[n].z, b[n].w);
      }
    }
#pragma unroll
    for (int n = 0; n < NB; ++n)
#pragma unroll
      for (int c = 0; c < 4; ++c) part[warp][g + 8 * (c >> 1)][n * 8 + 2 * t4 + (c & 1)] = acc[n][c];
  }
  __syncthreads();
  for (int i = threadIdx.x; i < 16 * NB * 8; i += 32 * kSideWarps) {
    const int r = i / (NB * 8), n = i % (NB * 8);
    float z = 0.f;
#pragma unroll
    for (int w = 0; w < kSideWarps; ++w) z += part[w][r][n];
    part[0][r][n] = z;
  }
  meet();
  // every block finishes its share of the gates and hands them to all of the cluster
  {
#pragma unroll
    for (int it = 0; it < ITER; ++it) {
      const int i = threadIdx.x + it * 32 * kSideWarps, idx = blockIdx.z * share + i, r = idx / (NB * 4), n = 2 * (idx % (NB * 4));
      if (i >= share) break;
      float v[2][8];
      const uint32_t at = smem_u32(&part[0][r][n]);
#pragma unroll
      for (int c = 0; c < 8; ++c) {                        // all in flight at once
        const bool there = cluster > 1 && c < cluster;
        v[0][c] = there ? ld_cluster_f32(cluster_map(at, c)) : 0.f;
        v[1][c] = there ? ld_cluster_f32(cluster_map(at, c) + 4) : 0.f;
      }
      float z[2];
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        z[k] = cluster > 1 ? ((v[k][0] + v[k][1]) + (v[k][2] + v[k][3])) + ((v[k][4] + v[k][5]) + (v[k][6] + v[k][7])) : part[0][r][n + k];
        z[k] = gelu_tanh_fast(z[k]) * e[it][k];
      }
      const uint32_t both = pack_bf16x2(z[0], z[1]), dst = smem_u32(&gs[r][n]);
      if (cluster > 1)
        for (int c = 0; c < cluster; ++c) st_cluster_u32(cluster_map(dst, c), both);
      else
        *reinterpret_cast<uint32_t*>(&gs[r][n]) = both;
    }
    if constexpr (NB * 8 < 32 * KC) {                      // columns behind the gates
      constexpr int REST = 32 * KC - NB * 8;
      for (int i = threadIdx.x; i < 16 * REST; i += 32 * kSideWarps) gs[i / REST][NB * 8 + i % REST] = __float2bfloat16(0.f);
    }
  }
  meet();
  // ---- y of this slice: a warp's 8 NTW columns in registers
  uint4 ga[KC][2];
#pragma unroll
  for (int c = 0; c < KC; ++c)
#pragma unroll
    for (int i = 0; i < 2; ++i) ga[c][i] = *reinterpret_cast<const uint4*>(&gs[g + 8 * i][32 * c + 8 * t4]);
  const int c_w = c_lo + warp * 8 * NTW;
  float y[NTW][4], ss[2] = {0.f, 0.f};
#pragma unroll
  for (int j = 0; j < NTW; ++j) {
    const int n = c_w + 8 * j + g;
#pragma unroll
    for (int c = 0; c < 4; ++c) y[j][c] = 0.f;
#pragma unroll
    for (int c = 0; c < KC; ++c) {
      const uint4 b = n < W ? *reinterpret_cast<const uint4*>(p.proj + static_cast<size_t>(n) * p.ldp + 32 * c + 8 * t4) : make_uint4(0, 0, 0, 0);
      const uint32_t a0[4] = {ga[c][0].x, ga[c][1].x, ga[c][0].y, ga[c][1].y}, a1[4] = {ga[c][0].z, ga[c][1].z, ga[c][0].w, ga[c][1].w};
      mma_bf16(y[j], a0, b.x, b.y);
      mma_bf16(y[j], a1, b.z, b.w);
    }
    ss[0] = fmaf(y[j][0], y[j][0], fmaf(y[j][1], y[j][1], ss[0]));
    ss[1] = fmaf(y[j][2], y[j][2], fmaf(y[j][3], y[j][3], ss[1]));
  }
  // 1 / rms of the thread's two rows from their sums of squares
  auto inv_rms = [&](int which, float (&q)[2]) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      q[i] += __shfl_xor_sync(0xffffffffu, q[i], 1);
      q[i] += __shfl_xor_sync(0xffffffffu, q[i], 2);
      if (t4 == 0) red[warp][g + 8 * i] = q[i];
    }
    __syncthreads();
    if (threadIdx.x < 16) {
      float z = 0.f;
#pragma unroll
      for (int w = 0; w < kSideWarps; ++w) z += red[w][threadIdx.x];
      sums[which][threadIdx.x] = z;
    }
    meet();
    if (cluster > 1) {                                     // eight lanes add a row's parts
      if (threadIdx.x < 128) {
        const int r = threadIdx.x >> 3, c = threadIdx.x & 7;
        float z = c < cluster ? ld_cluster_f32(cluster_map(smem_u32(&sums[which][r]), c)) : 0.f;
        z += __shfl_xor_sync(0xffffffffu, z, 1);
        z += __shfl_xor_sync(0xffffffffu, z, 2);
        z += __shfl_xor_sync(0xffffffffu, z, 4);
        if (c == 0) total[r] = z;
      }
      __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 2; ++i)
      q[i] = 1.f / sqrtf((cluster > 1 ? total : sums[which])[g + 8 * i] / static_cast<float>(W) + p.eps);
  };
  // x in the products' layout, eight column tiles at a time: all loads of a batch before its stores
  float2 xv[8][2];
  auto load_x = [&](int j0) {
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int c = c_w + 8 * (j0 + j) + 2 * t4, t = t0 + g + 8 * i;
        xv[j][i] = make_float2(0.f, 0.f);
        if (c < W && t < T) xv[j][i] = *reinterpret_cast<const float2*>(p.x + static_cast<size_t>(t) * W + c);
      }
  };
  auto weight2 = [&](const float* w, int c) { return c < W ? __ldg(reinterpret_cast<const float2*>(w + c)) : make_float2(0.f, 0.f); };
  load_x(0);
  inv_rms(0, ss);
  float s2[2] = {0.f, 0.f};
#pragma unroll
  for (int j0 = 0; j0 < NTW; j0 += 8) {
    if (j0) load_x(j0);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int c = c_w + 8 * (j0 + j) + 2 * t4;
      const float2 w = weight2(p.norm_w, c);
      float (&yj)[4] = y[j0 + j];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = t0 + g + 8 * i;
        yj[2 * i] = fmaf(yj[2 * i] * ss[i], w.x, xv[j][i].x);
        yj[2 * i + 1] = fmaf(yj[2 * i + 1] * ss[i], w.y, xv[j][i].y);
        if (c < W && t < T) *reinterpret_cast<float2*>(p.x + static_cast<size_t>(t) * W + c) = make_float2(yj[2 * i], yj[2 * i + 1]);
        s2[i] = fmaf(yj[2 * i], yj[2 * i], fmaf(yj[2 * i + 1], yj[2 * i + 1], s2[i]));
      }
    }
  }
  if (p.next_w) {
    inv_rms(1, s2);
    __syncwarp();
    if (cluster > 1) cluster_arrive();    // this block has read what it needs of the others
#pragma unroll
    for (int j = 0; j < NTW; ++j) {
      const int c = c_w + 8 * j + 2 * t4;
      const float2 w = weight2(p.next_w, c);
#pragma unroll
      for (int i = 0; i < 2; ++i)
        if (c < W && t0 + g + 8 * i < T)
          *reinterpret_cast<uint32_t*>(p.h + static_cast<size_t>(t0 + g + 8 * i) * p.ldh + c) =
              pack_bf16x2(y[j][2 * i] * s2[i] * w.x, y[j][2 * i + 1] * s2[i] * w.y);
    }
  } else if (cluster > 1) {
    __syncwarp();
    cluster_arrive();
  }
  __syncwarp();
  if (cluster > 1) cluster_wait();        // nobody leaves while others read its sums
}

// ------------------------------------------------------------------ fp32 matrix product
// y[m, n] = sum_k x[m, k] w[n, k] with fp32 x and bf16-stored weights (exact in fp32), fused multiply-adds in k order:
// the product of a model that runs in 32-bit.  64 x 64 tile, 4 x 4 results per thread.  Epilogue and block-diagonal
// weights as in the wide bf16 GEMM (wq_gemm_common.cuh).
struct F32Gemm {
  const float* x; int ldx, x_cols;
  const __nv_bfloat16* w;
  float* y; int ldy;
  const float* residual;
  float* y2; int ldy2, n_split, diag_n;
  int M, N, K;
  int glu;                    // gated silu (1), gelu (2) or clamped (3): 16 gate rows and 16 up rows of w in turn, y gets N / 2 features;
                              // with y2 only the rows below n_split are, and the others leave to y2 as they are
  float glu_limit;
  const float* rgate; int ldrg;     // [M, ldrg] or null: a feature times sigmoid(rgate[m, n] + rgate_b[n]) joins the residual
  const float* rgate_b;       // [N]
  const int* tiles;           // grouped: work list {count, then {expert, first row, up to 64 rows}}, w stacks the experts; null: one matrix
};

__global__ void __launch_bounds__(256)
f32_gemm_kernel(const F32Gemm p) {
  constexpr int BM = 64, BN = 64, BK = 16;
  __shared__ float xs[BK][BM + 4];
  __shared__ float ws[BK][BN + 4];
  const int n0 = blockIdx.x * BN;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  pdl_wait();
  pdl_launch_dependents();
  int m0 = blockIdx.y * BM, m_end = p.M;
  const __nv_bfloat16* wm = p.w;
  if (p.tiles) {
    const int item = blockIdx.y;
    if (item >= p.tiles[0]) return;
    wm += static_cast<size_t>(p.tiles[1 + 3 * item]) * p.N * p.K;
    m0 = p.tiles[2 + 3 * item];
    m_end = min(p.M, m0 + min(BM, p.tiles[3 + 3 * item]));
  }
  const int xc0 = p.diag_n ? (n0 / p.diag_n) * p.K : 0;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += BK) {
    for (int i = threadIdx.x; i < BM * BK; i += 256) {
      const int r = i / BK, k = i % BK;
      const int m = m0 + r, c = xc0 + k0 + k;
      xs[k][r] = (m < m_end && k0 + k < p.K && c < p.x_cols) ? p.x[static_cast<size_t>(m) * p.ldx + c] : 0.f;
      const int n = n0 + r;
      ws[k][r] = (n < p.N && k0 + k < p.K) ? __bfloat162float(wm[static_cast<size_t>(n) * p.K + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < BK; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = xs[k][ty * 4 + i]; b[i] = ws[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
  if (p.glu && !(p.y2 && n0 >= p.n_split)) {
    // a thread's four columns are gate columns of features f .. f + 3 (tx & 4 clear) or their up columns, which the thread
    // four places on holds
    const int f = (n0 >> 1) + (tx >> 3) * 16 + (tx & 3) * 4;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int m = m0 + ty * 4 + i;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float g = acc[i][j], u = __shfl_down_sync(0xffffffffu, g, 4);
        if (p.glu == 3) {
          g = fminf(g, p.glu_limit);
          u = fminf(fmaxf(u, -p.glu_limit), p.glu_limit);
          u = (u + 1.f) / (1.f + expf(-1.702f * g));
        } else {
          g = p.glu == 1 ? g / (1.f + expf(-g)) : gelu_tanh(g);
        }
        if (!(tx & 4) && m < m_end && f + j < ((p.y2 ? p.n_split : p.N) >> 1)) p.y[static_cast<size_t>(m) * p.ldy + f + j] = g * u;
      }
    }
    return;
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= m_end) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= p.N) continue;
      float v = acc[i][j];
      if (p.y2 && n >= p.n_split) {
        if (!p.glu) {
          v = fmaxf(v, 0.f);
          v *= v;
        }
        p.y2[static_cast<size_t>(m) * p.ldy2 + n - p.n_split] = v;
      } else {
        const size_t o = static_cast<size_t>(m) * p.ldy + n;
        if (p.rgate) v /= 1.f + expf(-(p.rgate[static_cast<size_t>(m) * p.ldrg + n] + p.rgate_b[n]));
        p.y[o] = p.residual ? v + p.residual[o] : v;
      }
    }
  }
}

}  // namespace cb

extern "C" {

// `f32`: the output rows are fp32 (else bf16)
int cb_row_norm(const void* x, const void* rows, const void* w, void* out, int ldo, int n, int W, float eps, int f32,
                void* stream) {
  using namespace cb;
  if (n <= 0) return 0;
  if (W <= 0 || ldo < W || (ldo & 3)) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32)
    return static_cast<int>(launch(row_norm_kernel<float>, dim3(n), dim3(kRowThreads), 0, st, static_cast<const float*>(x),
                                   static_cast<const long long*>(rows), static_cast<const float*>(w), static_cast<float*>(out),
                                   ldo, W, eps));
  return static_cast<int>(launch(row_norm_kernel<__nv_bfloat16>, dim3(n), dim3(kRowThreads), 0, st, static_cast<const float*>(x),
                                 static_cast<const long long*>(rows), static_cast<const float*>(w),
                                 static_cast<__nv_bfloat16*>(out), ldo, W, eps));
}

int cb_embed_norm(const void* ids, const void* table, const void* w, void* x, void* x0, int n, int W, int vocab, float eps,
                  void* stream) {
  using namespace cb;
  if (n <= 0) return 0;
  if (W <= 0 || vocab <= 0) return -10;
  return static_cast<int>(launch(embed_norm_kernel, dim3(n), dim3(kRowThreads), 0, static_cast<cudaStream_t>(stream),
                                 static_cast<const int*>(ids), static_cast<const __nv_bfloat16*>(table),
                                 static_cast<const float*>(w), static_cast<float*>(x), static_cast<float*>(x0), W, vocab, eps));
}

int cb_concat_rows(const void* x, const void* x0, void* out, int ldo, int n, int W, int f32, void* stream) {
  using namespace cb;
  if (n <= 0) return 0;
  if (W <= 0 || ldo < 2 * W) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32)
    return static_cast<int>(launch(concat_rows_kernel<float>, dim3(n), dim3(kRowThreads), 0, st, static_cast<const float*>(x),
                                   static_cast<const float*>(x0), static_cast<float*>(out), ldo, W));
  return static_cast<int>(launch(concat_rows_kernel<__nv_bfloat16>, dim3(n), dim3(kRowThreads), 0, st,
                                 static_cast<const float*>(x), static_cast<const float*>(x0),
                                 static_cast<__nv_bfloat16*>(out), ldo, W));
}

int cb_embed_rows(const void* ids, const void* table, const void* w, void* x, void* h, int ldh, int n, int W, int vocab, float eps,
                  float scale, int add, int f32, void* stream) {
  using namespace cb;
  if (n <= 0) return 0;
  if (W <= 0 || vocab <= 0 || ldh < W || (ldh & 3)) return -10;
  auto go = [&](auto kernel, auto* out) {
    return static_cast<int>(launch(kernel, dim3(n), dim3(kRowThreads), 0, static_cast<cudaStream_t>(stream),
                                   static_cast<const int*>(ids), static_cast<const __nv_bfloat16*>(table),
                                   static_cast<const float*>(w), static_cast<float*>(x), out, ldh, W, vocab, eps, scale, add));
  };
  return f32 ? go(embed_rows_kernel<float>, static_cast<float*>(h)) : go(embed_rows_kernel<__nv_bfloat16>, static_cast<__nv_bfloat16*>(h));
}

// `h` may be null
int cb_add_norm_rows(const void* y, int ldy, const void* w, void* x, const void* w2, void* h, int ldh, int n, int W, float eps,
                     int f32, void* stream) {
  using namespace cb;
  if (n <= 0) return 0;
  if (W <= 0 || ldy < W || (h && (ldh < W || (ldh & 3) || !w2))) return -10;
  auto go = [&](auto kernel, auto* src) {
    using P = decltype(src);
    return static_cast<int>(launch(kernel, dim3(n), dim3(kRowThreads), 0, static_cast<cudaStream_t>(stream), src, ldy,
                                   static_cast<const float*>(w), static_cast<float*>(x), static_cast<const float*>(w2),
                                   static_cast<P>(h), ldh, W, eps));
  };
  return f32 ? go(add_norm_rows_kernel<float>, static_cast<float*>(const_cast<void*>(y)))
             : go(add_norm_rows_kernel<__nv_bfloat16>, static_cast<__nv_bfloat16*>(const_cast<void*>(y)));
}

int cb_side_gate(const void* x, int W, const void* w, int ldw, const void* ids, const void* table, int ldt, int col, void* out,
                 int ldo, int n, int dim, int vocab, int f32, void* stream) {
  using namespace cb;
  if (n <= 0) return 0;
  if (W <= 0 || dim <= 0 || vocab <= 0 || ldw < (W + 31) / 32 * 32 || (ldw & 7) || ldo < dim || col < 0 || col + dim > ldt) return -10;
  SideGate p;
  p.x = static_cast<const float*>(x); p.W = W;
  p.w = static_cast<const __nv_bfloat16*>(w); p.ldw = ldw;
  p.ids = static_cast<const int*>(ids);
  p.table = static_cast<const __nv_bfloat16*>(table); p.ldt = ldt; p.col = col; p.vocab = vocab;
  p.out = out; p.ldo = ldo; p.T = n; p.dim = dim;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32) return static_cast<int>(launch(side_gate_f32_kernel, dim3(n), dim3(32 * kSideWarps), 0, st, p));
  const int nb = dim <= 8 ? 1 : dim <= 16 ? 2 : dim <= 32 ? 4 : 8;
  const int tiles = (n + 15) / 16, ny = (dim + nb * 8 - 1) / (nb * 8);
  if (ny > 65535) return -11;
  // few tokens: a cluster shares the columns, as long as every warp of it has at least two chunks
  int cluster = 1;
  while (cluster < 8 && tiles * ny * cluster * 2 <= 148 && (W + 31) / 32 >= 4 * cluster * kSideWarps) cluster *= 2;
  const dim3 grid(tiles, ny, cluster), shape(1, 1, cluster);
  switch (nb) {
    case 1: return static_cast<int>(launch(side_gate_mma_kernel<1>, grid, dim3(32 * kSideWarps), 0, st, shape, p));
    case 2: return static_cast<int>(launch(side_gate_mma_kernel<2>, grid, dim3(32 * kSideWarps), 0, st, shape, p));
    case 4: return static_cast<int>(launch(side_gate_mma_kernel<4>, grid, dim3(32 * kSideWarps), 0, st, shape, p));
  }
  return static_cast<int>(launch(side_gate_mma_kernel<8>, grid, dim3(32 * kSideWarps), 0, st, shape, p));
}

struct CbSideInput {
  void* x;
  const void* gate; int ldw;
  const void* ids;
  const void* table; int ldt, col, vocab;
  const void* proj; int ldp;
  const void* norm_w;
  const void* next_w;         // null: no h
  void* h; int ldh;
  int n, W, dim;
  float eps;
};

// Widths and side channels the one-kernel form takes.
int cb_side_input_fits(int W, int dim) { return W > 0 && dim > 0 && (W & 7) == 0 && W <= 8192 && dim <= 64; }

int cb_side_input(const CbSideInput* a, void* stream) {
  using namespace cb;
  if (!a || a->n <= 0) return 0;
  if (!cb_side_input_fits(a->W, a->dim) || a->vocab <= 0 || a->ldw < a->W || (a->ldw & 7) || a->ldp < (a->dim + 31) / 32 * 32 || (a->ldp & 7) ||
      a->col < 0 || a->col + a->dim > a->ldt || (a->next_w && (!a->h || a->ldh < a->W || (a->ldh & 1))))
    return -10;
  SideInput p;
  p.s.x = static_cast<const float*>(a->x); p.s.W = a->W;
  p.s.w = static_cast<const __nv_bfloat16*>(a->gate); p.s.ldw = a->ldw;
  p.s.ids = static_cast<const int*>(a->ids);
  p.s.table = static_cast<const __nv_bfloat16*>(a->table); p.s.ldt = a->ldt; p.s.col = a->col; p.s.vocab = a->vocab;
  p.s.out = nullptr; p.s.ldo = 0; p.s.T = a->n; p.s.dim = a->dim;
  p.x = static_cast<float*>(a->x);
  p.proj = static_cast<const __nv_bfloat16*>(a->proj); p.ldp = a->ldp;
  p.norm_w = static_cast<const float*>(a->norm_w); p.next_w = static_cast<const float*>(a->next_w);
  p.h = static_cast<__nv_bfloat16*>(a->h); p.ldh = a->ldh; p.eps = a->eps;
  // prompts: fewer blocks share the tokens, and each has more columns to hide its waits behind
  const int ntw = a->W > 4096 || (a->n + 15) / 16 * ((a->W + 511) / 512) > 296 ? 16 : 8;
  int cluster = 1;
  while (cluster * 64 * ntw < a->W) cluster *= 2;
  const dim3 grid((a->n + 15) / 16, 1, cluster), shape(1, 1, cluster);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  auto go = [&](auto kernel) { return static_cast<int>(launch(kernel, grid, dim3(32 * kSideWarps), 0, st, shape, p)); };
  if (ntw == 16) return a->dim <= 16 ? go(side_input_kernel<2, 16>) : a->dim <= 32 ? go(side_input_kernel<4, 16>) : go(side_input_kernel<8, 16>);
  return a->dim <= 16 ? go(side_input_kernel<2, 8>) : a->dim <= 32 ? go(side_input_kernel<4, 8>) : go(side_input_kernel<8, 8>);
}

struct CbF32Gemm {
  const void* x; int ldx, x_cols;
  const void* w;
  void* y; int ldy;
  const void* residual;
  void* y2; int ldy2, n_split, diag_n;
  int M, N, K;
  int glu;
  const void* tiles; int max_items;       // grouped form (see F32Gemm)
  float glu_limit;
  const void* rgate; int ldrg;
  const void* rgate_b;
};

int cb_f32_gemm(const CbF32Gemm* a, void* stream) {
  using namespace cb;
  if (!a || a->M <= 0 || a->N <= 0 || a->K <= 0 || a->x_cols > a->ldx) return -10;
  if (a->diag_n && (a->diag_n % 64) != 0) return -11;
  F32Gemm p;
  p.x = static_cast<const float*>(a->x); p.ldx = a->ldx; p.x_cols = a->x_cols;
  p.w = static_cast<const __nv_bfloat16*>(a->w);
  p.y = static_cast<float*>(a->y); p.ldy = a->ldy;
  p.residual = static_cast<const float*>(a->residual);
  p.y2 = static_cast<float*>(a->y2); p.ldy2 = a->ldy2; p.n_split = a->n_split; p.diag_n = a->diag_n;
  p.M = a->M; p.N = a->N; p.K = a->K;
  p.glu = a->glu;
  p.tiles = static_cast<const int*>(a->tiles);
  if (p.tiles && (a->max_items <= 0 || a->diag_n || a->glu || a->residual)) return -14;
  p.glu_limit = a->glu_limit;
  p.rgate = static_cast<const float*>(a->rgate); p.ldrg = a->ldrg;
  p.rgate_b = static_cast<const float*>(a->rgate_b);
  const int glu_rows = p.y2 ? p.n_split : p.N;
  if (p.glu && (p.glu < 1 || p.glu > 3 || p.residual || p.diag_n || (glu_rows % 32) != 0 || glu_rows > p.N || p.ldy < glu_rows / 2)) return -13;
  if (p.glu && p.y2 && ((glu_rows % 64) != 0 || p.ldy2 < p.N - glu_rows)) return -15;
  if (p.rgate && (p.y2 || p.glu || !p.rgate_b || p.ldrg < p.N)) return -16;
  const dim3 grid((a->N + 63) / 64, p.tiles ? a->max_items : (a->M + 63) / 64);
  if (grid.y > 65535) return -12;
  return static_cast<int>(launch(f32_gemm_kernel, grid, dim3(256), 0, static_cast<cudaStream_t>(stream), p));
}

}  // extern "C"
