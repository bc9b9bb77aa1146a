// Row kernels and the fp32 matrix product of the layered decoders (models/layered.py): the residual stream is fp32, a
// layer's norm writes the activation type T (bf16, or fp32 when the model runs in 32-bit).
#include "segments.cuh"
#include "launch.cuh"

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
};

__global__ void __launch_bounds__(256)
f32_gemm_kernel(const F32Gemm p) {
  constexpr int BM = 64, BN = 64, BK = 16;
  __shared__ float xs[BK][BM + 4];
  __shared__ float ws[BK][BN + 4];
  const int m0 = blockIdx.y * BM, n0 = blockIdx.x * BN;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  pdl_wait();
  pdl_launch_dependents();
  const int xc0 = p.diag_n ? (n0 / p.diag_n) * p.K : 0;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += BK) {
    for (int i = threadIdx.x; i < BM * BK; i += 256) {
      const int r = i / BK, k = i % BK;
      const int m = m0 + r, c = xc0 + k0 + k;
      xs[k][r] = (m < p.M && k0 + k < p.K && c < p.x_cols) ? p.x[static_cast<size_t>(m) * p.ldx + c] : 0.f;
      const int n = n0 + r;
      ws[k][r] = (n < p.N && k0 + k < p.K) ? __bfloat162float(p.w[static_cast<size_t>(n) * p.K + k0 + k]) : 0.f;
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
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= p.M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= p.N) continue;
      float v = acc[i][j];
      if (p.y2 && n >= p.n_split) {
        v = fmaxf(v, 0.f);
        p.y2[static_cast<size_t>(m) * p.ldy2 + n - p.n_split] = v * v;
      } else {
        const size_t o = static_cast<size_t>(m) * p.ldy + n;
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

struct CbF32Gemm {
  const void* x; int ldx, x_cols;
  const void* w;
  void* y; int ldy;
  const void* residual;
  void* y2; int ldy2, n_split, diag_n;
  int M, N, K;
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
  const dim3 grid((a->N + 63) / 64, (a->M + 63) / 64);
  if (grid.y > 65535) return -12;
  return static_cast<int>(launch(f32_gemm_kernel, grid, dim3(256), 0, static_cast<cudaStream_t>(stream), p));
}

}  // extern "C"
