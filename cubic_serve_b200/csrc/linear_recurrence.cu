// Additive linear recurrences: gated linear attention (a decay per key channel, no convolution) and state-space duality layers
// (a decay per head, convolution with a bias, a path from the value rows to the output), and the gated norm behind the latter.
#include "recurrence.cuh"

namespace cb {

// out = y silu(z) over its root mean square in equal parts of `width` columns, times w; a block per (part, token).
template <typename T>
__global__ void __launch_bounds__(128)
gated_parts_norm_kernel(const float* __restrict__ y, const T* __restrict__ z, int ldz, const float* __restrict__ w,
                        T* __restrict__ out, int ldo, int width, float eps) {
  __shared__ float red[4];
  pdl_wait();
  pdl_launch_dependents();
  const size_t t = blockIdx.y, c0 = static_cast<size_t>(blockIdx.x) * width;
  const float* yr = y + t * gridDim.x * width + c0;
  const T* zr = z + t * ldz + c0;
  T* dst = out + t * ldo + c0;
  auto gated = [&](int c) { return yr[c] * silu_of<T>(to_f(zr[c])); };
  float v[8], ss = 0.f;                                  // up to 1024 columns in registers
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int c = threadIdx.x + 128 * i;
    v[i] = c < width ? gated(c) : 0.f;
    ss = fmaf(v[i], v[i], ss);
  }
  for (int c = threadIdx.x + 1024; c < width; c += 128) { const float u = gated(c); ss = fmaf(u, u, ss); }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  const float inv = 1.f / sqrtf((red[0] + red[1] + red[2] + red[3]) / static_cast<float>(width) + eps);
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int c = threadIdx.x + 128 * i;
    if (c < width) dst[c] = from_f<T>(v[i] * inv * w[c0 + c]);
  }
  for (int c = threadIdx.x + 1024; c < width; c += 128) dst[c] = from_f<T>(gated(c) * inv * w[c0 + c]);
}

}  // namespace cb

extern "C" {

// Gated linear attention: q, k [H d] and v [H e] at their columns of x; a: decay logits [H d], or with `low` the inner columns of
// their low-rank projection (low_k of them readable, zero from low_rank on).
int cb_gated_linear_prepare(const CbRecPrep* a, const CbSegments* seg, void* stream) {
  if (!a || !seg || seg->num <= 0 || a->tokens <= 0) return 0;
  if (!cb::recurrence_sizes_ok(a->H, a->G, a->d, a->e, a->ds, a->es, seg) || a->G != a->H || !a->g || (a->ldx & 1)) return -10;
  if (a->low && (a->f32 || (a->lda & 7) || (a->low_k & 7) || a->low_rank <= 0 || a->low_rank > a->low_k || (a->low_k & 31))) return -11;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return a->f32 ? cb::prep_typed<float, cb::kGated>(a, seg, st) : cb::prep_typed<__nv_bfloat16, cb::kGated>(a, seg, st);
}

// State-space duality: k is B, q is C, v is x, all convolved; a: step size logits [H].
int cb_ssd_prepare(const CbRecPrep* a, const CbSegments* seg, void* stream) {
  if (!a || !seg || seg->num <= 0 || a->tokens <= 0) return 0;
  if (!cb::recurrence_sizes_ok(a->H, a->G, a->d, a->e, a->ds, a->es, seg) || !cb::convolution_ok(a) || a->g || !a->bias) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return a->f32 ? cb::prep_typed<float, cb::kSsd>(a, seg, st) : cb::prep_typed<__nv_bfloat16, cb::kSsd>(a, seg, st);
}

// The recurrence of both.  `norm_w` null: the outputs stay in `raw` (fp32 [tokens, H e]).
int cb_linear_walk(const CbRecWalk* a, const CbSegments* seg, void* stream) {
  if (!a || !seg || seg->num <= 0 || a->tokens <= 0) return 0;
  if (!cb::recurrence_sizes_ok(a->H, a->G, a->d, a->e, a->ds, a->es, seg)) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return a->f32 ? cb::walk_typed<float, false>(a, seg, st) : cb::walk_typed<__nv_bfloat16, false>(a, seg, st);
}

// y fp32 [tokens, parts width]
int cb_gated_parts_norm(const void* y, const void* z, int ldz, const void* w, void* out, int ldo, int tokens, int parts, int width,
                        float eps, int f32, void* stream) {
  using namespace cb;
  if (tokens <= 0) return 0;
  if (parts <= 0 || width <= 0 || ldz < parts * width || ldo < parts * width || tokens > 65535) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const dim3 grid(parts, tokens);
  if (f32)
    return static_cast<int>(launch(gated_parts_norm_kernel<float>, grid, dim3(128), 0, st, static_cast<const float*>(y),
                                   static_cast<const float*>(z), ldz, static_cast<const float*>(w), static_cast<float*>(out), ldo,
                                   width, eps));
  return static_cast<int>(launch(gated_parts_norm_kernel<__nv_bfloat16>, grid, dim3(128), 0, st, static_cast<const float*>(y),
                                 static_cast<const __nv_bfloat16*>(z), ldz, static_cast<const float*>(w),
                                 static_cast<__nv_bfloat16*>(out), ldo, width, eps));
}

}  // extern "C"
