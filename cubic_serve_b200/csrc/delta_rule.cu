// Gated delta rule layers of any head size, with one decay per head or one per key channel, and the short causal
// convolution in front of them (the fixed 128 x 128, four-tap form of the hybrid family is gdn.cu).
#include "recurrence.cuh"

extern "C" {

// x: q [G d] | k [G d] | v [H e] before the convolution; a: decay logits [H] or [H d] (then `g` is their scratch).
int cb_delta_prepare(const CbRecPrep* a, const CbSegments* seg, void* stream) {
  if (!a || !seg || seg->num <= 0 || a->tokens <= 0) return 0;
  if (!cb::recurrence_sizes_ok(a->H, a->G, a->d, a->e, a->ds, a->es, seg) || !cb::convolution_ok(a)) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return a->f32 ? cb::prep_typed<float, cb::kDelta>(a, seg, st) : cb::prep_typed<__nv_bfloat16, cb::kDelta>(a, seg, st);
}

// `decode`: every segment has at most one row.  `raw`: fp32 scratch [tokens, H e].
int cb_delta_walk(const CbRecWalk* a, const CbSegments* seg, void* stream) {
  if (!a || !seg || seg->num <= 0 || a->tokens <= 0) return 0;
  if (!cb::recurrence_sizes_ok(a->H, a->G, a->d, a->e, a->ds, a->es, seg) || !a->norm_w) return -10;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return a->f32 ? cb::walk_typed<float, true>(a, seg, st) : cb::walk_typed<__nv_bfloat16, true>(a, seg, st);
}

}  // extern "C"
