// A step's token rows grouped by request, and small helpers shared by the kernels of the layered decoders
// (delta_rule.cu, latent_attn.cu, layered.cu): activations are bf16 or fp32 (template parameter T), everything the
// kernels compute is fp32.
#pragma once
#include "ptx.cuh"

namespace cb {

struct Segments {
  const int* row0;      // [num] first row of the segment in the step's token order
  const int* count;     // [num] rows of the segment (0 = padding)
  const int* slot;      // [num] request slot: state row and page-table row
  const int* pos0;      // [num] absolute position of the first row (0 = fresh state)
  int num;
  int single;           // every segment has at most one row, row s belongs to segment s (decode)
};

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

__device__ __forceinline__ float gelu_tanh(float x) {
  return 0.5f * x * (1.f + tanhf(0.7978845608028654f * fmaf(0.044715f * x * x, x, x)));
}

// Tile `tile` of the step when every segment is cut into tiles of `rows` rows: its segment and first row inside the
// segment.  Called by whole warps; false when the step has fewer tiles.  The grid of a kernel that uses it holds at
// most (T + num (rows - 1)) / rows tiles.
__device__ __forceinline__ bool find_tile(const Segments& sg, int rows, int tile, int& seg, int& off) {
  if (sg.single) {
    seg = tile;
    off = 0;
    return tile < sg.num && sg.count[tile] > 0;
  }
  const int lane = threadIdx.x & 31;
  int base = 0;
  for (int s0 = 0; s0 < sg.num; s0 += 32) {
    const int s = s0 + lane;
    const int nb = s < sg.num ? (sg.count[s] + rows - 1) / rows : 0;
    int inc = nb;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, inc, o);
      if (lane >= o) inc += v;
    }
    const unsigned hit = __ballot_sync(0xffffffffu, base + inc > tile);
    if (hit) {
      const int l = __ffs(hit) - 1;
      seg = s0 + l;
      off = (tile - (base + __shfl_sync(0xffffffffu, inc - nb, l))) * rows;
      return true;
    }
    base += __shfl_sync(0xffffffffu, inc, 31);
  }
  return false;
}

static inline int max_tiles(int tokens, int segs, int rows) {
  const long long n = (static_cast<long long>(tokens) + static_cast<long long>(segs) * (rows - 1)) / rows;
  return static_cast<int>(n < tokens ? n : tokens);
}

}  // namespace cb

extern "C" {
struct CbSegments {
  const void* row0;
  const void* count;
  const void* slot;
  const void* pos0;
  int num;
};
}

namespace cb {
// `tokens`: rows of the step; as many rows as segments means one row each
static inline Segments make_segments(const CbSegments* s, int tokens) {
  return Segments{static_cast<const int*>(s->row0), static_cast<const int*>(s->count), static_cast<const int*>(s->slot),
                  static_cast<const int*>(s->pos0), s->num, tokens == s->num ? 1 : 0};
}
}  // namespace cb
