// What the chunked matrix memories share: chunk geometry, prefix sums over a chunk's tokens, head / remainder packing, tensor maps.
#pragma once
#include <cuda.h>

#include "rowops.cuh"
#include "softmax_math.cuh"

namespace b200 {

constexpr int MC_C = 128;                     // tokens per chunk
constexpr int MC_PANEL = MC_C * 128;          // 128 rows x 64 bf16
constexpr float LOG2E = 1.4426950408889634f;

// inclusive prefix over 128 threads in token order, in both halves of the CTA alike
template <bool MAX>
__device__ __forceinline__ float chunk_prefix(float v, float* red_all) {
  const int lane = threadIdx.x & 31, warp = (threadIdx.x >> 5) & 3;
  float* red = red_all + 4 * (threadIdx.x >> 7);
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float w = __shfl_up_sync(0xffffffffu, v, o);
    if (lane >= o) v = MAX ? fmaxf(v, w) : v + w;
  }
  named_barrier_sync(1, 256);                  // the eight warps that hold tokens
  if (lane == 31) red[warp] = v;
  named_barrier_sync(1, 256);
  for (int w = 0; w < warp; ++w) v = MAX ? fmaxf(v, red[w]) : v + red[w];
  return v;
}

__device__ __forceinline__ void split_pack(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(a, b);
  const float2 h = unpack_bf16x2(hi);
  lo = pack_bf16x2(a - h.x, b - h.y);
}

typedef CUresult (*EncodeTiledFnM)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                   const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                   CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// bf16 [planes, rows, cols] with the given pitches (elements); box: `box_rows` rows x 64 columns of one plane, 128-byte swizzle
static int make_tmap_planes(CUtensorMap* out, const void* base, uint64_t cols, uint64_t rows, uint64_t planes, uint64_t ld, uint64_t plane,
                            uint32_t box_rows) {
  static EncodeTiledFnM enc = nullptr;
  if (!enc) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess)
      return -1;
    enc = reinterpret_cast<EncodeTiledFnM>(ptr);
  }
  if ((reinterpret_cast<uintptr_t>(base) & 15) || (ld & 7) || (plane & 7)) return -2;
  cuuint64_t dims[3] = {cols, rows, planes};
  cuuint64_t strides[2] = {ld * 2, plane * 2};
  cuuint32_t box[3] = {64, box_rows, 1};
  cuuint32_t estr[3] = {1, 1, 1};
  return enc(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
             CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS ? 0 : -3;
}

}  // namespace b200
