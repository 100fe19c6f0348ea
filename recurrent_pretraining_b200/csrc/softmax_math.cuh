// Arithmetic of the softmax warps of the attention kernels.
#pragma once
#include "common.cuh"

namespace b200 {

__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp_approx(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// three-input max and packed two-wide fp32 arithmetic (sm_100): half the issue slots of the scalar forms
__device__ __forceinline__ float fmax3(float a, float b, float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}
__device__ __forceinline__ float2 ffma2(float2 a, float2 b, float2 c) {
  float2 d;
  asm("{\n"
      "  .reg .b64 ra, rb, rc, rd;\n"
      "  mov.b64 ra, {%2, %3};\n"
      "  mov.b64 rb, {%4, %5};\n"
      "  mov.b64 rc, {%6, %7};\n"
      "  fma.rn.f32x2 rd, ra, rb, rc;\n"
      "  mov.b64 {%0, %1}, rd;\n"
      "}\n"
      : "=f"(d.x), "=f"(d.y)
      : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y), "f"(c.x), "f"(c.y));
  return d;
}
__device__ __forceinline__ float2 fmul2(float2 a, float2 b) {
  float2 d;
  asm("{\n"
      "  .reg .b64 ra, rb, rd;\n"
      "  mov.b64 ra, {%2, %3};\n"
      "  mov.b64 rb, {%4, %5};\n"
      "  mul.rn.f32x2 rd, ra, rb;\n"
      "  mov.b64 {%0, %1}, rd;\n"
      "}\n"
      : "=f"(d.x), "=f"(d.y)
      : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y));
  return d;
}
__device__ __forceinline__ float2 fadd2(float2 a, float2 b) {
  float2 d;
  asm("{\n"
      "  .reg .b64 ra, rb, rd;\n"
      "  mov.b64 ra, {%2, %3};\n"
      "  mov.b64 rb, {%4, %5};\n"
      "  add.rn.f32x2 rd, ra, rb;\n"
      "  mov.b64 {%0, %1}, rd;\n"
      "}\n"
      : "=f"(d.x), "=f"(d.y)
      : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y));
  return d;
}

}  // namespace b200
