// What the kernels of linear attention share, whatever their decay: rows of a projection read and written four neighbouring
// values at a time, and the output gate.
#pragma once
#include "common.cuh"

__device__ __forceinline__ float la_gate(int act, float z) {
  const float s = 1.0f / (1.0f + expf(-z));
  return act == 1 ? z * s : s;
}
// Four neighbouring values of a row from column c on; columns >= n are zero.
__device__ __forceinline__ float4 la_load4(const float* row, int c, int n, bool vec) {
  if (vec && c + 3 < n) return *reinterpret_cast<const float4*>(row + c);
  float4 r;
  r.x = c < n ? row[c] : 0.f;
  r.y = c + 1 < n ? row[c + 1] : 0.f;
  r.z = c + 2 < n ? row[c + 2] : 0.f;
  r.w = c + 3 < n ? row[c + 3] : 0.f;
  return r;
}
__device__ __forceinline__ void la_store4(float* row, int c, int n, bool vec, float4 x) {
  if (vec && c + 3 < n) { *reinterpret_cast<float4*>(row + c) = x; return; }
  if (c < n) row[c] = x.x;
  if (c + 1 < n) row[c + 1] = x.y;
  if (c + 2 < n) row[c + 2] = x.z;
  if (c + 3 < n) row[c + 3] = x.w;
}
