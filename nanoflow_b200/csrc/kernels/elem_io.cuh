// Loads and stores of activations kept either as bf16 or as fp32 (NFK_BF16 / NFK_F32): kernels that exist in
// both storage types are templates over the element type and compute in fp32.
#pragma once
#include "common.cuh"
#include "kernels.h"

namespace nf {

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// Four consecutive elements (16-byte aligned fp32, 8-byte aligned bf16).
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}

// Latent pool pages: whether they are stored in 8 x 64 tiles, and the element offset of (row, column) of a page.
__host__ __device__ __forceinline__ bool latent_tiled(int dtype, long long ld, int page_size) {
  return dtype == NFK_BF16 && ld % 64 == 0 && page_size % 8 == 0;
}
__device__ __forceinline__ long long latent_offset(int page, int row, int col, int page_size, long long ld, bool tiled) {
  if (!tiled) return (static_cast<long long>(page) * page_size + row) * ld + col;
  return static_cast<long long>(page) * page_size * ld + (row >> 3) * 8 * ld + (col >> 6) * 512 + (row & 7) * 64 + (col & 63);
}

// Index of the page that holds position `pos` of request `req` in kv_indices, or -1 (reported): a request's
// page list starts at page slot kv_first[req] of its sequence (earlier pages have been given back).
__device__ __forceinline__ int page_of(int pos, int req, int page_size, const int* kv_indptr, const int* kv_indices,
                                       const int* kv_first, int num_pages, unsigned int* status) {
  const int slot = pos / page_size - (kv_first != nullptr ? kv_first[req] : 0);
  const int p0 = kv_indptr[req];
  int page = -1;
  if (slot >= 0 && p0 + slot < kv_indptr[req + 1]) page = kv_indices[p0 + slot];
  if (page < 0 || page >= num_pages) {
    report_status(status, NF_ST_BAD_INDEX);
    return -1;
  }
  return page;
}

}  // namespace nf
