// Layout of a page of latents, shared by everything that reads or writes one.
//
// Rows (tokens) in groups of 8, columns in slices of 64: a page is [page_size / 8][pitch / 64][8 rows][64 columns], and inside
// a row of a slice the 8-column chunk c lies at place c ^ (row & 7).  For bf16 that is the 128-byte-swizzled image the tensor
// cores read from shared memory, with one and the same distance between any two neighbouring row groups of consecutive
// pages -- so a page travels as ONE contiguous copy, and pages laid one after the other form one operand.
#pragma once
#include "common.cuh"

namespace mlora {

__host__ __device__ __forceinline__ int latent_offset(int row, int k, int pitch) {
  return (row >> 3) * 8 * pitch + (k >> 6) * 512 + (row & 7) * 64 + ((((k & 63) >> 3) ^ (row & 7)) << 3) + (k & 7);
}

}  // namespace mlora
