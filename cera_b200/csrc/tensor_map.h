// TMA tensor maps of row-major bf16 matrices.
#pragma once

#include <cuda.h>

#include "common.cuh"

namespace cera {

// [rows][ld] bf16 (ld a multiple of 8), boxes of box_cols x box_rows elements laid down with the 128-byte swizzle
// (box_cols = 64); elements outside read as zero.
int32_t tensor_map_bf16(CUtensorMap *map, const void *base, uint64_t rows, uint64_t ld, uint32_t box_cols, uint32_t box_rows);

}  // namespace cera
