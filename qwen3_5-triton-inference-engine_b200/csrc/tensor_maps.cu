// Host side of the tensor-map TMA loads: encoders over row-major bf16 data with the 128-byte swizzle (umma.cuh).
#include "umma.cuh"

namespace b200 {

bool encode_map_bf16_sw128(CUtensorMap* map, const void* base, int rank, const uint64_t* dims,
                           const uint64_t* strides_bytes, const uint32_t* box) {
  typedef CUresult (*EncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                               const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                               CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
  static EncodeFn encode = nullptr;
  if (!encode) {
    void* fn = nullptr;
    cudaDriverEntryPointQueryResult qres;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &qres) != cudaSuccess ||
        qres != cudaDriverEntryPointSuccess || fn == nullptr) {
      cudaGetLastError();
      return false;
    }
    encode = reinterpret_cast<EncodeFn>(fn);
  }
  if (rank < 3 || rank > 5 || dims[0] != 64 || box[0] != 64 || (reinterpret_cast<uintptr_t>(base) & 15) != 0) return false;
  cuuint64_t d[5], st[4];
  cuuint32_t bx[5], es[5];
  for (int i = 0; i < rank; ++i) {
    d[i] = dims[i];
    bx[i] = box[i];
    es[i] = 1;
    if (i + 1 < rank) {
      if (strides_bytes[i] % 16 != 0) return false;
      st[i] = strides_bytes[i];
    }
  }
  return encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, static_cast<cuuint32_t>(rank), const_cast<void*>(base), d, st, bx,
                es, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
                CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

bool encode_tile_map(CUtensorMap* map, const void* base, uint64_t rows, uint64_t cols, uint64_t row_stride_bytes,
                     uint32_t box_rows, uint32_t box_blocks) {
  if (cols % 64 != 0) return false;
  const uint64_t dims[3] = {64, rows, cols / 64};
  const uint64_t strides[2] = {row_stride_bytes, 128};
  const uint32_t box[3] = {64, box_rows, box_blocks};
  return encode_map_bf16_sw128(map, base, 3, dims, strides, box);
}

bool encode_head_map(CUtensorMap* map, const void* base, int64_t rows, int64_t row_stride, int blocks, int64_t head_stride, int heads,
                     int box_rows) {
  const uint64_t dims[4] = {64, static_cast<uint64_t>(rows), static_cast<uint64_t>(blocks), static_cast<uint64_t>(heads)};
  const uint64_t strides[3] = {static_cast<uint64_t>(row_stride) * 2, 128, static_cast<uint64_t>(head_stride) * 2};
  const uint32_t box[4] = {64, static_cast<uint32_t>(box_rows), static_cast<uint32_t>(blocks), 1};
  return encode_map_bf16_sw128(map, base, 4, dims, strides, box);
}

}  // namespace b200
