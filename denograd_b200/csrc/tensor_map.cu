// Encoded TMA tensor maps of the tensor-core projections, kept per operand (declared in tcgen05.cuh).
#include "tcgen05.cuh"

typedef CUresult (*encode_tiled_fn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                    const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                    CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
static encode_tiled_fn g_encode = nullptr;

// `bytes` = element size: 2 for fp16 operands (128-byte swizzle, the layout the MMA descriptors name), 1 for int8
// weight tiles, which land unswizzled (64-byte rows) for the converting warps
static int make_map(CUtensorMap* m, const void* base, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_rows, const char* what, int bytes, bool bf16) {
  if (!g_encode) {
    void* fn = nullptr;
    cudaDriverEntryPointQueryResult qres;
    cudaError_t e = cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &qres);
    if (e != cudaSuccess || fn == nullptr) {
      jg_set_error("cuTensorMapEncodeTiled is not available from this driver");
      return JG_ENOTSUP;
    }
    g_encode = (encode_tiled_fn)fn;
  }
  const cuuint64_t dims[2] = {cols, rows};           // innermost first
  const cuuint64_t strides[1] = {ld * (cuuint64_t)bytes};  // bytes between rows
  const cuuint32_t box[2] = {64, box_rows};
  const cuuint32_t estr[2] = {1, 1};
  const CUtensorMapDataType type = bytes == 1 ? CU_TENSOR_MAP_DATA_TYPE_UINT8 : (bf16 ? CU_TENSOR_MAP_DATA_TYPE_BFLOAT16 : CU_TENSOR_MAP_DATA_TYPE_FLOAT16);
  CUresult r = g_encode(m, type, 2, const_cast<void*>(base), dims,
                        strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                        bytes == 2 ? CU_TENSOR_MAP_SWIZZLE_128B : CU_TENSOR_MAP_SWIZZLE_NONE, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                        CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) {
    jg_set_error("tensor map for %s (%llu x %llu) rejected: CUresult %d", what, (unsigned long long)rows, (unsigned long long)cols, (int)r);
    return JG_EINVAL;
  }
  return JG_OK;
}

// Encoded maps are kept per (base, rows, cols, box rows): a model's weights and workspaces keep their addresses, so a
// step after the first finds all of its maps here instead of encoding three per launch.
struct MapKey { const void* base; uint64_t rows, cols, ld; uint32_t box_rows; int bytes; bool bf16; };
struct MapSlot { MapKey k; CUtensorMap m; bool used; };
constexpr int MAP_SLOTS = 8192;
static MapSlot g_maps[MAP_SLOTS];

int jg_tensor_map(CUtensorMap* out, const void* base, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_rows, const char* what,
                  int bytes, bool bf16) {
  uint64_t h = (uint64_t)(uintptr_t)base * 0x9E3779B97F4A7C15ull ^ (rows * 0xBF58476D1CE4E5B9ull) ^ (cols << 20) ^ (ld << 4) ^ box_rows ^ ((uint64_t)bytes << 40) ^ ((uint64_t)bf16 << 43);
  h ^= h >> 29;
  for (int probe = 0; probe < 8; probe++) {
    MapSlot& s = g_maps[(h + probe) % MAP_SLOTS];
    if (s.used && s.k.base == base && s.k.rows == rows && s.k.cols == cols && s.k.ld == ld && s.k.box_rows == box_rows && s.k.bytes == bytes &&
        s.k.bf16 == bf16) { *out = s.m; return JG_OK; }
    if (!s.used) {
      int rc = make_map(&s.m, base, rows, cols, ld, box_rows, what, bytes, bf16);
      if (rc) return rc;
      s.k = MapKey{base, rows, cols, ld, box_rows, bytes, bf16};
      s.used = true;
      *out = s.m;
      return JG_OK;
    }
  }
  MapSlot& s = g_maps[h % MAP_SLOTS];  // neighbourhood full: replace
  int rc = make_map(&s.m, base, rows, cols, ld, box_rows, what, bytes, bf16);
  if (rc) { s.used = false; return rc; }
  s.k = MapKey{base, rows, cols, ld, box_rows, bytes, bf16};
  s.used = true;
  *out = s.m;
  return JG_OK;
}
