// What the kernels of the recurrent layers that go chunk by chunk share: arguments, layout of a chunk, tensor-core helpers (gla.cu, delta.cu).
#pragma once
#include <cuda_bf16.h>

#include "gla.cuh"
#include "ptx.cuh"

constexpr int kC = 32;        // tokens of a chunk
constexpr int kScanWarps = 4;  // 16 value columns each
constexpr int kScanCols = kScanWarps * 16;

struct Gla {
  KvDev d;
  float* state;  // the layer's [slot][heads][dk][dv]
  int rec_elems;
  int heads, dk, dv, rank, dkp;
  int dva, dvs;  // columns of the state in use, and from row to row (matrix memory: one more than dv, padded)
  MatSrc src;
  const float *a2, *a2_bias, *norm;
  float q_scale, inv_tau, eps;
  void* out;
  int out_stride;
  const int *cu, *row_seq, *pos;
  int n_req, total_rows;
  bool chunked;  // longer portions are left to the chunk kernels
  unsigned char *chunks, *values;
  float* o;
  const int4* plan;
  const int* first_chunk;
  size_t chunk_bytes, v_bytes;
  int n_slices, stages;
  int cols, groups;  // step kernel: threads = columns of VEC values x groups of key channels
  const float4* gates;
  int col0;
  int col_g;  // column of src where the output gate starts
  float den_eps, out_scale;
  __device__ int col_k() const { return col0 + heads * dk; }
  __device__ int col_v() const { return col0 + 2 * heads * dk; }
  __device__ int col_a() const { return 2 * heads * dk + 2 * heads * dv; }
};

// ---- chunks: layout of what gla_chunk_kernel hands to gla_scan_kernel ----------------------------------------------
// Rows are padded by 16 bytes so that the 8 rows of an ldmatrix lie in different banks; a chunk and a slice of its values are
// contiguous, one bulk copy each.
__host__ __device__ constexpr int qk_row(int dkp) { return dkp * 2 + 16; }
constexpr int kARow = kC * 2 + 16;
constexpr int kVRow = kScanCols * 2 + 16;
__host__ __device__ constexpr size_t off_part(int dkp, int i) { return (size_t)i * kC * qk_row(dkp); }  // 0 q, 1 q rest, 2 k, 3 k rest
__host__ __device__ constexpr size_t off_a(int dkp, int i) { return off_part(dkp, 4) + (size_t)i * kC * kARow; }
__host__ __device__ constexpr size_t off_decay(int dkp) { return off_a(dkp, 2); }
__host__ __device__ constexpr size_t chunk_size(int dkp) { return (off_decay(dkp) + sizeof(float) * dkp + 127) / 128 * 128; }
constexpr size_t kVSlice = kC * kVRow;
// Chunks of the delta rule hold two more parts behind that, the rows of W (value and remainder), and their values are f32, [column][token].
__host__ __device__ constexpr size_t off_w(int dkp, int i) { return chunk_size(dkp) + (size_t)i * kC * qk_row(dkp); }
__host__ __device__ constexpr size_t delta_chunk_size(int dkp) { return (off_w(dkp, 2) + 127) / 128 * 128; }
constexpr int kUStride = kC + 8;
constexpr size_t kUSlice = sizeof(float) * kScanCols * kUStride;

__device__ __forceinline__ void split_bf16(float p0, float p1, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(p0, p1);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(p0 - f.x, p1 - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_trans(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}

// The walk over a step's chunks (delta: by the delta rule), and norm and gate of the rows it leaves in a.o.
b200_status b200_gla_scan(Gla& a, int n_req, bool delta, cudaStream_t s);
b200_status b200_gla_out(const Gla& a, int chunks, bool wide, cudaStream_t s);
inline int pad_channels(int dk) { return (dk + 31) / 32 * 32; }
inline int slices_of(int dv) { return (dv + kScanCols - 1) / kScanCols; }
