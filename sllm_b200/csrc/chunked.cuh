// What the kernels that run a recurrence over prompt portions a chunk of 64 tokens at a time share (retention.cu, state_space.cu): copies
// into shared memory, a float32 product of rows and a block there, small pieces.  All arithmetic is float32 on the CUDA cores.
#pragma once

#include "common.cuh"

namespace sllm {

constexpr int RC = 64;                  // tokens per chunk
constexpr int RC_OUT_THREADS = 128;     // chunk_out: four warps of 16 tokens
constexpr int RC_SCAN_THREADS = 256;
constexpr int RC_SLICE = 32;            // rows of the state in shared memory at a time (two slices in flight)

__device__ __forceinline__ void rc_cp16(float* dst, const float* src, bool ok) {
  const unsigned sm = (unsigned)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(sm), "l"(src), "r"(ok ? 16 : 0));
}
__device__ __forceinline__ void rc_commit() { asm volatile("cp.async.commit_group;\n" ::); }

__device__ __forceinline__ float4 rc_load4(const float* p, bool ok) { return ok ? *reinterpret_cast<const float4*>(p) : make_float4(0.f, 0.f, 0.f, 0.f); }
// `rows` rows of `cols` floats (ld apart) into dst[i * LD + j] (DR x DC of it), zeros beyond; by cp.async where `vec`
template <int DR, int DC, int LD>
__device__ __forceinline__ void load_block(float* __restrict__ dst, const float* __restrict__ src, size_t ld, int rows, int cols, bool vec) {
  if (vec) {
#pragma unroll 4
    for (int e = threadIdx.x; e < DR * (DC / 4); e += blockDim.x) {
      const int i = e / (DC / 4), j = (e % (DC / 4)) * 4;
      const bool ok = i < rows && j < cols;
      rc_cp16(dst + i * LD + j, ok ? src + i * ld + j : src, ok);
    }
  } else {
#pragma unroll 4
    for (int e = threadIdx.x; e < DR * DC; e += blockDim.x) {
      const int i = e / DC, j = e % DC;
      dst[i * LD + j] = (i < rows && j < cols) ? src[i * ld + j] : 0.f;
    }
  }
  rc_commit();
}

// acc[r][c] += sum_k A[r][k] B[k][c] over k in [0, K), K a multiple of 4: A's rows lie along k (row stride LDA), B's along the columns;
// a lane's columns are 4 (lane % 16) + 64 g
template <int LDA, int LDB, int TN>
__device__ __forceinline__ void rows_times_block(float (&acc)[8][TN], const float* __restrict__ A, const float* __restrict__ B, int K) {
  const float* b = B + 4 * (threadIdx.x & 15);
#pragma unroll 1
  for (int k = 0; k < K; k += 4) {
    float4 bv[4][TN / 4];
#pragma unroll
    for (int q = 0; q < 4; ++q)
#pragma unroll
      for (int g = 0; g < TN / 4; ++g) bv[q][g] = *reinterpret_cast<const float4*>(b + (k + q) * LDB + 64 * g);
#pragma unroll
    for (int r = 0; r < 8; ++r) {
      const float4 a = *reinterpret_cast<const float4*>(A + r * LDA + k);
#pragma unroll
      for (int g = 0; g < TN / 4; ++g) {
        float* o = acc[r] + 4 * g;
        o[0] = fmaf(a.x, bv[0][g].x, o[0]); o[1] = fmaf(a.x, bv[0][g].y, o[1]); o[2] = fmaf(a.x, bv[0][g].z, o[2]); o[3] = fmaf(a.x, bv[0][g].w, o[3]);
        o[0] = fmaf(a.y, bv[1][g].x, o[0]); o[1] = fmaf(a.y, bv[1][g].y, o[1]); o[2] = fmaf(a.y, bv[1][g].z, o[2]); o[3] = fmaf(a.y, bv[1][g].w, o[3]);
        o[0] = fmaf(a.z, bv[2][g].x, o[0]); o[1] = fmaf(a.z, bv[2][g].y, o[1]); o[2] = fmaf(a.z, bv[2][g].z, o[2]); o[3] = fmaf(a.z, bv[2][g].w, o[3]);
        o[0] = fmaf(a.w, bv[3][g].x, o[0]); o[1] = fmaf(a.w, bv[3][g].y, o[1]); o[2] = fmaf(a.w, bv[3][g].z, o[2]); o[3] = fmaf(a.w, bv[3][g].w, o[3]);
      }
    }
  }
}

// z * sigmoid(z); the result is rounded to bfloat16 in the fast form
template <typename TO> __device__ __forceinline__ float rc_silu(float z) { return z * sigmoid_f32(z); }
template <> __device__ __forceinline__ float rc_silu<__nv_bfloat16>(float z) { return __fdividef(z, 1.0f + __expf(-z)); }

__device__ __forceinline__ void rc_store4(float* o, const float (&v)[4]) { *reinterpret_cast<float4*>(o) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void rc_store4(__nv_bfloat16* o, const float (&v)[4]) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  *reinterpret_cast<uint2*>(o) = make_uint2(*reinterpret_cast<const unsigned*>(&a), *reinterpret_cast<const unsigned*>(&b));
}

template <typename K>
static int rc_smem(K kernel, size_t bytes, size_t& allowed) {
  if (bytes > allowed) {
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) != cudaSuccess) {
      cudaGetLastError();
      set_error("chunks: a kernel's shared memory could not be raised");
      return SLLM_ERR_LAUNCH;
    }
    allowed = bytes;
  }
  return SLLM_OK;
}

}  // namespace sllm
