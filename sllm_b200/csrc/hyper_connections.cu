// A residual stream of several copies that every sublayer reads as a weighted sum and mixes anew, and the embedding that starts it.
//
//   embed_streams   every copy of a token's stream = its embedding row times a scale, plus (where there is a table of them) the row
//                   named by the pair (token before, token): (before * mul_prev + token * mul_cur) mod buckets; the last row at a
//                   sequence's start.  The token before a portion's first one comes from the request's state row, which the same
//                   CTA then sets to the portion's last token.  A CTA per token.
//   streams_step    the border between two sublayers, a CTA per token:
//                     x_r <- sum_s mix[s, r] x_s + share[r] term       (the term may be a stack of k-split partial sums; absent: no change)
//                     h = u / rms(u) * gain,  u = sum_s into[s] x_s    (absent at the end of a model whose streams are kept)
//                   Every stream is read once and written once; the sum stays in shared memory until its norm is known.  With `rows`
//                   only those rows are computed and no stream is written (the model's last norm).
//
// All arithmetic is float32.
#include "common.cuh"

namespace sllm {

constexpr int HC_THREADS = 256;
constexpr int HC_MAX_STREAMS = 16;

__device__ __forceinline__ float4 load4_of(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4_of(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(a.x, a.y, b.x, b.y);
}

template <typename T>
__global__ void __launch_bounds__(HC_THREADS)
embed_streams_kernel(const T* __restrict__ table, const int* __restrict__ ids, float* __restrict__ out, int H, int V, float scale, int copies,
                     const T* __restrict__ pair_table, unsigned long long buckets, unsigned long long mul_prev, unsigned long long mul_cur,
                     const int* __restrict__ positions, const int* __restrict__ seq_of_token, const int* __restrict__ q_start,
                     const int* __restrict__ state_slots, float* __restrict__ before, int vec) {
  __shared__ int prev_s;
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  auto clamp_id = [&](int id) { return id < 0 ? 0 : (id >= V ? V - 1 : id); };
  const int id = clamp_id(ids[t]);
  const T* pair = nullptr;
  if (pair_table != nullptr) {
    const int seq = seq_of_token[t], first = q_start[seq];
    if (t == first) {                             // this CTA alone reads and writes the request's row
      if (threadIdx.x == 0) {
        float* row = before + state_slots[seq];
        prev_s = clamp_id((int)*row);
        *row = (float)ids[q_start[seq + 1] - 1];
      }
      __syncthreads();
    }
    const int prev = t == first ? prev_s : clamp_id(ids[t - 1]);
    const unsigned long long row = positions[t] == 0 ? buckets : ((unsigned long long)prev * mul_prev + (unsigned long long)id * mul_cur) % buckets;
    pair = pair_table + row * H;
  }
  const T* src = table + (size_t)id * H;
  float* dst = out + (size_t)t * copies * H;
  if (vec) {                                      // rows in whole pieces of four channels
    for (int i = threadIdx.x * 4; i < H; i += HC_THREADS * 4) {
      float4 v = load4_of(src + i);
      v.x *= scale; v.y *= scale; v.z *= scale; v.w *= scale;
      if (pair != nullptr) {
        const float4 q = load4_of(pair + i);
        v.x += q.x; v.y += q.y; v.z += q.z; v.w += q.w;
      }
      for (int c = 0; c < copies; ++c) *reinterpret_cast<float4*>(dst + (size_t)c * H + i) = v;
    }
    return;
  }
  for (int i = threadIdx.x; i < H; i += HC_THREADS) {
    float v = to_f32(src[i]) * scale;
    if (pair != nullptr) v += to_f32(pair[i]);
    for (int c = 0; c < copies; ++c) dst[(size_t)c * H + i] = v;
  }
}

template <int V> struct HcVec;
template <> struct HcVec<1> {
  float v[1];
  __device__ __forceinline__ static HcVec load(const float* p) { HcVec r; r.v[0] = *p; return r; }
  __device__ __forceinline__ void store(float* p) const { *p = v[0]; }
};
template <> struct HcVec<4> {
  float v[4];
  __device__ __forceinline__ static HcVec load(const float* p) {
    const float4 q = *reinterpret_cast<const float4*>(p);
    HcVec r; r.v[0] = q.x; r.v[1] = q.y; r.v[2] = q.z; r.v[3] = q.w;
    return r;
  }
  __device__ __forceinline__ void store(float* p) const { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
};
__device__ __forceinline__ void hc_out(float* p, const float (&v)[1]) { *p = v[0]; }
__device__ __forceinline__ void hc_out(__nv_bfloat16* p, const float (&v)[1]) { *p = __float2bfloat16_rn(v[0]); }
__device__ __forceinline__ void hc_out(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void hc_out(__nv_bfloat16* p, const float (&v)[4]) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&a), *reinterpret_cast<const unsigned*>(&b));
}

// NS > 0: that many streams, their channels and weights in registers; 0: `ns` streams (up to HC_MAX_STREAMS), weights in shared memory.
// VEC channels a thread at a time.
template <int NS, int VEC, typename TO>
__global__ void __launch_bounds__(HC_THREADS, NS > 0 && NS <= 4 ? 3 : 1)
streams_step_kernel(float* __restrict__ streams, const float* __restrict__ term, int parts, size_t part_stride, const float* __restrict__ mix,
                    const float* __restrict__ share, const float* __restrict__ into, const float* __restrict__ gain, float eps,
                    const int* __restrict__ rows, TO* __restrict__ h, int T, int ns, int W) {
  constexpr int CAP = NS > 0 ? NS : HC_MAX_STREAMS;
  extern __shared__ __align__(16) float hc_u[];              // [W] the weighted sum
  __shared__ float red[33];
  __shared__ float mix_s[CAP * CAP], share_s[CAP], into_s[CAP];
  const int S = NS > 0 ? NS : ns, tid = threadIdx.x;
  // (the weights are no kernel's output: read before the wait)
  if (term != nullptr) {
    for (int i = tid; i < S * S; i += HC_THREADS) mix_s[i] = mix[i];
    if (tid < S) share_s[tid] = share[tid];
  }
  if (gain != nullptr && tid < S) into_s[tid] = into[tid];
  __syncthreads();
  pdl_launch_dependents();
  pdl_wait();
  size_t t = blockIdx.x;
  if (rows != nullptr) {
    const int r = rows[blockIdx.x];
    t = r < 0 ? 0 : (r >= T ? T - 1 : r);
  }
  float* x = streams + t * S * W;
  const float* y = term != nullptr ? term + t * W : nullptr;
  const bool keep = rows == nullptr && term != nullptr;
  float ss = 0.f;
  for (int i = tid * VEC; i < W; i += HC_THREADS * VEC) {
    HcVec<VEC> old[CAP], v;
#pragma unroll
    for (int s = 0; s < CAP; ++s)
      if (s < S) old[s] = HcVec<VEC>::load(x + (size_t)s * W + i);
    if (y != nullptr) {
      v = HcVec<VEC>::load(y + i);
      for (int p = 1; p < parts; ++p) {
        const HcVec<VEC> w = HcVec<VEC>::load(y + p * part_stride + i);
#pragma unroll
        for (int c = 0; c < VEC; ++c) v.v[c] += w.v[c];
      }
    }
    HcVec<VEC> u;
#pragma unroll
    for (int c = 0; c < VEC; ++c) u.v[c] = 0.f;
#pragma unroll
    for (int r = 0; r < CAP; ++r) {
      if (r >= S) break;
      HcVec<VEC> n;
      if (y != nullptr) {
#pragma unroll
        for (int c = 0; c < VEC; ++c) {
          float a = share_s[r] * v.v[c];
#pragma unroll
          for (int s = 0; s < CAP; ++s)
            if (s < S) a = fmaf(mix_s[s * S + r], old[s].v[c], a);
          n.v[c] = a;
        }
        if (keep) n.store(x + (size_t)r * W + i);
      } else {
        n = old[r];
      }
      if (gain != nullptr) {
#pragma unroll
        for (int c = 0; c < VEC; ++c) u.v[c] = fmaf(into_s[r], n.v[c], u.v[c]);
      }
    }
    if (gain != nullptr) {
      u.store(hc_u + i);
#pragma unroll
      for (int c = 0; c < VEC; ++c) ss = fmaf(u.v[c], u.v[c], ss);
    }
  }
  if (gain == nullptr) return;
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)W + eps);
  for (int i = tid * VEC; i < W; i += HC_THREADS * VEC) {    // (each thread reads the sums it wrote itself)
    const HcVec<VEC> u = HcVec<VEC>::load(hc_u + i), g = HcVec<VEC>::load(gain + i);
    float o[VEC];
#pragma unroll
    for (int c = 0; c < VEC; ++c) o[c] = u.v[c] * inv * g.v[c];
    hc_out(h + (size_t)blockIdx.x * W + i, o);
  }
}

template <int NS, int VEC, typename TO>
static int launch_streams_step(float* streams, const float* term, int parts, size_t part_stride, const float* mix, const float* share, const float* into,
                               const float* gain, float eps, const int* rows, TO* h, int R, int T, int ns, int W, cudaStream_t stream) {
  const size_t smem = gain != nullptr ? (size_t)W * sizeof(float) : 0;
  static size_t allowed = 48 * 1024;              // (per instantiation)
  if (smem > allowed) {
    if (cudaFuncSetAttribute(streams_step_kernel<NS, VEC, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
      cudaGetLastError();
      set_error("streams_step: rows so wide do not fit the shared memory");
      return SLLM_ERR_LAUNCH;
    }
    allowed = smem;
  }
  launch_kernel(streams_step_kernel<NS, VEC, TO>, (unsigned)R, HC_THREADS, smem, stream, streams, term, parts, part_stride, mix, share, into, gain, eps,
                rows, h, T, ns, W);
  return launch_status("streams_step");
}

template <int VEC, typename TO>
static int dispatch_streams_step(float* streams, const float* term, int parts, size_t part_stride, const float* mix, const float* share, const float* into,
                                 const float* gain, float eps, const int* rows, TO* h, int R, int T, int ns, int W, cudaStream_t stream) {
#define HC_GO(NS_) return launch_streams_step<NS_, VEC, TO>(streams, term, parts, part_stride, mix, share, into, gain, eps, rows, h, R, T, ns, W, stream)
  switch (ns) {
    case 1: HC_GO(1);
    case 2: HC_GO(2);
    case 3: HC_GO(3);
    case 4: HC_GO(4);
    case 6: HC_GO(6);
    case 8: HC_GO(8);
    default:               // (any other number, one channel at a time)
      return launch_streams_step<0, 1, TO>(streams, term, parts, part_stride, mix, share, into, gain, eps, rows, h, R, T, ns, W, stream);
  }
#undef HC_GO
}

}  // namespace sllm

using namespace sllm;

SLLM_EXPORT int sllm_embed_streams(const void* table, int dtype, const int* ids, float* out, int T, int H, int V, float scale, int copies,
                                   const void* pair_table, long long buckets, long long mul_prev, long long mul_cur, const int* positions,
                                   const int* seq_of_token, const int* q_start, const int* state_slots, float* before, cudaStream_t stream) {
  SLLM_REQUIRE(T >= 0 && H > 0 && V > 0 && copies >= 1, "embed_streams: bad sizes T=%d H=%d V=%d copies=%d", T, H, V, copies);
  SLLM_REQUIRE(pair_table == nullptr || (buckets >= 1 && mul_prev >= 0 && mul_cur >= 0 && positions && seq_of_token && q_start && state_slots && before),
               "embed_streams: pairs of tokens need their buckets, the batch's description and the tokens before");
  if (T == 0) return SLLM_OK;
  const int vec = H % 4 == 0 && (((uintptr_t)table | (uintptr_t)pair_table | (uintptr_t)out) & 15) == 0;
#define ES(T_)                                                                                                                      \
  launch_kernel(embed_streams_kernel<T_>, (unsigned)T, HC_THREADS, 0, stream, (const T_*)table, ids, out, H, V, scale, copies,       \
                (const T_*)pair_table, (unsigned long long)buckets, (unsigned long long)mul_prev, (unsigned long long)mul_cur, positions, \
                seq_of_token, q_start, state_slots, before, vec)
  if (dtype == SLLM_F32) ES(float);
  else if (dtype == SLLM_BF16) ES(__nv_bfloat16);
  else SLLM_REQUIRE(false, "embed_streams: unknown dtype %d", dtype);
#undef ES
  return launch_status("embed_streams");
}

// streams [T, ns, W] float32.  term null: the streams stay as they are; gain null: no sum, no norm (then rows must be null); rows
// [R] (else R == T): only these rows, no stream written; h [R, W] in h_dtype.
SLLM_EXPORT int sllm_streams_step(float* streams, const float* term, int parts, size_t part_stride, const float* mix, const float* share, const float* into,
                                  const float* gain, float eps, const int* rows, void* h, int h_dtype, int R, int T, int ns, int W, cudaStream_t stream) {
  SLLM_REQUIRE(T >= 0 && R >= 0 && W > 0 && (rows != nullptr || R == T), "streams_step: bad sizes R=%d T=%d W=%d", R, T, W);
  SLLM_REQUIRE(ns >= 1 && ns <= HC_MAX_STREAMS, "streams_step: %d streams are outside 1..%d", ns, HC_MAX_STREAMS);
  SLLM_REQUIRE(term == nullptr || (mix && share && parts >= 1), "streams_step: a term needs the streams' mix and its shares");
  SLLM_REQUIRE((gain == nullptr) == (h == nullptr) && (gain == nullptr || into != nullptr), "streams_step: a norm needs its gain, the sum's weights and an output");
  SLLM_REQUIRE(gain != nullptr || (term != nullptr && rows == nullptr), "streams_step: nothing to do");
  SLLM_REQUIRE((long)W * 4 <= 200 * 1024, "streams_step: rows of %d channels do not fit the shared memory", W);
  if (T == 0 || R == 0) return SLLM_OK;
  const bool vec = W % 4 == 0 && part_stride % 4 == 0 && (((uintptr_t)streams | (uintptr_t)term | (uintptr_t)gain | (uintptr_t)h) & 15) == 0;
#define SS(TO_)                                                                                                                                   \
  return vec ? dispatch_streams_step<4, TO_>(streams, term, parts, part_stride, mix, share, into, gain, eps, rows, (TO_*)h, R, T, ns, W, stream)   \
             : dispatch_streams_step<1, TO_>(streams, term, parts, part_stride, mix, share, into, gain, eps, rows, (TO_*)h, R, T, ns, W, stream)
  if (h == nullptr || h_dtype == SLLM_F32) SS(float);
  if (h_dtype == SLLM_BF16) SS(__nv_bfloat16);
#undef SS
  SLLM_REQUIRE(false, "streams_step: unknown dtype %d", h_dtype);
}
