// Retention (linear attention with one fixed decay per head on rotated queries and keys, see delta_rule.cu) over prompt
// portions, a chunk of 64 tokens at a time instead of token by token.
//
//   S_t = d S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t
//
// With ONE decay per head a chunk's part of the recurrence is three small matrix products.  For a chunk of n tokens that
// meets the state S (t, s counted from the chunk's first token):
//
//   o_t = d^(t+1) S^T q_t + sum_(s <= t) d^(t-s) (q_t . k_s) v_s          S' = d^n S + sum_s d^(n-1-s) k_s v_s^T
//
// so everything but the passing on of S runs side by side over all chunks and heads:
//   1. chunk_state  per (chunk, head): what the chunk adds to a state, sum_s d^(n-1-s) k_s v_s^T, to scratch;
//   2. chunk_scan   per (request, head, element): from the request's state slot through its chunks in order; scratch then
//                   holds the state each chunk meets, the slot the portion's last state;
//   3. chunk_out    per (chunk, head): the two terms of o above, then what follows the recurrence in a layer: each head's o
//                   over its root mean square, times silu of the gate projection, in the compute dtype.
//
// All arithmetic is float32 on the CUDA cores (plain multiply-adds, no reduced-precision matrix mode): the state, all that
// enters the recurrence and all sums.  Operands lie in shared memory as they lie in memory, a token or state row after the other; a
// warp owns 16 rows of a product and all its columns, a lane 8 rows and every sixteenth piece of four columns.  So the scores a
// warp computes are the scores it multiplies the values with (no other warp waits for them, and what lies above the diagonal
// is skipped in steps of 16 tokens), and a row's root mean square is a sum over half a warp.  Rotation (channel i with i + rot/2)
// and the key's scale happen as the rows are loaded; the state and the values arrive by cp.async under the products before them.
#include <math.h>

#include "chunked.cuh"

namespace sllm {

struct RetentionParams {
  const float* proj;           // [T, ld]
  int ld, off_q, off_k, off_v, off_g;
  const float* decay;          // [H]
  const float* table;          // [max_pos][2][rot / 2]
  int rot, max_pos;
  float k_scale, eps;
  float* state;                // [slots, H, dk, dv]
  const int* state_slots;      // [S]
  const int* chunk_t0;         // [chunks] first token (row of proj)
  const int* chunk_pos;        // [chunks] the first token's position in its sequence
  const int* chunk_n;          // [chunks] tokens, 1 .. 64
  const int* run_seq;          // [runs] a request ...
  const int* run_first;        // [runs] ... its first chunk ...
  const int* run_count;        // [runs] ... and how many it has
  float* scratch;              // [chunks, H, dk, dv]
  int H, dk, dv;
  int vec_qk, vec_v, vec_o;    // queries, keys and the table / values / gate and output lie in whole 16-byte (output: 4-element) pieces
};

// (x c - y s) w and (y c + x s) w
__device__ __forceinline__ void rc_turn4(float* lo, float* hi, float4 x, float4 y, float4 c, float4 s, float w) {
  *reinterpret_cast<float4*>(lo) = make_float4((x.x * c.x - y.x * s.x) * w, (x.y * c.y - y.y * s.y) * w, (x.z * c.z - y.z * s.z) * w, (x.w * c.w - y.w * s.w) * w);
  *reinterpret_cast<float4*>(hi) = make_float4((y.x * c.x + x.x * s.x) * w, (y.y * c.y + x.y * s.y) * w, (y.z * c.z + x.z * s.z) * w, (y.w * c.w + x.w * s.w) * w);
}

// NX = 1 or 2 tensors of head h for the chunk's tokens (keys; queries and keys), rotated, tensor x times mul[x] and (if given)
// weight[t], into dst[x] + t * LD[x] + j; zeros beyond the chunk's tokens and the head's channels.  Eight lanes a token, the loads of
// four tokens a lane (two tensors: two tokens) in flight together.
template <int DK, int NX, int LD0, int LD1, int THREADS>
__device__ __forceinline__ void load_rotated(const RetentionParams& p, float* d0, float* d1, int off0, int off1, float mul0, float mul1,
                                             const float* __restrict__ weight, int h, int t0, int pos0, int n) {
  const int half = p.rot >> 1, dk = p.dk, l8 = threadIdx.x & 7;
  constexpr int TPP = THREADS / 8, AT = NX == 1 ? 4 : 2;                   // tokens a pass, passes whose loads are in flight
  static_assert(RC % (TPP * AT) == 0 || RC % TPP == 0, "whole passes");
  const float* base = p.proj + (size_t)t0 * p.ld + h * dk;
  if (p.vec_qk) {                       // whole 16-byte pieces everywhere
    for (int tb = threadIdx.x >> 3; tb < RC; tb += TPP * AT) {
      for (int i = 4 * l8; i < half; i += 32) {
        float4 x[AT][NX], y[AT][NX], c[AT], s[AT];
#pragma unroll
        for (int q = 0; q < AT; ++q) {
          const int t = tb + q * TPP;
          const bool ok = t < n;
          const float* r = base + (size_t)(ok ? t : 0) * p.ld + i;
          int pos = pos0 + t;
          pos = pos < 0 ? 0 : (pos >= p.max_pos ? p.max_pos - 1 : pos);
          const float* cs = p.table + (size_t)pos * p.rot + i;
          c[q] = rc_load4(cs, ok);
          s[q] = rc_load4(cs + half, ok);
#pragma unroll
          for (int e = 0; e < NX; ++e) {
            const float* src = r + (e == 0 ? off0 : off1);
            x[q][e] = rc_load4(src, ok);
            y[q][e] = rc_load4(src + half, ok);
          }
        }
#pragma unroll
        for (int q = 0; q < AT; ++q) {
          const int t = tb + q * TPP;
          if (t >= RC) break;
          const float w = weight != nullptr ? weight[t] : 1.0f;
#pragma unroll
          for (int e = 0; e < NX; ++e) {
            float* d = e == 0 ? d0 + t * LD0 + i : d1 + t * LD1 + i;
            rc_turn4(d, d + half, x[q][e], y[q][e], c[q], s[q], (e == 0 ? mul0 : mul1) * w);
          }
        }
      }
      for (int j = p.rot + 4 * l8; j < DK; j += 32) {
#pragma unroll
        for (int q = 0; q < AT; ++q) {
          const int t = tb + q * TPP;
          if (t >= RC) break;
          const float w = weight != nullptr ? weight[t] : 1.0f;
#pragma unroll
          for (int e = 0; e < NX; ++e) {
            const float4 x = rc_load4(base + (size_t)t * p.ld + (e == 0 ? off0 : off1) + j, t < n && j < dk);
            const float m = (e == 0 ? mul0 : mul1) * w;
            *reinterpret_cast<float4*>(e == 0 ? d0 + t * LD0 + j : d1 + t * LD1 + j) = make_float4(x.x * m, x.y * m, x.z * m, x.w * m);
          }
        }
      }
    }
    return;
  }
  for (int t = threadIdx.x >> 3; t < RC; t += TPP) {
    const bool ok = t < n;
    const float* r = base + (size_t)t * p.ld;
    int pos = pos0 + t;
    pos = pos < 0 ? 0 : (pos >= p.max_pos ? p.max_pos - 1 : pos);
    const float* cs = p.table + (size_t)pos * p.rot;
    const float w = weight != nullptr ? weight[t] : 1.0f;
#pragma unroll
    for (int e = 0; e < NX; ++e) {
      const float* src = r + (e == 0 ? off0 : off1);
      float* d = e == 0 ? d0 + t * LD0 : d1 + t * LD1;
      const float m = (e == 0 ? mul0 : mul1) * w;
      for (int i = l8; i < half; i += 8) {
        const float x = ok ? src[i] : 0.f, y = ok ? src[i + half] : 0.f, c = ok ? cs[i] : 0.f, sn = ok ? cs[half + i] : 0.f;
        d[i] = (x * c - y * sn) * m;
        d[i + half] = (y * c + x * sn) * m;
      }
      for (int j = p.rot + l8; j < DK; j += 8) d[j] = (ok && j < dk) ? src[j] * m : 0.f;
    }
  }
}

// grid (chunks, H), 2 DK threads: a warp owns 16 of the state's rows
template <int DK, int DV>
__global__ void __launch_bounds__(2 * DK) chunk_state_kernel(const RetentionParams p) {
  extern __shared__ __align__(16) float rc_sm[];
  float* ks = rc_sm;                   // [RC][DK]
  float* vs = ks + RC * DK;            // [RC][DV]
  float* pw = vs + RC * DV;            // [RC] d^(n-1-s)
  pdl_wait();
  const int chunk = blockIdx.x, h = blockIdx.y;
  const int t0 = p.chunk_t0[chunk], n = p.chunk_n[chunk];
  load_block<RC, DV, DV>(vs, p.proj + (size_t)t0 * p.ld + p.off_v + h * p.dv, p.ld, n, p.dv, p.vec_v != 0);
  if (threadIdx.x < RC) pw[threadIdx.x] = (int)threadIdx.x < n ? powf(p.decay[h], (float)(n - 1 - (int)threadIdx.x)) : 0.f;
  __syncthreads();
  load_rotated<DK, 1, DK, DK, 2 * DK>(p, ks, nullptr, p.off_k, 0, p.k_scale, 0.f, pw, h, t0, p.chunk_pos[chunk], n);
  asm volatile("cp.async.wait_group 0;\n" ::);
  __syncthreads();
  constexpr int TN = DV / 16;
  const int row = 16 * (threadIdx.x >> 5) + 8 * ((threadIdx.x >> 4) & 1), col = 4 * (threadIdx.x & 15);
  float acc[8][TN];
#pragma unroll
  for (int r = 0; r < 8; ++r)
#pragma unroll
    for (int c = 0; c < TN; ++c) acc[r][c] = 0.f;
#pragma unroll 2
  for (int s = 0; s < n; ++s) {
    const float4 a0 = *reinterpret_cast<const float4*>(ks + s * DK + row), a1 = *reinterpret_cast<const float4*>(ks + s * DK + row + 4);
    const float av[8] = {a0.x, a0.y, a0.z, a0.w, a1.x, a1.y, a1.z, a1.w};
#pragma unroll
    for (int g = 0; g < TN / 4; ++g) {
      const float4 b = *reinterpret_cast<const float4*>(vs + s * DV + col + 64 * g);
#pragma unroll
      for (int r = 0; r < 8; ++r) {
        acc[r][4 * g] = fmaf(av[r], b.x, acc[r][4 * g]);
        acc[r][4 * g + 1] = fmaf(av[r], b.y, acc[r][4 * g + 1]);
        acc[r][4 * g + 2] = fmaf(av[r], b.z, acc[r][4 * g + 2]);
        acc[r][4 * g + 3] = fmaf(av[r], b.w, acc[r][4 * g + 3]);
      }
    }
  }
  pdl_launch_dependents();
  float* out = p.scratch + ((size_t)chunk * p.H + h) * p.dk * p.dv;
  const bool vec = p.dv % 4 == 0;
#pragma unroll
  for (int r = 0; r < 8; ++r) {
    const int i = row + r;
    if (i >= p.dk) break;
#pragma unroll
    for (int g = 0; g < TN / 4; ++g) {
      const int j = col + 64 * g;
      if (vec && j < p.dv) {
        *reinterpret_cast<float4*>(out + i * p.dv + j) = make_float4(acc[r][4 * g], acc[r][4 * g + 1], acc[r][4 * g + 2], acc[r][4 * g + 3]);
      } else {
#pragma unroll
        for (int c = 0; c < 4; ++c)
          if (j + c < p.dv) out[i * p.dv + j + c] = acc[r][4 * g + c];
      }
    }
  }
}

// grid (ceil(dk dv / 256), H, runs): an element of a state a thread, through the request's chunks in order
__global__ void __launch_bounds__(RC_SCAN_THREADS) chunk_scan_kernel(const RetentionParams p) {
  pdl_wait();
  const int h = blockIdx.y, run = blockIdx.z, size = p.dk * p.dv;
  const int e = blockIdx.x * RC_SCAN_THREADS + threadIdx.x;
  const int first = p.run_first[run], count = p.run_count[run];
  if (e < size) {
    float* slot = p.state + ((size_t)p.state_slots[p.run_seq[run]] * p.H + h) * size + e;
    float* sc = p.scratch + ((size_t)first * p.H + h) * size + e;
    const size_t step = (size_t)p.H * size;
    const float d = p.decay[h], dfull = powf(d, (float)RC), dlast = powf(d, (float)p.chunk_n[first + count - 1]);   // (all but the last are full)
    float S = *slot;
    constexpr int AHEAD = 16;
    for (int c0 = 0; c0 < count; c0 += AHEAD) {
      float kv[AHEAD];
#pragma unroll
      for (int q = 0; q < AHEAD; ++q)
        if (c0 + q < count) kv[q] = sc[(size_t)(c0 + q) * step];
#pragma unroll
      for (int q = 0; q < AHEAD; ++q)
        if (c0 + q < count) {
          sc[(size_t)(c0 + q) * step] = S;
          S = fmaf(c0 + q + 1 < count ? dfull : dlast, S, kv[q]);
        }
    }
    *slot = S;
  }
  pdl_launch_dependents();
}

template <int DK, int DV> struct ChunkOutSmem {
  static constexpr int LQ = DK + 4, LKV = (DK > DV ? DK : DV) + 4;      // row strides: a multiple of 4 that walks the banks
  static constexpr int Q = RC * LQ;                                      // queries; then, row by row, the warps' scores
  static constexpr int KV = RC * LKV;                                    // keys, then values
  static constexpr int S = 2 * RC_SLICE * DV;                            // two slices of the state
  static constexpr int BYTES = (Q + KV + S + RC + 4) * 4;
};

// grid (chunks, H).  out[t, h*dv + j] (rows of out_ld) = o[t, j] / sqrt(mean_j(o[t, :]^2) + eps) * silu(gate[t, h*dv + j])
template <int DK, int DV, typename TO>
__global__ void __launch_bounds__(RC_OUT_THREADS) chunk_out_kernel(const RetentionParams p, TO* __restrict__ out, int out_ld) {
  using L = ChunkOutSmem<DK, DV>;
  extern __shared__ __align__(16) float rc_sm[];
  float* qs = rc_sm;
  float* kv = qs + L::Q;
  float* ss = kv + L::KV;
  float* pw = ss + L::S;               // [RC + 1] d^i
  constexpr int TN = DV / 16, SLICES = DK / RC_SLICE;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row = 16 * warp + 8 * (lane >> 4), l16 = lane & 15;
  pdl_wait();
  const int chunk = blockIdx.x, h = blockIdx.y;
  const int t0 = p.chunk_t0[chunk], n = p.chunk_n[chunk];
  const float* S = p.scratch + ((size_t)chunk * p.H + h) * p.dk * p.dv;
  const bool vec_s = p.dv % 4 == 0;
  auto load_slice = [&](int sl) {
    load_block<RC_SLICE, DV, DV>(ss + (sl & 1) * RC_SLICE * DV, S + (size_t)(sl * RC_SLICE < p.dk ? sl * RC_SLICE : 0) * p.dv, p.dv,
                                 p.dk - sl * RC_SLICE, p.dv, vec_s);
  };
  load_slice(0);
  load_slice(1);                       // (SLICES >= 2)
  if (threadIdx.x <= RC) pw[threadIdx.x] = powf(p.decay[h], (float)threadIdx.x);
  load_rotated<DK, 2, L::LQ, L::LKV, RC_OUT_THREADS>(p, qs, kv, p.off_q, p.off_k, 1.0f, p.k_scale, nullptr, h, t0, p.chunk_pos[chunk], n);
  __syncthreads();
  // scores of the lane's 8 tokens against keys l16 + 16 c, c up to the warp's own 16 tokens
  float sc[8][4];
#pragma unroll
  for (int r = 0; r < 8; ++r)
#pragma unroll
    for (int c = 0; c < 4; ++c) sc[r][c] = 0.f;
#pragma unroll 1
  for (int k = 0; k < DK; k += 4) {
    float4 a[8];
#pragma unroll
    for (int r = 0; r < 8; ++r) a[r] = *reinterpret_cast<const float4*>(qs + (row + r) * L::LQ + k);
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      if (c > warp) break;             // (whole warps)
      const float4 b = *reinterpret_cast<const float4*>(kv + (l16 + 16 * c) * L::LKV + k);
#pragma unroll
      for (int r = 0; r < 8; ++r)
        sc[r][c] = fmaf(a[r].w, b.w, fmaf(a[r].z, b.z, fmaf(a[r].y, b.y, fmaf(a[r].x, b.x, sc[r][c]))));
    }
  }
  __syncthreads();                     // the keys are read: their place takes the values
  load_block<RC, DV, L::LKV>(kv, p.proj + (size_t)t0 * p.ld + p.off_v + h * p.dv, p.ld, n, p.dv, p.vec_v != 0);
  float acc[8][TN];
#pragma unroll
  for (int r = 0; r < 8; ++r)
#pragma unroll
    for (int c = 0; c < TN; ++c) acc[r][c] = 0.f;
  // groups in flight by age: slice 0, slice 1, the values, slice 2, slice 3
#pragma unroll
  for (int sl = 0; sl < SLICES; ++sl) {
    if (sl == 0) asm volatile("cp.async.wait_group 2;\n" ::);
    else if (sl == 1) asm volatile("cp.async.wait_group %0;\n" ::"n"(SLICES > 2 ? 2 : 1));
    else if (sl == 2) asm volatile("cp.async.wait_group 1;\n" ::);
    else asm volatile("cp.async.wait_group 0;\n" ::);
    __syncthreads();
    rows_times_block<L::LQ, DV, TN>(acc, qs + row * L::LQ + sl * RC_SLICE, ss + (sl & 1) * RC_SLICE * DV, RC_SLICE);
    if (sl + 2 < SLICES) {
      __syncthreads();
      load_slice(sl + 2);
    }
  }
#pragma unroll
  for (int r = 0; r < 8; ++r)
#pragma unroll
    for (int c = 0; c < TN; ++c) acc[r][c] *= pw[row + r + 1];
  // the warp's scores, decayed, take the place of its queries (no other warp reads those)
  __syncwarp();
#pragma unroll
  for (int c = 0; c < 4; ++c) {
    if (c > warp) break;
    const int s = l16 + 16 * c;
#pragma unroll
    for (int r = 0; r < 8; ++r) qs[(row + r) * L::LQ + s] = s <= row + r ? sc[r][c] * pw[row + r - s] : 0.f;
  }
  // the gates of the lane's rows and columns, under the last product
  const bool vec_o = p.vec_o != 0;
  constexpr bool AHEAD_GATE = TN == 4;
  float4 zg[AHEAD_GATE ? 8 : 1];
  if (AHEAD_GATE && vec_o) {
#pragma unroll
    for (int r = 0; r < 8; ++r) zg[AHEAD_GATE ? r : 0] = rc_load4(p.proj + (size_t)(t0 + row + r) * p.ld + p.off_g + h * p.dv + 4 * l16, row + r < n && 4 * l16 < p.dv);
  }
  asm volatile("cp.async.wait_group 0;\n" ::);
  __syncthreads();                     // the values have landed
  rows_times_block<L::LQ, L::LKV, TN>(acc, qs + row * L::LQ, kv, 16 * (warp + 1));
  pdl_launch_dependents();
#pragma unroll
  for (int r = 0; r < 8; ++r) {
    float q2 = 0.f;
#pragma unroll
    for (int c = 0; c < TN; ++c) q2 = fmaf(acc[r][c], acc[r][c], q2);      // (channels beyond dv are zeros)
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) q2 += __shfl_xor_sync(0xffffffffu, q2, o);
    const int t = row + r;
    if (t >= n) continue;
    const float inv = 1.0f / sqrtf(q2 / (float)p.dv + p.eps);
    const float* g = p.proj + (size_t)(t0 + t) * p.ld + p.off_g + h * p.dv + 4 * l16;
    TO* o = out + (size_t)(t0 + t) * out_ld + h * p.dv + 4 * l16;
#pragma unroll
    for (int q = 0; q < TN / 4; ++q) {
      if (4 * l16 + 64 * q >= p.dv) continue;
      if (vec_o) {
        const float4 z = AHEAD_GATE ? zg[AHEAD_GATE ? r : 0] : *reinterpret_cast<const float4*>(g + 64 * q);
        const float v[4] = {acc[r][4 * q] * inv * rc_silu<TO>(z.x), acc[r][4 * q + 1] * inv * rc_silu<TO>(z.y),
                            acc[r][4 * q + 2] * inv * rc_silu<TO>(z.z), acc[r][4 * q + 3] * inv * rc_silu<TO>(z.w)};
        rc_store4(o + 64 * q, v);
      } else {
#pragma unroll
        for (int c = 0; c < 4; ++c)
          if (4 * l16 + 64 * q + c < p.dv) o[64 * q + c] = from_f32<TO>(acc[r][4 * q + c] * inv * rc_silu<TO>(g[64 * q + c]));
      }
    }
  }
}

template <int DK, int DV, typename TO>
static int launch_chunked(const RetentionParams& p, int chunks, int runs, TO* out, int out_ld, cudaStream_t stream) {
  static size_t allowed_state = 48 * 1024, allowed_out = 48 * 1024;      // (per instantiation)
  constexpr size_t smem_state = (size_t)(RC * DK + RC * DV + RC) * 4, smem_out = ChunkOutSmem<DK, DV>::BYTES;
  int rc = rc_smem(chunk_state_kernel<DK, DV>, smem_state, allowed_state);
  if (rc == SLLM_OK) rc = rc_smem(chunk_out_kernel<DK, DV, TO>, smem_out, allowed_out);
  if (rc != SLLM_OK) return rc;
  const dim3 grid((unsigned)chunks, (unsigned)p.H);
  launch_kernel(chunk_state_kernel<DK, DV>, grid, 2 * DK, smem_state, stream, p);
  launch_kernel(chunk_scan_kernel, dim3((unsigned)((p.dk * p.dv + RC_SCAN_THREADS - 1) / RC_SCAN_THREADS), (unsigned)p.H, (unsigned)runs), RC_SCAN_THREADS, 0, stream, p);
  launch_kernel(chunk_out_kernel<DK, DV, TO>, grid, RC_OUT_THREADS, smem_out, stream, p, out, out_ld);
  return launch_status("retention_chunked");
}

}  // namespace sllm

using namespace sllm;

SLLM_EXPORT int sllm_retention_chunked_supports(int dk, int dv) { return dk >= 1 && dk <= 128 && dv >= 1 && dv <= 128; }

// q | k | v | gate columns of `proj` [T, ld]; `chunks` pieces of at most 64 tokens (chunk_t0: rows, chunk_pos: positions, chunk_n) that belong to `runs`
// requests (run_seq: rows of state_slots; run_first, run_count: their chunks, consecutive, all but a request's last 64 tokens
// long).  scratch: float32 [chunks, H, dk, dv].  Rows of other requests are neither read nor written.
SLLM_EXPORT int sllm_retention_chunked(const float* proj, int ld, int off_q, int off_k, int off_v, int off_g, const float* decay,
                                       const float* table, int rot, int max_pos, float k_scale, float eps, float* state,
                                       const int* state_slots, const int* chunk_t0, const int* chunk_pos, const int* chunk_n, int chunks,
                                       const int* run_seq, const int* run_first, const int* run_count, int runs, float* scratch,
                                       void* out, int out_dtype, int out_ld, int H, int dk, int dv, cudaStream_t stream) {
  SLLM_REQUIRE(chunks >= 0 && runs >= 0 && runs <= 65535 && H > 0 && H <= 65535, "retention_chunked: bad sizes chunks=%d runs=%d H=%d", chunks, runs, H);
  SLLM_REQUIRE(sllm_retention_chunked_supports(dk, dv), "retention_chunked: heads of %d x %d are outside 1..128", dk, dv);
  SLLM_REQUIRE(off_q >= 0 && off_k >= 0 && off_v >= 0 && off_g >= 0 && off_q + H * dk <= ld && off_k + H * dk <= ld &&
                   off_v + H * dv <= ld && off_g + H * dv <= ld, "retention_chunked: columns outside the product's %d", ld);
  SLLM_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= dk && (rot == 0 || (table && max_pos > 0)),
               "retention_chunked: %d rotated channels of %d need an even number and a table", rot, dk);
  SLLM_REQUIRE(scratch != nullptr && ((uintptr_t)scratch & 15) == 0 && ((uintptr_t)state & 15) == 0 && out_ld >= H * dv,
               "retention_chunked: scratch and state must be 16-byte aligned, the output's rows of %d hold %d", out_ld, H * dv);
  if (chunks == 0 || runs == 0) return SLLM_OK;
  RetentionParams p;
  p.proj = proj; p.ld = ld; p.off_q = off_q; p.off_k = off_k; p.off_v = off_v; p.off_g = off_g; p.decay = decay;
  p.chunk_pos = chunk_pos; p.table = table; p.rot = rot; p.max_pos = max_pos > 0 ? max_pos : 1; p.k_scale = k_scale; p.eps = eps;
  p.state = state; p.state_slots = state_slots; p.chunk_t0 = chunk_t0; p.chunk_n = chunk_n;
  p.run_seq = run_seq; p.run_first = run_first; p.run_count = run_count; p.scratch = scratch; p.H = H; p.dk = dk; p.dv = dv;
  const bool base16 = ((uintptr_t)proj & 15) == 0 && ld % 4 == 0;
  p.vec_qk = base16 && off_q % 4 == 0 && off_k % 4 == 0 && dk % 4 == 0 && rot % 8 == 0 && ((uintptr_t)table & 15) == 0;
  p.vec_v = base16 && off_v % 4 == 0 && dv % 4 == 0;
  p.vec_o = base16 && off_g % 4 == 0 && dv % 4 == 0 && out_ld % 4 == 0 && ((uintptr_t)out & 15) == 0;
#define RCGO(TO_)                                                                                                       \
  do {                                                                                                                  \
    if (dk <= 64 && dv <= 64) return launch_chunked<64, 64, TO_>(p, chunks, runs, (TO_*)out, out_ld, stream);           \
    if (dk <= 64) return launch_chunked<64, 128, TO_>(p, chunks, runs, (TO_*)out, out_ld, stream);                      \
    if (dv <= 64) return launch_chunked<128, 64, TO_>(p, chunks, runs, (TO_*)out, out_ld, stream);                      \
    return launch_chunked<128, 128, TO_>(p, chunks, runs, (TO_*)out, out_ld, stream);                                   \
  } while (0)
  if (out_dtype == SLLM_F32) RCGO(float);
  if (out_dtype == SLLM_BF16) RCGO(__nv_bfloat16);
#undef RCGO
  SLLM_REQUIRE(false, "retention_chunked: unknown dtype %d", out_dtype);
}
