// The state-space recurrence with one decay per token and head (see delta_rule.cu, which walks it token by token) over prompt portions, a
// chunk of 64 tokens at a time, and the gated norm behind it.
//
//   S_t = a_t S_(t-1) + dt_t B_t x_t^T,   y_t = S_t^T C_t + D x_t,      a_t = exp(-exp(A_log) dt_t),   dt_t = softplus(z_t + dt_bias)
//
// With L_t the sum of log a over the chunk's tokens up to t, a chunk of n tokens that meets the state S gives (t, s from its first token)
//
//   y_t = exp(L_t) S^T C_t + sum_(s <= t) exp(L_t - L_s) dt_s (C_t . B_s) x_s + D x_t
//   S'  = exp(L_(n-1)) S + sum_s exp(L_(n-1) - L_s) dt_s B_s x_s^T
//
// and every exponent is at most zero.  Three kernels, everything but the passing on of S side by side over all chunks and heads:
//   1. ssd_state  per (chunk, head): what the chunk adds to a state, to scratch, and its decay exp(L_(n-1)); per (chunk, group), as CTAs of
//                 the same launch: the products C_t . B_s, which all heads of a group share, to scratch;
//   2. ssd_scan   per (request, head, element): from the request's state slot through its chunks in order; scratch then holds the
//                 state each chunk meets, the slot the portion's last state;
//   3. ssd_out    per (chunk, head): y.
// Where every request of a step brings one token, ssd_token is all there is: a CTA per (request, head) streams the state through its registers.
// Heads share B and C in groups.  All arithmetic is float32 multiply-adds on the CUDA cores; a warp owns 16 rows of a product and all
// its columns (retention.cu says how the operands lie).
//
// gated_group_norm: v = y * silu(z), its channels in equal parts each over its own root mean square, times a gain; a CTA per (token, part).
#include <math.h>

#include "chunked.cuh"

namespace sllm {

struct SsdParams {
  const float* xbc;            // [T, ldx]: x at h * dv, B at off_b + g * dk, C at off_c + g * dk
  const float* dtp;            // [T, ldd]: step logits at off_dt + h
  int ldx, off_b, off_c, ldd, off_dt;
  const float* dt_bias;        // [H]
  const float* a_log;          // [H]
  const float* skip;           // [H]
  float* state;                // [slots, H, dk, dv]
  const int* state_slots;      // [S]
  const int* chunk_t0;         // [chunks] first token
  const int* chunk_n;          // [chunks] tokens, 1 .. 64
  const int* run_seq;          // [runs] a request ...
  const int* run_first;        // [runs] ... its first chunk ...
  const int* run_count;        // [runs] ... and how many it has
  float* scratch;              // [chunks, H, dk, dv]
  float* scores;               // [chunks, groups, RC, RC]: C_t . B_s at [t][s] (s <= t)
  float* keeps;                // [chunks, H]
  float* out;                  // [T, H * dv]
  int H, hdiv, dk, dv;         // hdiv: heads per group
  int groups;
  int vec_bc, vec_x;           // B and C / x and the output lie in whole 16-byte pieces
};

__device__ __forceinline__ float ssd_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// step sizes dt[RC] and sums of log decays L[RC] of head h over the chunk's tokens, by the CTA's first two warps (beyond n: steps of
// zero, the sum stays); total: scratch of one float.  Ends with a barrier.
__device__ __forceinline__ void ssd_steps(const SsdParams& p, int h, int t0, int n, float* dt_s, float* L_s, float* total) {
  const int t = threadIdx.x, lane = t & 31;
  float sum = 0.f;
  if (t < RC) {
    const float dt = t < n ? ssd_softplus(p.dtp[(size_t)(t0 + t) * p.ldd + p.off_dt + h] + p.dt_bias[h]) : 0.f;
    dt_s[t] = dt;
    sum = -expf(p.a_log[h]) * dt;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += v;
    }
    if (t == 31) *total = sum;
  }
  __syncthreads();
  if (t < RC) L_s[t] = t >= 32 ? sum + *total : sum;
  __syncthreads();
}

// The products C_t . B_s of one chunk and group by a CTA of THREADS threads: a lane has 1024 / THREADS tokens t and every sixteenth s.
template <int DK, int THREADS>
__device__ __forceinline__ void ssd_scores(const SsdParams& p, float* sm, int chunk, int grp) {
  constexpr int LD = DK + 4, R = RC * 16 / THREADS;
  float* cs = sm;                      // [RC][LD]
  float* bs = sm + RC * LD;            // [RC][LD]
  const int t0 = p.chunk_t0[chunk], n = p.chunk_n[chunk];
  const float* row0 = p.xbc + (size_t)t0 * p.ldx;
  load_block<RC, DK, LD>(cs, row0 + p.off_c + grp * p.dk, p.ldx, n, p.dk, p.vec_bc != 0);
  load_block<RC, DK, LD>(bs, row0 + p.off_b + grp * p.dk, p.ldx, n, p.dk, p.vec_bc != 0);
  asm volatile("cp.async.wait_group 0;\n" ::);
  __syncthreads();
  const int row = (int)(threadIdx.x >> 4) * R, l16 = threadIdx.x & 15;
  const int last_c = (2 * R * (int)(threadIdx.x >> 5) + 2 * R - 1) / 16;      // the block of 16 tokens that holds the warp's last
  float sc[R][4];
#pragma unroll
  for (int r = 0; r < R; ++r)
#pragma unroll
    for (int c = 0; c < 4; ++c) sc[r][c] = 0.f;
#pragma unroll 2
  for (int k = 0; k < DK; k += 4) {
    float4 a[R];
#pragma unroll
    for (int r = 0; r < R; ++r) a[r] = *reinterpret_cast<const float4*>(cs + (row + r) * LD + k);
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      if (c > last_c) break;           // (whole warps)
      const float4 b = *reinterpret_cast<const float4*>(bs + (l16 + 16 * c) * LD + k);
#pragma unroll
      for (int r = 0; r < R; ++r)
        sc[r][c] = fmaf(a[r].w, b.w, fmaf(a[r].z, b.z, fmaf(a[r].y, b.y, fmaf(a[r].x, b.x, sc[r][c]))));
    }
  }
  pdl_launch_dependents();
  float* out = p.scores + ((size_t)chunk * p.groups + grp) * RC * RC;
#pragma unroll
  for (int r = 0; r < R; ++r)
#pragma unroll
    for (int c = 0; c < 4; ++c) out[(row + r) * RC + l16 + 16 * c] = sc[r][c];
}

// grid (chunks, H + groups), 2 DK threads: a warp owns 16 of the state's rows; the last `groups` rows of CTAs make the scores
template <int DK, int DV>
__global__ void __launch_bounds__(2 * DK) ssd_state_kernel(const SsdParams p) {
  extern __shared__ __align__(16) float rc_sm[];
  float* ks = rc_sm;                   // [RC][DK]
  float* vs = ks + RC * DK;            // [RC][DV]
  float* dt_s = vs + RC * DV;          // [RC]
  float* L_s = dt_s + RC;              // [RC]
  pdl_wait();
  const int chunk = blockIdx.x, h = blockIdx.y;
  if (h >= p.H) {
    ssd_scores<DK, 2 * DK>(p, rc_sm, chunk, h - p.H);
    return;
  }
  const int t0 = p.chunk_t0[chunk], n = p.chunk_n[chunk];
  const float* row0 = p.xbc + (size_t)t0 * p.ldx;
  load_block<RC, DK, DK>(ks, row0 + p.off_b + (h / p.hdiv) * p.dk, p.ldx, n, p.dk, p.vec_bc != 0);
  load_block<RC, DV, DV>(vs, row0 + h * p.dv, p.ldx, n, p.dv, p.vec_x != 0);
  ssd_steps(p, h, t0, n, dt_s, L_s, L_s + RC);
  asm volatile("cp.async.wait_group 0;\n" ::);
  __syncthreads();
  const float last = L_s[RC - 1];
  for (int e = threadIdx.x; e < RC * (DV / 4); e += 2 * DK) {        // the values take their tokens' weights
    const int s = e / (DV / 4);
    float4* v = reinterpret_cast<float4*>(vs) + e;
    const float w = expf(last - L_s[s]) * dt_s[s];
    *v = make_float4(v->x * w, v->y * w, v->z * w, v->w * w);
  }
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
  if (threadIdx.x == 0) p.keeps[(size_t)chunk * p.H + h] = expf(last);
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

// grid (ceil(dk dv / (256 VEC)), H, runs): VEC elements of a state a thread, through the request's chunks in order
template <int VEC>
__global__ void __launch_bounds__(RC_SCAN_THREADS) ssd_scan_kernel(const SsdParams p) {
  struct alignas(4 * VEC) Piece { float v[VEC]; };
  pdl_wait();
  const int h = blockIdx.y, run = blockIdx.z, size = p.dk * p.dv;
  const int e = (blockIdx.x * RC_SCAN_THREADS + threadIdx.x) * VEC;
  const int first = p.run_first[run], count = p.run_count[run];
  if (e < size) {
    Piece* slot = reinterpret_cast<Piece*>(p.state + ((size_t)p.state_slots[p.run_seq[run]] * p.H + h) * size + e);
    float* sc = p.scratch + ((size_t)first * p.H + h) * size + e;
    const float* keep = p.keeps + (size_t)first * p.H + h;
    const size_t step = (size_t)p.H * size;
    Piece S = *slot;
    constexpr int AHEAD = 8;
    for (int c0 = 0; c0 < count; c0 += AHEAD) {
      Piece kv[AHEAD];
      float d[AHEAD];
#pragma unroll
      for (int q = 0; q < AHEAD; ++q)
        if (c0 + q < count) {
          kv[q] = *reinterpret_cast<const Piece*>(sc + (size_t)(c0 + q) * step);
          d[q] = keep[(size_t)(c0 + q) * p.H];
        }
#pragma unroll
      for (int q = 0; q < AHEAD; ++q)
        if (c0 + q < count) {
          *reinterpret_cast<Piece*>(sc + (size_t)(c0 + q) * step) = S;
#pragma unroll
          for (int i = 0; i < VEC; ++i) S.v[i] = fmaf(d[q], S.v[i], kv[q].v[i]);
        }
    }
    *slot = S;
  }
  pdl_launch_dependents();
}

template <int DK, int DV> struct SsdOutSmem {
  static constexpr int LQ = DK + 4, LX = DV + 4;                         // row strides: a multiple of 4 that walks the banks
  static constexpr int Q = RC * LQ;                                      // C; then, row by row, the warps' weighted scores
  static constexpr int X = RC * LX;
  static constexpr int S = 2 * RC_SLICE * DV;                            // two slices of the state
  static constexpr int BYTES = (Q + X + S + 2 * RC + 4) * 4;
};

// grid (chunks, H)
template <int DK, int DV>
__global__ void __launch_bounds__(RC_OUT_THREADS) ssd_out_kernel(const SsdParams p) {
  using L = SsdOutSmem<DK, DV>;
  extern __shared__ __align__(16) float rc_sm[];
  float* qs = rc_sm;
  float* xs = qs + L::Q;
  float* ss = xs + L::X;
  float* dt_s = ss + L::S;             // [RC]
  float* L_s = dt_s + RC;              // [RC]
  constexpr int TN = DV / 16, SLICES = DK / RC_SLICE;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row = 16 * warp + 8 * (lane >> 4), l16 = lane & 15;
  pdl_wait();
  const int chunk = blockIdx.x, h = blockIdx.y, grp = h / p.hdiv;
  const int t0 = p.chunk_t0[chunk], n = p.chunk_n[chunk];
  const float* row0 = p.xbc + (size_t)t0 * p.ldx;
  const float* S = p.scratch + ((size_t)chunk * p.H + h) * p.dk * p.dv;
  const bool vec_s = p.dv % 4 == 0;
  auto load_slice = [&](int sl) {
    load_block<RC_SLICE, DV, DV>(ss + (sl & 1) * RC_SLICE * DV, S + (size_t)(sl * RC_SLICE < p.dk ? sl * RC_SLICE : 0) * p.dv, p.dv,
                                 p.dk - sl * RC_SLICE, p.dv, vec_s);
  };
  load_block<RC, DK, L::LQ>(qs, row0 + p.off_c + grp * p.dk, p.ldx, n, p.dk, p.vec_bc != 0);
  load_slice(0);
  load_slice(1);                       // (SLICES >= 2)
  load_block<RC, DV, L::LX>(xs, row0 + h * p.dv, p.ldx, n, p.dv, p.vec_x != 0);
  // the scores of the lane's 8 tokens against tokens l16 + 16 c, c up to the warp's own 16 tokens
  float sc[8][4];
  const float* scores = p.scores + ((size_t)chunk * p.groups + grp) * RC * RC;
#pragma unroll
  for (int c = 0; c < 4; ++c)
#pragma unroll
    for (int r = 0; r < 8; ++r) sc[r][c] = c <= warp ? scores[(row + r) * RC + l16 + 16 * c] : 0.f;
  ssd_steps(p, h, t0, n, dt_s, L_s, L_s + RC);
  float acc[8][TN];
#pragma unroll
  for (int r = 0; r < 8; ++r)
#pragma unroll
    for (int c = 0; c < TN; ++c) acc[r][c] = 0.f;
  // groups in flight by age: C, slice 0, slice 1, x, slice 2, slice 3
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
  for (int r = 0; r < 8; ++r) {
    const float e = expf(L_s[row + r]);
#pragma unroll
    for (int c = 0; c < TN; ++c) acc[r][c] *= e;
  }
  // the warp's scores, weighted, take the place of its rows of C (no other warp reads those)
  __syncwarp();
#pragma unroll
  for (int c = 0; c < 4; ++c) {
    if (c > warp) break;
    const int s = l16 + 16 * c;
#pragma unroll
    for (int r = 0; r < 8; ++r) qs[(row + r) * L::LQ + s] = s <= row + r ? sc[r][c] * (expf(L_s[row + r] - L_s[s]) * dt_s[s]) : 0.f;
  }
  asm volatile("cp.async.wait_group 0;\n" ::);
  __syncthreads();                     // x has landed
  rows_times_block<L::LQ, L::LX, TN>(acc, qs + row * L::LQ, xs, 16 * (warp + 1));
  pdl_launch_dependents();
  const float skip = p.skip[h];
#pragma unroll
  for (int r = 0; r < 8; ++r) {
    const int t = row + r;
    if (t >= n) break;
    float* o = p.out + ((size_t)(t0 + t) * p.H + h) * p.dv + 4 * l16;
    const float* x = xs + t * L::LX + 4 * l16;
#pragma unroll
    for (int q = 0; q < TN / 4; ++q) {
      if (4 * l16 + 64 * q >= p.dv) continue;
      if (p.vec_x) {
        *reinterpret_cast<float4*>(o + 64 * q) =
            make_float4(fmaf(skip, x[64 * q], acc[r][4 * q]), fmaf(skip, x[64 * q + 1], acc[r][4 * q + 1]),
                        fmaf(skip, x[64 * q + 2], acc[r][4 * q + 2]), fmaf(skip, x[64 * q + 3], acc[r][4 * q + 3]));
      } else {
#pragma unroll
        for (int c = 0; c < 4; ++c)
          if (4 * l16 + 64 * q + c < p.dv) o[64 * q + c] = fmaf(skip, x[64 * q + c], acc[r][4 * q + c]);
      }
    }
  }
}

constexpr int ST_THREADS = 256;

struct SsdTokenParams {
  const float* xbc; const float* dtp;
  int ldx, off_b, off_c, ldd, off_dt;
  const float *dt_bias, *a_log, *skip;
  float* state;                // [slots, H, N, dv]
  const int* state_slots;      // [S]
  float* out;                  // [S, H * dv]
  int H, hdiv, N, dv;
};

// One token a request (request s's is row s): grid (S, H).  A thread holds PER pieces of four columns of the state, PER rows apart by
// 256 / (dv / 4); all of them are in flight while the step size and the rows of B and C arrive.  dv / 4 divides 256.
template <int PER>
__global__ void __launch_bounds__(ST_THREADS) ssd_token_kernel(const SsdTokenParams p) {
  __shared__ __align__(16) float4 part[ST_THREADS];
  pdl_wait();
  const int s = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int quads = p.dv >> 2, cq = tid % quads, r0 = tid / quads, rows = ST_THREADS / quads;
  float4* S = reinterpret_cast<float4*>(p.state + ((size_t)p.state_slots[s] * p.H + h) * p.N * p.dv) + cq;
  float4 v[PER];
#pragma unroll
  for (int k = 0; k < PER; ++k) {
    const int r = r0 + k * rows;
    v[k] = r < p.N ? S[(size_t)r * quads] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const float* row = p.xbc + (size_t)s * p.ldx;
  const float* B = row + p.off_b + (h / p.hdiv) * p.N;
  const float* C = row + p.off_c + (h / p.hdiv) * p.N;
  const float dt = ssd_softplus(p.dtp[(size_t)s * p.ldd + p.off_dt + h] + p.dt_bias[h]), keep = expf(-expf(p.a_log[h]) * dt);
  const float* xp = row + h * p.dv + 4 * cq;
  const float4 x = make_float4(xp[0], xp[1], xp[2], xp[3]);
  float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int k = 0; k < PER; ++k) {
    const int r = r0 + k * rows;
    if (r >= p.N) break;
    const float b = B[r] * dt, c = C[r];
    v[k].x = fmaf(b, x.x, keep * v[k].x); v[k].y = fmaf(b, x.y, keep * v[k].y);
    v[k].z = fmaf(b, x.z, keep * v[k].z); v[k].w = fmaf(b, x.w, keep * v[k].w);
    S[(size_t)r * quads] = v[k];
    y.x = fmaf(c, v[k].x, y.x); y.y = fmaf(c, v[k].y, y.y); y.z = fmaf(c, v[k].z, y.z); y.w = fmaf(c, v[k].w, y.w);
  }
  pdl_launch_dependents();
  part[tid] = y;
  __syncthreads();
  for (int half = rows >> 1; half > 0; half >>= 1) {      // (rows is a power of two)
    if (r0 < half) {
      const float4 o = part[tid + half * quads];
      float4 m = part[tid];
      m.x += o.x; m.y += o.y; m.z += o.z; m.w += o.w;
      part[tid] = m;
    }
    __syncthreads();
  }
  if (r0 == 0) {
    const float4 m = part[tid];
    const float d = p.skip[h];
    float* o = p.out + ((size_t)s * p.H + h) * p.dv + 4 * cq;
    o[0] = fmaf(d, x.x, m.x); o[1] = fmaf(d, x.y, m.y); o[2] = fmaf(d, x.z, m.z); o[3] = fmaf(d, x.w, m.w);
  }
}

template <int DK, int DV>
static int launch_ssd(const SsdParams& p, int chunks, int runs, cudaStream_t stream) {
  static size_t allowed_state = 48 * 1024, allowed_out = 48 * 1024;      // (per instantiation)
  constexpr size_t for_state = (size_t)(RC * DK + RC * DV + 2 * RC + 4) * 4, for_scores = (size_t)2 * RC * (DK + 4) * 4;
  constexpr size_t smem_state = for_state > for_scores ? for_state : for_scores, smem_out = SsdOutSmem<DK, DV>::BYTES;
  int rc = rc_smem(ssd_state_kernel<DK, DV>, smem_state, allowed_state);
  if (rc == SLLM_OK) rc = rc_smem(ssd_out_kernel<DK, DV>, smem_out, allowed_out);
  if (rc != SLLM_OK) return rc;
  const dim3 grid((unsigned)chunks, (unsigned)p.H);
  launch_kernel(ssd_state_kernel<DK, DV>, dim3((unsigned)chunks, (unsigned)(p.H + p.groups)), 2 * DK, smem_state, stream, p);
  const int size = p.dk * p.dv;
  const bool vec = size % 4 == 0 && (((uintptr_t)p.state | (uintptr_t)p.scratch) & 15) == 0;
  const int per_cta = RC_SCAN_THREADS * (vec ? 4 : 1);
  const dim3 scan((unsigned)((size + per_cta - 1) / per_cta), (unsigned)p.H, (unsigned)runs);
  if (vec) launch_kernel(ssd_scan_kernel<4>, scan, RC_SCAN_THREADS, 0, stream, p);
  else launch_kernel(ssd_scan_kernel<1>, scan, RC_SCAN_THREADS, 0, stream, p);
  launch_kernel(ssd_out_kernel<DK, DV>, grid, RC_OUT_THREADS, smem_out, stream, p);
  return launch_status("state_space_chunked");
}

// VEC channels a thread at a time; the gated row waits in shared memory for its root mean square
template <typename TO, int VEC>
__global__ void __launch_bounds__(512)
gated_group_norm_kernel(const float* __restrict__ y, const float* __restrict__ gate, int ldg, int off_g, const float* __restrict__ gain, float eps,
                        int groups, TO* __restrict__ out, int n) {
  extern __shared__ __align__(16) float gg_v[];          // [n / groups]
  __shared__ float red[33];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x / groups, part = blockIdx.x % groups, size = n / groups;
  const float* x = y + (size_t)t * n + (size_t)part * size;
  const float* z = gate + (size_t)t * ldg + off_g + part * size;
  TO* o = out + (size_t)t * n + (size_t)part * size;
  gain += part * size;
  float ss = 0.f;
  for (int i = threadIdx.x * VEC; i < size; i += blockDim.x * VEC) {
    if constexpr (VEC == 4) {
      const float4 a = *reinterpret_cast<const float4*>(x + i), g = *reinterpret_cast<const float4*>(z + i);
      const float4 v = make_float4(a.x * rc_silu<TO>(g.x), a.y * rc_silu<TO>(g.y), a.z * rc_silu<TO>(g.z), a.w * rc_silu<TO>(g.w));
      *reinterpret_cast<float4*>(gg_v + i) = v;
      ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
    } else {
      const float v = x[i] * rc_silu<TO>(z[i]);
      gg_v[i] = v;
      ss = fmaf(v, v, ss);
    }
  }
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)size + eps);
  for (int i = threadIdx.x * VEC; i < size; i += blockDim.x * VEC) {      // (each thread reads what it wrote itself)
    if constexpr (VEC == 4) {
      const float4 v = *reinterpret_cast<const float4*>(gg_v + i), w = *reinterpret_cast<const float4*>(gain + i);
      const float r[4] = {v.x * inv * w.x, v.y * inv * w.y, v.z * inv * w.z, v.w * inv * w.w};
      rc_store4(o + i, r);
    } else {
      o[i] = from_f32<TO>(gg_v[i] * inv * gain[i]);
    }
  }
}

}  // namespace sllm

using namespace sllm;

SLLM_EXPORT int sllm_state_space_chunked_supports(int n, int dv) { return n >= 1 && n <= 128 && dv >= 1 && dv <= 128; }

// x | B | C in the columns of `xbc` [T, ldx] (x head by head, B and C group by group), step logits at columns off_dt + h of `dtp` [T, ldd].  `chunks` pieces
// of at most 64 tokens that belong to `runs` requests (run_seq: rows of state_slots; run_first, run_count: their chunks, consecutive).
// scratch: float32 [chunks, H, N, dv], scores [chunks, groups, 64, 64], keeps [chunks, H].  Rows of other requests are neither read nor written.
SLLM_EXPORT int sllm_state_space_chunked(const float* xbc, int ldx, const float* dtp, int ldd, int off_dt, const float* dt_bias, const float* a_log,
                                         const float* skip, float* state, const int* state_slots, const int* chunk_t0, const int* chunk_n, int chunks,
                                         const int* run_seq, const int* run_first, const int* run_count, int runs, float* scratch, float* scores, float* keeps, float* out,
                                         int H, int groups, int N, int dv, cudaStream_t stream) {
  SLLM_REQUIRE(chunks >= 0 && runs >= 0 && runs <= 65535 && H > 0 && groups > 0 && H + groups <= 65535 && H % groups == 0, "state_space_chunked: bad sizes chunks=%d runs=%d H=%d groups=%d",
               chunks, runs, H, groups);
  SLLM_REQUIRE(sllm_state_space_chunked_supports(N, dv), "state_space_chunked: states of %d x %d are outside 1..128", N, dv);
  SLLM_REQUIRE(ldx >= H * dv + 2 * groups * N && off_dt >= 0 && off_dt + H <= ldd, "state_space_chunked: columns outside the inputs' %d and %d", ldx, ldd);
  SLLM_REQUIRE(scratch != nullptr && scores != nullptr && keeps != nullptr && ((uintptr_t)scratch & 15) == 0, "state_space_chunked: scratch must be 16-byte aligned");
  if (chunks == 0 || runs == 0) return SLLM_OK;
  SsdParams p;
  p.xbc = xbc; p.ldx = ldx; p.off_b = H * dv; p.off_c = H * dv + groups * N; p.dtp = dtp; p.ldd = ldd; p.off_dt = off_dt;
  p.dt_bias = dt_bias; p.a_log = a_log; p.skip = skip; p.state = state; p.state_slots = state_slots; p.chunk_t0 = chunk_t0; p.chunk_n = chunk_n;
  p.run_seq = run_seq; p.run_first = run_first; p.run_count = run_count; p.scratch = scratch; p.scores = scores; p.groups = groups; p.keeps = keeps; p.out = out;
  p.H = H; p.hdiv = H / groups; p.dk = N; p.dv = dv;
  const bool base16 = ((uintptr_t)xbc & 15) == 0 && ldx % 4 == 0;
  p.vec_bc = base16 && N % 4 == 0 && (H * dv) % 4 == 0;
  p.vec_x = base16 && dv % 4 == 0 && ((uintptr_t)out & 15) == 0;
  if (N <= 64 && dv <= 64) return launch_ssd<64, 64>(p, chunks, runs, stream);
  if (N <= 64) return launch_ssd<64, 128>(p, chunks, runs, stream);
  if (dv <= 64) return launch_ssd<128, 64>(p, chunks, runs, stream);
  return launch_ssd<128, 128>(p, chunks, runs, stream);
}

SLLM_EXPORT int sllm_state_space_token_supports(int N, int dv) {
  const int quads = dv / 4;
  return N >= 1 && dv % 4 == 0 && quads >= 1 && quads <= ST_THREADS && (quads & (quads - 1)) == 0 && (N + ST_THREADS / quads - 1) / (ST_THREADS / quads) <= 32;
}

// One token a request: row s of `xbc` and `dtp` is request s's.
SLLM_EXPORT int sllm_state_space_token(const float* xbc, int ldx, const float* dtp, int ldd, int off_dt, const float* dt_bias, const float* a_log,
                                       const float* skip, float* state, const int* state_slots, float* out, int S, int H, int groups, int N, int dv,
                                       cudaStream_t stream) {
  SLLM_REQUIRE(S >= 0 && H > 0 && H <= 65535 && groups > 0 && H % groups == 0, "state_space_token: bad sizes S=%d H=%d groups=%d", S, H, groups);
  SLLM_REQUIRE(sllm_state_space_token_supports(N, dv), "state_space_token: a state of %d x %d is not taken", N, dv);
  SLLM_REQUIRE(ldx >= H * dv + 2 * groups * N && off_dt >= 0 && off_dt + H <= ldd, "state_space_token: columns outside the inputs' %d and %d", ldx, ldd);
  SLLM_REQUIRE(((uintptr_t)state & 15) == 0, "state_space_token: the states must be 16-byte aligned");
  if (S == 0) return SLLM_OK;
  SsdTokenParams p;
  p.xbc = xbc; p.dtp = dtp; p.ldx = ldx; p.off_b = H * dv; p.off_c = H * dv + groups * N; p.ldd = ldd; p.off_dt = off_dt;
  p.dt_bias = dt_bias; p.a_log = a_log; p.skip = skip; p.state = state; p.state_slots = state_slots; p.out = out;
  p.H = H; p.hdiv = H / groups; p.N = N; p.dv = dv;
  const int rows = ST_THREADS / (dv / 4), per = (N + rows - 1) / rows;
  const dim3 grid((unsigned)S, (unsigned)H);
  if (per <= 2) launch_kernel(ssd_token_kernel<2>, grid, ST_THREADS, 0, stream, p);
  else if (per <= 4) launch_kernel(ssd_token_kernel<4>, grid, ST_THREADS, 0, stream, p);
  else if (per <= 8) launch_kernel(ssd_token_kernel<8>, grid, ST_THREADS, 0, stream, p);
  else if (per <= 16) launch_kernel(ssd_token_kernel<16>, grid, ST_THREADS, 0, stream, p);
  else launch_kernel(ssd_token_kernel<32>, grid, ST_THREADS, 0, stream, p);
  return launch_status("state_space_token");
}

SLLM_EXPORT int sllm_gated_group_norm(const float* y, const float* gate, int ldg, int off_g, const float* gain, float eps, int groups, void* out,
                                      int out_dtype, int T, int n, cudaStream_t stream) {
  SLLM_REQUIRE(T >= 0 && n > 0 && groups > 0 && n % groups == 0 && off_g >= 0 && off_g + n <= ldg, "gated_group_norm: bad sizes T=%d n=%d groups=%d", T, n, groups);
  const size_t smem = (size_t)(n / groups) * sizeof(float);
  SLLM_REQUIRE(smem <= 200 * 1024, "gated_group_norm: parts of %d channels do not fit the shared memory", n / groups);
  if (T == 0) return SLLM_OK;
  const unsigned blocks = (unsigned)T * (unsigned)groups;
  const int size = n / groups;
  const bool vec = size % 4 == 0 && ldg % 4 == 0 && off_g % 4 == 0 && (((uintptr_t)y | (uintptr_t)gate | (uintptr_t)gain | (uintptr_t)out) & 15) == 0;
  const int per = vec ? size / 4 : size, threads = per >= 512 ? 512 : (per + 31) / 32 * 32;
#define GG(TO_, VEC_)                                                                                                                        \
  do {                                                                                                                                       \
    static size_t allowed = 48 * 1024;                                                                                                       \
    if (int rc = rc_smem(gated_group_norm_kernel<TO_, VEC_>, smem, allowed)) return rc;                                                      \
    launch_kernel(gated_group_norm_kernel<TO_, VEC_>, blocks, threads, smem, stream, y, gate, ldg, off_g, gain, eps, groups, (TO_*)out, n);   \
    return launch_status("gated_group_norm");                                                                                                \
  } while (0)
  if (out_dtype == SLLM_F32) { if (vec) GG(float, 4); else GG(float, 1); }
  if (out_dtype == SLLM_BF16) { if (vec) GG(__nv_bfloat16, 4); else GG(__nv_bfloat16, 1); }
#undef GG
  SLLM_REQUIRE(false, "gated_group_norm: unknown dtype %d", out_dtype);
}
