// hy_delta.cuh — gated delta rule with one decay per head, and what its neighbour in the layer needs: cosine / sine tables of
// a step and the preparation of queries, rotated keys and unrotated keys-as-values (libjf_hybrid.so).
//
// Per head, S [dim, vdim], unit vectors k, q (q also times dim^(-1/2)), decay g and step size beta:
//   S <- g S ;  u = beta (v - S^T k) ;  S <- S + k u^T ;  o = S^T q        (the read-out sees the current token's write)
// Both dot products are taken over the state as the token finds it, side by side:
//   p = S^T k, r = S^T q ;  u = beta (v - g p) ;  o = g r + (k.q) u ;  S <- g S + k u^T
// so a token costs one pass over the state, one exchange between lanes and one update.  Value columns are independent of each
// other, so a head is cut into blocks of 128 / PARTS columns that run side by side on different SMs, and PARTS lanes share a
// column, each holding DR / PARTS of its key rows in registers.  With one warp per scheduler the recurrence runs at about a
// third of the issue rate whatever the layout, so its time is its instruction count: everything that does not depend on the
// state (convolutions, unit vectors, k.q, decays, step sizes; rotations) is made beforehand, once per token and key head, by
// kernels of their own that leave fp32 rows, and the recurrence copies those asynchronously.
#pragma once
#include "hy_kernels.cuh"
#include "hy_mixers.cuh"
#include "jf_ptx.cuh"

namespace hy {

// ---- cosines and sines of a step's positions, one table per distinct rotation of the model -----------------------------------------
// out [T, ld]: cosines of the pairs, then their sines (both times mag), zeros up to ld; angles in fp64.
struct RotTable { const double* freq; int pairs; float mag; float* out; int ld; };

__global__ void rot_tables_kernel(Batch b, const RotTable* __restrict__ tables) {
  const RotTable r = tables[blockIdx.y];
  const int t = blockIdx.x;
  const double pos = (double)b.tok_pos[t];
  float* row = r.out + (size_t)t * r.ld;
  for (int i = threadIdx.x; i < r.pairs; i += blockDim.x) {
    double s, c;
    sincos(pos * r.freq[i], &s, &c);
    row[i] = (float)c * r.mag;
    row[r.pairs + i] = (float)s * r.mag;
  }
  for (int i = 2 * r.pairs + threadIdx.x; i < r.ld; i += blockDim.x) row[i] = 0.0f;
}

// Dimension k < 2 pairs of a rotated row: its partner's index, and its value from its own and its partner's.
struct RotPair {
  int pairs, half;                                           // half: dimension i turns with i + pairs, else 2i with 2i + 1
  __device__ __forceinline__ int partner(int k) const { return half ? (k < pairs ? k + pairs : k - pairs) : k ^ 1; }
  __device__ __forceinline__ float turn(const float* cs, int k, float own, float other) const {
    const int p = half ? (k < pairs ? k : k - pairs) : k >> 1;
    const float c = cs[p], s = cs[pairs + p];
    return (half ? k >= pairs : k & 1) ? fmaf(own, c, other * s) : fmaf(own, c, -other * s);
  }
};

// ---- attention whose values are its unrotated keys: queries rotated in place, keys into their pages rotated and as they are -------
// in [T, ld]: queries at col_q (H heads of dim), keys at col_k (G heads of dim); cs [T, ldc] from rot_tables_kernel.
template <typename AT>
__global__ void __launch_bounds__(128) key_value_prep_kernel(Batch b, AT* __restrict__ in, int ld, int col_q, int col_k, int H, int G, int dim,
                                                             const float* __restrict__ cs, int ldc, RotPair r, AT* __restrict__ kc,
                                                             AT* __restrict__ vc) {
  const int t = blockIdx.x;
  const int e = b.tok_ent[t], pos = b.tok_pos[t];
  const int page = b.pages[(size_t)e * b.max_pages + pos / b.page_size], in_page = pos % b.page_size;
  AT* row = in + (size_t)t * ld;
  const float* c = cs + (size_t)t * ldc;
  for (int i = threadIdx.x; i < H * r.pairs; i += blockDim.x) {
    AT* qh = row + col_q + (i / r.pairs) * dim;
    const int k = r.half ? i % r.pairs : 2 * (i % r.pairs), k2 = r.partner(k);
    const float u = to_f(qh[k]), v = to_f(qh[k2]);
    qh[k] = from_f<AT>(r.turn(c, k, u, v));
    qh[k2] = from_f<AT>(r.turn(c, k2, v, u));
  }
  for (int i = threadIdx.x; i < G * dim; i += blockDim.x) {
    const int g = i / dim, d = i % dim;
    const AT* kh = row + col_k + g * dim;
    const AT k = kh[d];
    const size_t at = (((size_t)page * G + g) * b.page_size + in_page) * dim + d;
    vc[at] = k;
    kc[at] = d < 2 * r.pairs ? from_f<AT>(r.turn(c, d, to_f(k), to_f(kh[r.partner(d)]))) : k;
  }
}

// ---- operands of a matrix-state recurrence: fp32 rows [T][heads][q dim | k dim] ------------------------------------------------------
// Rotated (rp.pairs > 0: the first 2 pairs dimensions, cs [T, ldc] from rot_tables_kernel), queries times dim^(-1/2).
template <typename AT>
__global__ void __launch_bounds__(1024) linear_rows_kernel(const AT* __restrict__ in, int ld, int col_q, int col_k, int H, int dim,
                                                          const float* __restrict__ cs, int ldc, RotPair rp, float* __restrict__ qk) {
  const int t = blockIdx.x;
  const AT* row = in + (size_t)t * ld;
  const float* c = rp.pairs > 0 ? cs + (size_t)t * ldc : nullptr;
  float* out = qk + (size_t)t * H * 2 * dim;
  const float qscale = 1.0f / sqrtf((float)dim);
  for (int i = threadIdx.x; i < H * dim; i += blockDim.x) {
    const int h = i / dim, k = i % dim;
    const AT* qh = row + col_q + h * dim;
    const AT* kh = row + col_k + h * dim;
    float q = to_f(qh[k]), kk = to_f(kh[k]);
    if (k < 2 * rp.pairs) {
      const int p = rp.partner(k);
      q = rp.turn(c, k, q, to_f(qh[p]));
      kk = rp.turn(c, k, kk, to_f(kh[p]));
    }
    out[(size_t)h * 2 * dim + k] = q * qscale;
    out[(size_t)h * 2 * dim + dim + k] = kk;
  }
}

// The delta rule's: causal convolution over time with silu of the columns [q (G heads of dim) | k | v (H heads of vdim)] at col0
// (see conv_kernel: w [C, taps], state [slot][taps - 1][C]), values into v [T, ldv] in the activation type, queries and keys made
// unit vectors per head, and per head (decay, step size, k.q) into sc [T][H].  ba [T, ldba] fp32: step-size pre-activations at
// column h, decay pre-activations at column H + h.  One block per token.
template <typename AT, typename WT>
__global__ void __launch_bounds__(1024) delta_rows_kernel(Batch b, const AT* __restrict__ u, int ldu, int col0, int H, int G, int dim, int vdim,
                                                         int taps, const WT* __restrict__ w, const float* __restrict__ state,
                                                         const float* __restrict__ ba, int ldba, const float* __restrict__ A_log,
                                                         const float* __restrict__ dt_bias, AT* __restrict__ v, int ldv,
                                                         float* __restrict__ qk, float4* __restrict__ sc) {
  extern __shared__ __align__(16) unsigned char hy_smem[];
  float* row = reinterpret_cast<float*>(hy_smem);              // [2 G dim] convolved queries, then keys
  const int t = blockIdx.x, e = b.tok_ent[t];
  const int start = b.ent_start[e], pos0 = b.ent_pos0[e], j = t - start;
  const int nk = G * dim, C = 2 * nk + H * vdim;
  const float* st = state + (size_t)b.ent_slot[e] * (taps - 1) * C;
  for (int c = threadIdx.x; c < C; c += blockDim.x) {
    float acc = 0.0f;
    for (int i = 0; i < taps; ++i) {
      const int src = j - (taps - 1) + i;
      float x = 0.0f;
      if (src >= 0) x = to_f(u[(size_t)(start + src) * ldu + col0 + c]);
      else if (pos0 + src >= 0) x = st[(size_t)(taps - 1 + src) * C + c];
      acc = fmaf(to_f(w[(size_t)c * taps + i]), x, acc);
    }
    acc = silu_f(acc);
    if (c < 2 * nk) row[c] = acc;
    else v[(size_t)t * ldv + c - 2 * nk] = from_f<AT>(acc);
  }
  __syncthreads();
  const int lane = threadIdx.x & 31, R = H / G;
  const float qscale = 1.0f / sqrtf((float)dim);
  for (int g = threadIdx.x >> 5; g < G; g += blockDim.x >> 5) {
    const float* qr = row + g * dim;
    const float* kr = row + nk + g * dim;
    float q2 = 0.0f, k2 = 0.0f, kq = 0.0f;
    for (int k = lane; k < dim; k += 32) { q2 = fmaf(qr[k], qr[k], q2); k2 = fmaf(kr[k], kr[k], k2); kq = fmaf(qr[k], kr[k], kq); }
    q2 = warp_sum(q2); k2 = warp_sum(k2); kq = warp_sum(kq);
    const float qi = qscale / sqrtf(q2 + 1e-6f), ki = 1.0f / sqrtf(k2 + 1e-6f);
    float* out = qk + ((size_t)t * G + g) * 2 * dim;
    for (int k = lane; k < dim; k += 32) { out[k] = qr[k] * qi; out[dim + k] = kr[k] * ki; }
    for (int r = lane; r < R; r += 32) {
      const int h = g * R + r;
      const float decay = expf(-expf(A_log[h]) * softplus_f(ba[(size_t)t * ldba + H + h] + dt_bias[h]));
      sc[(size_t)t * H + h] = make_float4(decay, sigmoid_f(ba[(size_t)t * ldba + h]), kq * qi * ki, 0.0f);
    }
  }
}

// ---- staging shared by the recurrences -----------------------------------------------------------------------------------------------
// tokens per batch; two buffers of fp32 rows q | k (DR each, zero beyond dim) and of value rows in the activation type
__host__ __device__ constexpr int lin_tb(int dr) { return dr <= 128 ? 32 : dr <= 256 ? 16 : dr <= 512 ? 8 : 4; }
__host__ __device__ constexpr int lin_cpb(int parts) { return 128 / parts; }
template <typename AT>
__host__ __device__ constexpr size_t lin_smem(int dr, int parts, int more_floats) {      // more_floats: per token, beside q and k
  return 2 * (size_t)lin_tb(dr) * ((2 * (size_t)dr + more_floats) * 4 + (lin_cpb(parts) < 8 ? 8 : lin_cpb(parts)) * sizeof(AT));
}

// n floats of each of nb rows (row r at src + r * ld) to dst + r * dld: asynchronous 16-byte copies where everything is aligned
__device__ __forceinline__ void copy_rows(float* dst, int dld, const float* src, size_t ld, int nb, int n, bool vec) {
  if (vec) {
    const int nc = n / 4;
    for (int i = threadIdx.x; i < nb * nc; i += 128) {
      const int r = i / nc, c = i % nc * 4;
      jf::cp_async_16(dst + r * dld + c, src + (size_t)r * ld + c, 16u);
    }
  } else {
    for (int i = threadIdx.x; i < nb * n; i += 128) dst[i / n * dld + i % n] = src[(size_t)(i / n) * ld + i % n];
  }
}
template <typename AT>
__device__ __forceinline__ void copy_values(AT* dst, int dld, const AT* src, size_t ld, int nb, int n, bool vec) {
  constexpr int CH = 16 / (int)sizeof(AT);
  if (vec) {
    const int nc = n / CH;
    for (int i = threadIdx.x; i < nb * nc; i += 128) {
      const int r = i / nc, c = i % nc * CH;
      jf::cp_async_16(dst + r * dld + c, src + (size_t)r * ld + c, 16u);
    }
  } else {
    for (int i = threadIdx.x; i < nb * n; i += 128) dst[i / n * dld + i % n] = src[(size_t)(i / n) * ld + i % n];
  }
}

// ---- gated delta rule, one decay per head ---------------------------------------------------------------------------------------------
// qk [T][G][q dim | k dim] and sc [T][H] from delta_rows_kernel, v [T, ldv] (H heads of vdim).  o [T, ldo] fp32 (H heads of vdim),
// before the output norm.  state [slot][H][dim][vdim] fp32.  grid (H * blocks_per_head, entries), 128 threads.
// Lane layout: column = warp * (32 / PARTS) + lane % (32 / PARTS), part = lane / (32 / PARTS); part r holds the key rows
// 4 (r + PARTS i) .. + 3, so the PARTS row quadruples a warp reads from shared memory at once lie next to each other.  vec: key
// rows are multiples of 16 bytes; vvec: a block's value rows are.
template <typename AT, int DR, int PARTS>
__global__ void __launch_bounds__(128) delta_head_kernel(Batch b, const float* __restrict__ qk, const AT* __restrict__ v, int ldv,
                                                         const float4* __restrict__ scal, int H, int G, int dim, int vdim,
                                                         int blocks_per_head, int vec, int vvec, float* __restrict__ state,
                                                         float* __restrict__ o, int ldo) {
  constexpr int TB = lin_tb(DR), RP = DR / PARTS, CW = 32 / PARTS, CPB = lin_cpb(PARTS), VW = CPB < 8 ? 8 : CPB;
  extern __shared__ __align__(16) unsigned char hy_smem[];
  float* sqk = reinterpret_cast<float*>(hy_smem);              // [2][TB][2 DR]
  float4* ssc = reinterpret_cast<float4*>(sqk + 2 * TB * 2 * DR);      // [2][TB]
  AT* sv = reinterpret_cast<AT*>(ssc + 2 * TB);                // [2][TB][VW]
  const int h = blockIdx.x / blocks_per_head, c0 = (blockIdx.x % blocks_per_head) * CPB, e = blockIdx.y;
  const int g = h / (H / G);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int cl = warp * CW + lane % CW, part = lane / CW, col = c0 + cl;
  const int ncol = min(CPB, vdim - c0);
  const bool live = col < vdim;
  const int start = b.ent_start[e], cnt = b.ent_start[e + 1] - start, pos0 = b.ent_pos0[e];
  float* st = state + ((size_t)b.ent_slot[e] * H + h) * dim * vdim;
  float S[RP];
#pragma unroll
  for (int i = 0; i < RP; ++i) {
    const int r = 4 * (part + PARTS * (i / 4)) + (i & 3);
    S[i] = (live && r < dim && pos0 > 0) ? st[(size_t)r * vdim + col] : 0.0f;
  }
  if (dim < DR)                                                // rows beyond the head's key size stay zero
    for (int i = tid; i < 2 * TB * 2 * DR; i += 128) if (i % DR >= dim) sqk[i] = 0.0f;
  auto fetch = [&](int j0, int buf) {
    const int nb = min(TB, cnt - j0);
    const size_t t0 = (size_t)(start + j0);
    float* d = sqk + (size_t)buf * TB * 2 * DR;
    const float* src = qk + (t0 * G + g) * 2 * dim;
    const size_t ld = (size_t)G * 2 * dim;
    copy_rows(d, 2 * DR, src, ld, nb, dim, vec);
    copy_rows(d + DR, 2 * DR, src + dim, ld, nb, dim, vec);
    if (tid < nb) jf::cp_async_16(ssc + buf * TB + tid, scal + (t0 + tid) * H + h, 16u);
    copy_values(sv + (size_t)buf * TB * VW, VW, v + t0 * ldv + h * vdim + c0, ldv, nb, ncol, vvec);
    jf::cp_async_commit();
  };
  fetch(0, 0);
  int buf = 0;
  for (int j0 = 0; j0 < cnt; j0 += TB, buf ^= 1) {
    const int nb = min(TB, cnt - j0);
    jf::cp_async_wait_all();
    __syncthreads();                                           // this batch has landed; the batch before it is finished
    if (j0 + TB < cnt) fetch(j0 + TB, buf ^ 1);
    const float* qb = sqk + (size_t)buf * TB * 2 * DR + 4 * part;
    const AT* vb = sv + (size_t)buf * TB * VW + min(cl, ncol - 1);
    float* po = o + (size_t)(start + j0) * ldo + h * vdim + col;
    float keep = 0.0f;                                         // lane `part` keeps the read-out of token tt = part (mod PARTS)
    float k[RP], q[RP], vv;
    float4 s;
    auto rows = [&](int tt) {
#pragma unroll
      for (int i = 0; i < RP / 4; ++i) {
        const float4 qq = *reinterpret_cast<const float4*>(qb + tt * 2 * DR + 4 * PARTS * i);
        const float4 kk = *reinterpret_cast<const float4*>(qb + tt * 2 * DR + DR + 4 * PARTS * i);
        q[4 * i] = qq.x; q[4 * i + 1] = qq.y; q[4 * i + 2] = qq.z; q[4 * i + 3] = qq.w;
        k[4 * i] = kk.x; k[4 * i + 1] = kk.y; k[4 * i + 2] = kk.z; k[4 * i + 3] = kk.w;
      }
      s = ssc[buf * TB + tt];
      vv = to_f(vb[tt * VW]);
    };
    rows(0);
#pragma unroll 2
    for (int tt = 0; tt < nb; ++tt) {
      float p0 = 0.0f, p1 = 0.0f, r0 = 0.0f, r1 = 0.0f, kc[RP];
#pragma unroll
      for (int i = 0; i < RP; i += 2) {
        p0 = fmaf(S[i], k[i], p0); p1 = fmaf(S[i + 1], k[i + 1], p1);
        r0 = fmaf(S[i], q[i], r0); r1 = fmaf(S[i + 1], q[i + 1], r1);
      }
      float p = p0 + p1, r = r0 + r1;
      const float4 sn = s;
      const float vn = vv;
#pragma unroll
      for (int i = 0; i < RP; ++i) kc[i] = k[i];
      rows(min(tt + 1, nb - 1));                               // the next token's rows fly under the exchange
#pragma unroll
      for (int x = CW; x < 32; x <<= 1) { p += __shfl_xor_sync(0xffffffffu, p, x); r += __shfl_xor_sync(0xffffffffu, r, x); }
      const float u = sn.y * fmaf(-sn.x, p, vn);
#pragma unroll
      for (int i = 0; i < RP; ++i) S[i] = fmaf(sn.x, S[i], kc[i] * u);
      const int slot = tt & (PARTS - 1);
      if (slot == part) keep = fmaf(sn.z, u, sn.x * r);
      if ((slot == PARTS - 1 || tt == nb - 1) && live && part <= slot) po[(size_t)(tt - slot + part) * ldo] = keep;
    }
  }
  if (live) {
#pragma unroll
    for (int i = 0; i < RP; ++i) {
      const int r = 4 * (part + PARTS * (i / 4)) + (i & 3);
      if (r < dim) st[(size_t)r * vdim + col] = S[i];
    }
  }
}

}  // namespace hy
