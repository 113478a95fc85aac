// hy_delta.cuh — gated delta rule with one decay per head, and what its neighbour in the layer needs: cosine / sine tables of
// a step and the preparation of queries, rotated keys and unrotated keys-as-values (libjf_hybrid.so).
//
// Per head, S [dim, vdim], unit vectors k, q (q also times dim^(-1/2)), decay g and step size beta:
//   S <- g S ;  u = beta (v - S^T k) ;  S <- S + k u^T ;  o = S^T q        (the read-out sees the current token's write)
// Both dot products are taken over the state as the token finds it, side by side:
//   p = S^T k, r = S^T q ;  u = beta (v - g p) ;  o = g r + (k.q) u ;  S <- g S + k u^T
// so a token costs one pass over the state, one exchange between lanes and one update.  Value columns are independent of each
// other, so a head is cut into blocks of 256 / PARTS columns that run side by side on different SMs, and PARTS lanes share a
// pair of columns, each holding DR / PARTS of their key rows in registers (the layout of gla_kernel).  The next token's rows
// are read from shared memory while the current token's dot products travel between lanes.
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

// ---- gated delta rule, one decay per head ---------------------------------------------------------------------------------------------
// tokens staged per batch and shared memory: fp32 rows q, k | values | 3 scalars per token; two buffers of raw q, k, v rows
__host__ __device__ constexpr int delta_tb(int dr) { return dr <= 128 ? 32 : dr <= 256 ? 16 : dr <= 512 ? 8 : 4; }
template <typename AT>
__host__ __device__ constexpr size_t delta_head_smem(int dr, int parts) {
  const size_t tb = (size_t)delta_tb(dr), cpb = 256 / (size_t)parts, d2 = 2 * (size_t)dr;
  return (tb * (d2 + cpb + 4)) * 4 + 2 * tb * (d2 + (cpb < 8 ? 8 : cpb)) * sizeof(AT);
}

// in [T, ld] (after convolution and activation): q at col_q, k at col_k (G heads of dim each), v at col_v (H heads of vdim).
// ba [T, ldba] fp32: step-size pre-activations at column h, decay pre-activations at column H + h.
// o [T, ldo] fp32 (H heads of vdim), before the output norm.  state [slot][H][dim][vdim] fp32.
// grid (H * blocks_per_head, entries), 128 threads; lane layout and async_ok as in gla_kernel.
template <typename AT, int DR, int PARTS>
__global__ void __launch_bounds__(128) delta_head_kernel(Batch b, const AT* __restrict__ in, int ld, int col_q, int col_k, int col_v,
                                                         const float* __restrict__ ba, int ldba, const float* __restrict__ A_log,
                                                         const float* __restrict__ dt_bias, int H, int G, int dim, int vdim,
                                                         int blocks_per_head, int async_ok, float* __restrict__ state,
                                                         float* __restrict__ o, int ldo) {
  constexpr int TB = delta_tb(DR), RP = DR / PARTS, CW = 32 / PARTS, CPB = 8 * CW, CH = 16 / (int)sizeof(AT);
  constexpr int RW = 2 * DR + (CPB < 8 ? 8 : CPB);
  extern __shared__ __align__(16) unsigned char hy_smem[];
  float* sq = reinterpret_cast<float*>(hy_smem);               // [TB][DR] unit queries times dim^(-1/2)
  float* sk = sq + TB * DR;                                    // [TB][DR] unit keys
  float* sv = sk + TB * DR;                                    // [TB][CPB] values
  float4* sc = reinterpret_cast<float4*>(sv + TB * CPB);       // [TB] decay, step size, k.q
  AT* raw = reinterpret_cast<AT*>(sc + TB);                    // [2][TB][RW] raw q | k | v rows in flight
  const int h = blockIdx.x / blocks_per_head, c0 = (blockIdx.x % blocks_per_head) * CPB, e = blockIdx.y;
  const int g = h / (H / G);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int cl = 2 * (warp * CW + lane % CW), part = lane / CW, col = c0 + cl;
  const int ncol = min(CPB, vdim - c0);
  const int start = b.ent_start[e], cnt = b.ent_start[e + 1] - start, pos0 = b.ent_pos0[e];
  float* st = state + ((size_t)b.ent_slot[e] * H + h) * dim * vdim;
  float S[2][RP];
#pragma unroll
  for (int i = 0; i < RP; ++i) {
    const int r = 4 * (part + PARTS * (i / 4)) + (i & 3);
#pragma unroll
    for (int c = 0; c < 2; ++c) S[c][i] = (col + c < vdim && r < dim && pos0 > 0) ? st[(size_t)r * vdim + col + c] : 0.0f;
  }
  const float rate = expf(A_log[h]), bias = dt_bias[h], qscale = 1.0f / sqrtf((float)dim);
  const bool ahead = async_ok && cnt > 1;
  const AT* inq = in + col_q + g * dim;
  const AT* ink = in + col_k + g * dim;
  const AT* inv = in + col_v + h * vdim + c0;
  auto fetch = [&](int j0, int nb, int buf) {
    AT* dst = raw + (size_t)buf * TB * RW;
    const size_t t0 = (size_t)(start + j0);
    constexpr int QC = DR / CH, VC = CPB >= CH ? CPB / CH : 1;
    for (int i = tid; i < nb * QC; i += 128) {
      const int tt = i / QC, k = i % QC * CH;
      if (k >= dim) continue;
      jf::cp_async_16(dst + (size_t)tt * RW + k, inq + (t0 + tt) * ld + k, 16u);
      jf::cp_async_16(dst + (size_t)tt * RW + DR + k, ink + (t0 + tt) * ld + k, 16u);
    }
    for (int i = tid; i < nb * VC; i += 128) {
      const int tt = i / VC, k = i % VC * CH;
      if (k < ncol) jf::cp_async_16(dst + (size_t)tt * RW + 2 * DR + k, inv + (t0 + tt) * ld + k, 16u);
    }
    jf::cp_async_commit();
  };
  if (ahead) fetch(0, min(TB, cnt), 0);
  int buf = 0;
  for (int j0 = 0; j0 < cnt; j0 += TB, buf ^= 1) {
    const int nb = min(TB, cnt - j0);
    if (ahead) jf::cp_async_wait_all();
    __syncthreads();                                           // raw rows have landed; the previous batch is finished
    const AT* src = raw + (size_t)buf * TB * RW;
    // decays and step sizes: one thread per token; unit vectors and k.q: one warp per token
    float* scf = reinterpret_cast<float*>(sc);
    if (tid < nb) {
      const size_t t = (size_t)(start + j0 + tid);
      scf[4 * tid] = expf(-rate * softplus_f(ba[t * ldba + H + h] + bias));
      scf[4 * tid + 1] = sigmoid_f(ba[t * ldba + h]);
    }
#pragma unroll 2
    for (int tt = warp; tt < nb; tt += 4) {
      constexpr int EL = (DR + 31) / 32;
      const size_t t = (size_t)(start + j0 + tt);
      float qv[EL], kv[EL];
      float q2 = 0.0f, k2 = 0.0f, qk = 0.0f;
#pragma unroll
      for (int i = 0; i < EL; ++i) {
        const int k = lane + 32 * i;
        const bool ok = k < dim;
        qv[i] = ok ? to_f(ahead ? src[(size_t)tt * RW + k] : inq[t * ld + k]) : 0.0f;
        kv[i] = ok ? to_f(ahead ? src[(size_t)tt * RW + DR + k] : ink[t * ld + k]) : 0.0f;
        q2 = fmaf(qv[i], qv[i], q2); k2 = fmaf(kv[i], kv[i], k2); qk = fmaf(qv[i], kv[i], qk);
      }
      q2 = warp_sum(q2); k2 = warp_sum(k2); qk = warp_sum(qk);
      const float qi = qscale / sqrtf(q2 + 1e-6f), ki = 1.0f / sqrtf(k2 + 1e-6f);
#pragma unroll
      for (int i = 0; i < EL; ++i) {
        const int k = lane + 32 * i;
        if (k < DR) { sq[tt * DR + k] = qv[i] * qi; sk[tt * DR + k] = kv[i] * ki; }
      }
      if (lane == 0) scf[4 * tt + 2] = qk * qi * ki;
    }
    for (int i = tid; i < nb * CPB; i += 128) {
      const int tt = i / CPB, k = i % CPB;
      sv[i] = k < ncol ? to_f(ahead ? src[(size_t)tt * RW + 2 * DR + k] : inv[(size_t)(start + j0 + tt) * ld + k]) : 0.0f;
    }
    __syncthreads();
    if (ahead && j0 + TB < cnt) fetch(j0 + TB, min(TB, cnt - j0 - TB), buf ^ 1);     // that buffer was read before the barrier above
    float* po = o + (size_t)(start + j0) * ldo + h * vdim + col;
    float keep0 = 0.0f, keep1 = 0.0f;                          // lane `part` keeps the read-outs of token tt = part (mod PARTS)
    float k[RP], q[RP];
    float4 s; float2 v;
    auto rows = [&](int tt) {
      const float4* k4 = reinterpret_cast<const float4*>(sk + tt * DR) + part;
      const float4* q4 = reinterpret_cast<const float4*>(sq + tt * DR) + part;
#pragma unroll
      for (int i = 0; i < RP / 4; ++i) {
        const float4 kk = k4[i * PARTS], qq = q4[i * PARTS];
        k[4 * i] = kk.x; k[4 * i + 1] = kk.y; k[4 * i + 2] = kk.z; k[4 * i + 3] = kk.w;
        q[4 * i] = qq.x; q[4 * i + 1] = qq.y; q[4 * i + 2] = qq.z; q[4 * i + 3] = qq.w;
      }
      s = sc[tt];
      v = *reinterpret_cast<const float2*>(sv + tt * CPB + cl);
    };
    rows(0);
    for (int tt = 0; tt < nb; ++tt) {
      // values 0, 1: S^T k of both columns, 2, 3: S^T q
      float d[4] = {0.0f, 0.0f, 0.0f, 0.0f}, f[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
      for (int i = 0; i < RP; i += 2) {
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          d[c] = fmaf(S[c][i], k[i], d[c]);     f[c] = fmaf(S[c][i + 1], k[i + 1], f[c]);
          d[2 + c] = fmaf(S[c][i], q[i], d[2 + c]); f[2 + c] = fmaf(S[c][i + 1], q[i + 1], f[2 + c]);
        }
      }
      float kc[RP];
      const float4 sn = s;
      const float2 vn = v;
#pragma unroll
      for (int i = 0; i < RP; ++i) kc[i] = k[i];
      if (tt + 1 < nb) rows(tt + 1);
#pragma unroll
      for (int c = 0; c < 4; ++c) d[c] += f[c];
#pragma unroll
      for (int x = CW; x < 32; x <<= 1) {
#pragma unroll
        for (int c = 0; c < 4; ++c) d[c] += __shfl_xor_sync(0xffffffffu, d[c], x);
      }
      const float u0 = sn.y * fmaf(-sn.x, d[0], vn.x), u1 = sn.y * fmaf(-sn.x, d[1], vn.y);
#pragma unroll
      for (int i = 0; i < RP; ++i) {
        S[0][i] = fmaf(sn.x, S[0][i], kc[i] * u0);
        S[1][i] = fmaf(sn.x, S[1][i], kc[i] * u1);
      }
      const int slot = tt & (PARTS - 1);
      if (slot == part) { keep0 = fmaf(sn.z, u0, sn.x * d[2]); keep1 = fmaf(sn.z, u1, sn.x * d[3]); }
      if ((slot == PARTS - 1 || tt == nb - 1) && part <= slot) {
        float* row = po + (size_t)(tt - slot + part) * ldo;
        if (col < vdim) row[0] = keep0;
        if (col + 1 < vdim) row[1] = keep1;
      }
    }
  }
#pragma unroll
  for (int i = 0; i < RP; ++i) {
    const int r = 4 * (part + PARTS * (i / 4)) + (i & 3);
#pragma unroll
    for (int c = 0; c < 2; ++c)
      if (col + c < vdim && r < dim) st[(size_t)r * vdim + col + c] = S[c][i];
  }
}

}  // namespace hy
