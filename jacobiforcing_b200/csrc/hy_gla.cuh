// hy_gla.cuh — gated linear attention with one decay per key channel, retention (one fixed decay per head, rotated queries and
// keys), and the row kernels between the sublayers of blocks with plain RMS weights (libjf_hybrid.so).
//
// Per head, S [dim, vdim]:  S <- diag(a) S + k v^T ;  o = S^T q dim^(-1/2)   (the read-out sees the current token's write)
//   out = o / rms(o) * norm_w * silu(g)        (norm over the head's vdim, one weight shared by the heads)
// The decay a = sigmoid(z)^(1 / tau) leaves the decay projection's epilogue as fp32 (gemm_store).  Retention is the same
// recurrence with one number per head for a and with q, k rotated at their position (in fp32, between the projections and the
// recurrence) and no weight in the norm.
//
// The recurrence has no feedback from the read-out and its value columns are independent, so a head is cut into blocks of
// CPB = 128 / PARTS columns that run side by side on different SMs, and PARTS lanes share a column, each holding DR / PARTS
// of its key rows in registers; what does not depend on the state is made beforehand (linear_rows_kernel).  The norm needs
// whole heads: it follows in a kernel of its own (gla_out_kernel).
#pragma once
#include "hy_kernels.cuh"
#include "hy_delta.cuh"
#include "jf_ptx.cuh"

namespace hy {

// qk [T][H][q dim | k dim] fp32 from linear_rows_kernel, v [T, ldv] (H heads of vdim).  Decays: decay [T, ldd] fp32 (H heads of dim),
// or with HEAD one number per head, head_decay [H].  o [T, ldo] fp32 (H heads of vdim).  state [slot][H][dim][vdim] fp32.
// grid (H * blocks_per_head, entries), 128 threads.  Lane layout, vec and vvec as in delta_head_kernel.
template <typename AT, int DR, int PARTS, bool HEAD>
__global__ void __launch_bounds__(128) gla_kernel(Batch b, const float* __restrict__ qk, const AT* __restrict__ v, int ldv,
                                                  const float* __restrict__ decay, int ldd, const float* __restrict__ head_decay, int H,
                                                  int dim, int vdim, int blocks_per_head, int vec, int vvec, float* __restrict__ state,
                                                  float* __restrict__ o, int ldo) {
  constexpr int TB = lin_tb(DR), RP = DR / PARTS, CW = 32 / PARTS, CPB = lin_cpb(PARTS), VW = CPB < 8 ? 8 : CPB;
  constexpr int RW = HEAD ? 2 * DR : 3 * DR;                   // floats of a staged row: q | k (| decays)
  extern __shared__ __align__(16) unsigned char hy_smem[];
  float* sqk = reinterpret_cast<float*>(hy_smem);              // [2][TB][RW]
  AT* sv = reinterpret_cast<AT*>(sqk + 2 * TB * RW);           // [2][TB][VW]
  const int h = blockIdx.x / blocks_per_head, c0 = (blockIdx.x % blocks_per_head) * CPB, e = blockIdx.y;
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
  const float hd = HEAD ? head_decay[h] : 0.0f;
  if (dim < DR)                                                // rows beyond the head's key size stay zero
    for (int i = tid; i < 2 * TB * RW; i += 128) if (i % DR >= dim) sqk[i] = 0.0f;
  auto fetch = [&](int j0, int buf) {
    const int nb = min(TB, cnt - j0);
    const size_t t0 = (size_t)(start + j0);
    float* d = sqk + (size_t)buf * TB * RW;
    const float* src = qk + (t0 * H + h) * 2 * dim;
    const size_t ld = (size_t)H * 2 * dim;
    copy_rows(d, RW, src, ld, nb, dim, vec);
    copy_rows(d + DR, RW, src + dim, ld, nb, dim, vec);
    if (!HEAD) copy_rows(d + 2 * DR, RW, decay + t0 * ldd + h * dim, ldd, nb, dim, vec);
    copy_values(sv + (size_t)buf * TB * VW, VW, v + t0 * ldv + h * vdim + c0, ldv, nb, ncol, vvec);
    jf::cp_async_commit();
  };
  fetch(0, 0);
  constexpr int TG = TB < 8 ? TB : 8;                          // tokens whose read-outs are reduced together
  int buf = 0;
  for (int j0 = 0; j0 < cnt; j0 += TB, buf ^= 1) {
    const int nb = min(TB, cnt - j0);
    jf::cp_async_wait_all();
    __syncthreads();                                           // this batch has landed; the batch before it is finished
    if (j0 + TB < cnt) fetch(j0 + TB, buf ^ 1);
    const float* rb = sqk + (size_t)buf * TB * RW + 4 * part;
    const AT* vb = sv + (size_t)buf * TB * VW + min(cl, ncol - 1);
    float* po = o + (size_t)(start + j0) * ldo + h * vdim + col;
    // one token's update of this lane's key rows; returns its part of the read-out
    auto update = [&](int tt) {
      const float vv = to_f(vb[tt * VW]);
      float p0 = 0.0f, p1 = 0.0f;
#pragma unroll
      for (int i = 0; i < RP / 4; ++i) {
        const float4 q = *reinterpret_cast<const float4*>(rb + tt * RW + 4 * PARTS * i);
        const float4 k = *reinterpret_cast<const float4*>(rb + tt * RW + DR + 4 * PARTS * i);
        const float4 a = HEAD ? make_float4(hd, hd, hd, hd) : *reinterpret_cast<const float4*>(rb + tt * RW + 2 * DR + 4 * PARTS * i);
        float* R = &S[4 * i];
        R[0] = fmaf(a.x, R[0], k.x * vv); p0 = fmaf(R[0], q.x, p0);
        R[1] = fmaf(a.y, R[1], k.y * vv); p1 = fmaf(R[1], q.y, p1);
        R[2] = fmaf(a.z, R[2], k.z * vv); p0 = fmaf(R[2], q.z, p0);
        R[3] = fmaf(a.w, R[3], k.w * vv); p1 = fmaf(R[3], q.w, p1);
      }
      return p0 + p1;
    };
    int tt = 0;
    for (; tt + TG <= nb; tt += TG) {
      // TG tokens without a shuffle between them, then one exchange in which every step halves the tokens a lane keeps
      float p[TG];
#pragma unroll
      for (int u = 0; u < TG; ++u) p[u] = update(tt + u);
      int n = TG, base = 0;
#pragma unroll
      for (int s = 16; s >= CW; s >>= 1) {
        const bool hi = (lane & s) != 0;
        if (n > 1) {
          n >>= 1;
#pragma unroll
          for (int u = 0; u < TG / 2; ++u) {
            if (u >= n) break;
            const float other = __shfl_xor_sync(0xffffffffu, hi ? p[u] : p[u + n], s);
            p[u] = (hi ? p[u + n] : p[u]) + other;
          }
          base += hi ? n : 0;
        } else {
          p[0] += __shfl_xor_sync(0xffffffffu, p[0], s);
        }
      }
      constexpr int LEFT = TG > PARTS ? TG / PARTS : 1, SAME = PARTS > TG ? PARTS / TG : 1;     // tokens per lane, lanes per token
      if (live && (part & (SAME - 1)) == 0) {
#pragma unroll
        for (int u = 0; u < LEFT; ++u) po[(size_t)(tt + base + u) * ldo] = p[u];
      }
    }
    for (; tt < nb; ++tt) {
      float p = update(tt);
#pragma unroll
      for (int s = CW; s < 32; s <<= 1) p += __shfl_xor_sync(0xffffffffu, p, s);
      if (live && part == 0) po[(size_t)tt * ldo] = p;
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

// Norm per head, weight (NULL: none), output gate: out[t, h, :] = o / rms(o) * w * silu(g) * out_scale.  One warp per (token, head).
template <typename AT>
__global__ void __launch_bounds__(128) gla_out_kernel(int T, int H, int vdim, const float* __restrict__ o, int ldi,
                                                      const AT* __restrict__ g, int ldg, const float* __restrict__ w, float eps,
                                                      float out_scale, AT* __restrict__ out, int ldo) {
  const int unit = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (unit >= T * H) return;
  const size_t t = unit / H, c0 = (size_t)(unit % H) * vdim;
  const float* orow = o + t * ldi + c0;
  float ss = 0.0f;
  for (int k = lane; k < vdim; k += 32) ss = fmaf(orow[k], orow[k], ss);
  const float inv = out_scale / sqrtf(warp_sum(ss) / (float)vdim + eps);
  for (int k = lane; k < vdim; k += 32)
    out[t * ldo + c0 + k] = from_f<AT>(orow[k] * inv * (w ? w[k] : 1.0f) * silu_f(to_f(g[t * ldg + c0 + k])));
}

// ---- one token's row between two sublayers ----------------------------------------------------------------------------------
// x += a sublayer's result: its rows (y), or the mixture of a routed feed-forward (rows), or nothing (both NULL); through an
// RMS norm of its own first when post_w is given.  Then what the next sublayer reads: the RMS norm of the row (norm_w), or
// the row itself (cast_out: the stream's half of the loop projection's operand), in the activation type.
// A choice >= n_experts stands for the sublayer's input: h [T, width] in the activation type, the buffer the norm is then
// written to (a thread reads a channel before it writes it).
struct RowClose {
  const float* rows; int ldr; const int* pair_row; const int* ids; const float* wts; int top, n_experts;
  const void* norm_w; float eps;
  void* cast_out; int ld_cast;
  const float* y; int ldy; const void* post_w;
};

// V channels per thread at a time (V = 4: width and all leading dimensions are multiples of 4).
constexpr int HY_CLOSE_TOP = 64;                               // choices whose rows and weights are staged in shared memory
template <typename AT, typename WT, int V>
__global__ void __launch_bounds__(256) row_close_kernel(RowClose c, int width, float* __restrict__ x, AT* h) {
  typedef VecN<float, V> F;
  extern __shared__ __align__(16) unsigned char hy_smem[];
  float* xs = reinterpret_cast<float*>(hy_smem);               // [width]
  __shared__ float red[33];
  __shared__ int srow[HY_CLOSE_TOP];
  __shared__ float swt[HY_CLOSE_TOP];
  const int t = blockIdx.x;
  const int first = threadIdx.x * V, step = blockDim.x * V;
  const bool adds = c.rows || c.y;
  if (c.rows) {                                                // row of every staged choice, -1: an identity choice
    for (int k = threadIdx.x; k < min(c.top, HY_CLOSE_TOP); k += blockDim.x) {
      const int i = t * c.top + k;
      srow[k] = c.ids[i] >= c.n_experts ? -1 : c.pair_row ? c.pair_row[i] : i;
      swt[k] = c.wts[i];
    }
    __syncthreads();
  }
  float ss = 0.0f;
  auto result = [&](int ch) {
    if (c.y) return *reinterpret_cast<const F*>(c.y + (size_t)t * c.ldy + ch);
    F y{}, own{};
    {
      const VecN<AT, V> hv = *reinterpret_cast<const VecN<AT, V>*>(h + (size_t)t * width + ch);
#pragma unroll
      for (int j = 0; j < V; ++j) own.v[j] = to_f(hv.v[j]);
    }
#pragma unroll 4
    for (int k = 0; k < c.top; ++k) {
      int row; float w;
      if (k < HY_CLOSE_TOP) { row = srow[k]; w = swt[k]; }
      else {
        const int i = t * c.top + k;
        row = c.ids[i] >= c.n_experts ? -1 : c.pair_row ? c.pair_row[i] : i;
        w = c.wts[i];
      }
      const F r = row < 0 ? own : *reinterpret_cast<const F*>(c.rows + (size_t)row * c.ldr + ch);
#pragma unroll
      for (int j = 0; j < V; ++j) y.v[j] = fmaf(w, r.v[j], y.v[j]);
    }
    return y;
  };
  float pinv = 1.0f;
  if (c.post_w) {
    for (int ch = first; ch < width; ch += step) {
      const F y = result(ch);
      *reinterpret_cast<F*>(xs + ch) = y;
#pragma unroll
      for (int j = 0; j < V; ++j) ss = fmaf(y.v[j], y.v[j], ss);
    }
    pinv = 1.0f / sqrtf(block_sum(ss, red) / (float)width + c.eps);
    ss = 0.0f;
  }
  for (int ch = first; ch < width; ch += step) {
    F v = *reinterpret_cast<const F*>(x + (size_t)t * width + ch);
    if (adds) {
      if (c.post_w) {
        const F y = *reinterpret_cast<const F*>(xs + ch);
        const VecN<WT, V> w = *reinterpret_cast<const VecN<WT, V>*>((const WT*)c.post_w + ch);
#pragma unroll
        for (int j = 0; j < V; ++j) v.v[j] += y.v[j] * pinv * to_f(w.v[j]);
      } else {
        const F y = result(ch);
#pragma unroll
        for (int j = 0; j < V; ++j) v.v[j] += y.v[j];
      }
      *reinterpret_cast<F*>(x + (size_t)t * width + ch) = v;
    }
    *reinterpret_cast<F*>(xs + ch) = v;
#pragma unroll
    for (int j = 0; j < V; ++j) ss = fmaf(v.v[j], v.v[j], ss);
  }
  auto out = [&](AT* row, int ch, float f, const WT* w) {
    const F v = *reinterpret_cast<const F*>(xs + ch);
    VecN<AT, V> o;
#pragma unroll
    for (int j = 0; j < V; ++j) o.v[j] = from_f<AT>(w ? v.v[j] * f * to_f(w[ch + j]) : v.v[j]);
    *reinterpret_cast<VecN<AT, V>*>(row + ch) = o;
  };
  if (c.cast_out)
    for (int ch = first; ch < width; ch += step) out((AT*)c.cast_out + (size_t)t * c.ld_cast, ch, 1.0f, nullptr);
  if (!c.norm_w) return;
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)width + c.eps);
  for (int ch = first; ch < width; ch += step) out(h + (size_t)t * width, ch, inv, (const WT*)c.norm_w);
}

// The embedding output x0 into the second half of the loop projection's operand [T, 2 width].
template <typename AT>
__global__ void loop_origin_kernel(const float* __restrict__ x, int width, AT* __restrict__ out) {
  const int t = blockIdx.x;
  for (int c = threadIdx.x; c < width; c += blockDim.x) out[(size_t)t * 2 * width + width + c] = from_f<AT>(x[(size_t)t * width + c]);
}

}  // namespace hy
