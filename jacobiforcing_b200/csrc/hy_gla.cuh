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
// CPB = 256 / PARTS columns that run side by side on different SMs; PARTS lanes share a pair of columns, each holding DR / PARTS
// of their key rows in registers (two columns per lane: the rows read from shared memory per token, which bound the kernel with
// one column per lane, serve twice the work).  The norm needs whole heads: it follows in a kernel of its own (gla_out_kernel).
#pragma once
#include "hy_kernels.cuh"
#include "hy_delta.cuh"
#include "jf_ptx.cuh"

namespace hy {

// key rows staged per token and tokens staged per batch: about 48 KB of fp32 rows whatever the key size
__host__ __device__ constexpr int gla_tb(int dr) { return dr <= 128 ? 32 : dr <= 256 ? 16 : dr <= 512 ? 8 : 4; }
template <typename AT>
__host__ __device__ constexpr size_t gla_smem(int dr, int parts) {
  const size_t tb = (size_t)gla_tb(dr), cpb = 256 / (size_t)parts, d2 = 2 * (size_t)dr;
  // fp32 rows q, k | values; two buffers of raw q, k, v rows (values padded to 16 bytes) and of decays in flight
  return (tb * (d2 + cpb)) * 4 + 2 * tb * ((d2 + (cpb < 8 ? 8 : cpb)) * sizeof(AT) + (size_t)dr * 4);
}

// in [T, ld]: q at col_q, k at col_k (heads * dim each), v at col_v (heads * vdim).  decay [T, ldd] fp32 (heads * dim).
// o [T, ldo] fp32 (heads * vdim).  state [slot][H][dim][vdim] fp32.  grid (H * blocks_per_head, entries), 128 threads.
// Lane layout: columns 2 c, 2 c + 1 with c = warp * (32 / PARTS) + lane % (32 / PARTS), part = lane / (32 / PARTS); part r holds the key rows
// 4 (r + PARTS i) .. + 3, so the PARTS row quadruples a warp reads from shared memory at once lie next to each other.
// async_ok: head sizes, leading dimensions and column offsets are multiples of 16 bytes, and so is CPB: raw rows of the next batch of tokens travel by asynchronous
// copies while the current batch runs; short entries (decode steps) and odd sizes stage directly.
// ROT (retention): `decay` holds the cosines and sines of the step's positions instead (rot_tables_kernel; the first 2 pairs
// dimensions rotate as `rp` says), head_decay [H] the decays.
template <typename AT, int DR, int PARTS, bool ROT = false>
__global__ void __launch_bounds__(128) gla_kernel(Batch b, const AT* __restrict__ in, int ld, int col_q, int col_k, int col_v,
                                                  const float* __restrict__ decay, int ldd, int H, int dim, int vdim,
                                                  int blocks_per_head, int async_ok, float* __restrict__ state,
                                                  float* __restrict__ o, int ldo, const float* __restrict__ head_decay, RotPair rp) {
  constexpr int TB = gla_tb(DR), RP = DR / PARTS, CW = 32 / PARTS, CPB = 8 * CW, CH = 16 / (int)sizeof(AT);
  extern __shared__ __align__(16) unsigned char hy_smem[];
  float* sq = reinterpret_cast<float*>(hy_smem);               // [TB][DR] scaled queries
  float* sk = sq + TB * DR;                                    // [TB][DR] keys
  float* sv = sk + TB * DR;                                    // [TB][CPB] values
  float* sa = sv + TB * CPB;                                   // [2][TB][DR] decays (used in place), or cosines | sines
  constexpr int RW = 2 * DR + (CPB < 8 ? 8 : CPB);
  AT* raw = reinterpret_cast<AT*>(sa + 2 * TB * DR);           // [2][TB][RW] raw q | k | v rows in flight
  const int h = blockIdx.x / blocks_per_head, c0 = (blockIdx.x % blocks_per_head) * CPB, e = blockIdx.y;
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
  const float qscale = 1.0f / sqrtf((float)dim);
  const bool ahead = async_ok && cnt > 1;
  const AT* inq = in + col_q + h * dim;
  const AT* ink = in + col_k + h * dim;
  const AT* inv = in + col_v + h * vdim + c0;
  const float* dec = decay + (ROT ? 0 : h * dim);
  const int ndec = ROT ? 2 * rp.pairs : dim;                   // floats of a token's row of `decay` that are used
  const float hd = ROT ? head_decay[h] : 0.0f;
  // copies of a batch's raw rows: 16 bytes at a time, the row pitches are compile-time so no division by a run-time size
  auto fetch = [&](int j0, int nb, int buf) {
    AT* dst = raw + (size_t)buf * TB * RW;
    float* da = sa + (size_t)buf * TB * DR;
    const size_t t0 = (size_t)(start + j0);
    constexpr int QC = DR / CH, VC = CPB >= CH ? CPB / CH : 1, AC = DR / 4;
    for (int i = tid; i < nb * QC; i += 128) {
      const int tt = i / QC, k = i % QC * CH;
      if (k >= dim) continue;
      jf::cp_async_16(dst + (size_t)tt * RW + k, inq + (t0 + tt) * ld + k, 16u);
      jf::cp_async_16(dst + (size_t)tt * RW + DR + k, ink + (t0 + tt) * ld + k, 16u);
    }
    for (int i = tid; i < nb * AC; i += 128) {
      const int tt = i / AC, k = i % AC * 4;
      if (k < ndec) jf::cp_async_16(da + (size_t)tt * DR + k, dec + (t0 + tt) * ldd + k, 16u);
    }
    for (int i = tid; i < nb * VC; i += 128) {
      const int tt = i / VC, k = i % VC * CH;
      if (k < ncol) jf::cp_async_16(dst + (size_t)tt * RW + 2 * DR + k, inv + (t0 + tt) * ld + k, 16u);
    }
    jf::cp_async_commit();
  };
  if (ahead) {
    // rows beyond the head's key size are never copied: q and k are zero there, so the decay only has to be a number
    if (!ROT)
      for (int i = tid; i < 2 * TB * DR; i += 128) if (i % DR >= dim) sa[i] = 0.0f;
    fetch(0, min(TB, cnt), 0);
  }
  // one token's update of this lane's key rows; leaves its part of both columns' read-outs in p[0], p[1]
  auto update = [&](const float* ca, int tt, float* p) {
    const float4* a4 = reinterpret_cast<const float4*>(ca + tt * DR) + part;
    const float4* k4 = reinterpret_cast<const float4*>(sk + tt * DR) + part;
    const float4* q4 = reinterpret_cast<const float4*>(sq + tt * DR) + part;
    const float2 v2 = *reinterpret_cast<const float2*>(sv + tt * CPB + cl);
    float x[2] = {0.0f, 0.0f}, y[2] = {0.0f, 0.0f};
#pragma unroll
    for (int i = 0; i < RP / 4; ++i) {
      const float4 k = k4[i * PARTS], q = q4[i * PARTS];
      const float4 a = ROT ? make_float4(hd, hd, hd, hd) : a4[i * PARTS];
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        const float v = c ? v2.y : v2.x;
        float* R = &S[c][4 * i];
        R[0] = fmaf(a.x, R[0], k.x * v); x[c] = fmaf(R[0], q.x, x[c]);
        R[1] = fmaf(a.y, R[1], k.y * v); y[c] = fmaf(R[1], q.y, y[c]);
        R[2] = fmaf(a.z, R[2], k.z * v); x[c] = fmaf(R[2], q.z, x[c]);
        R[3] = fmaf(a.w, R[3], k.w * v); y[c] = fmaf(R[3], q.w, y[c]);
      }
    }
    p[0] = x[0] + y[0];
    p[1] = x[1] + y[1];
  };
  constexpr int TG = TB < 8 ? TB : 8;                          // tokens whose read-outs are reduced together
  int buf = 0;
  for (int j0 = 0; j0 < cnt; j0 += TB, buf ^= 1) {
    const int nb = min(TB, cnt - j0);
    if (ahead) jf::cp_async_wait_all();
    __syncthreads();                                           // raw rows have landed; the previous batch is finished
    float* ca = sa + (size_t)buf * TB * DR;
    if (ahead) {
      const AT* src = raw + (size_t)buf * TB * RW;
      constexpr int QC = DR / CH;
      for (int i = tid; i < nb * QC; i += 128) {
        const int tt = i / QC, k = i % QC * CH;
        VecN<AT, CH> rq{}, rk{};
        if (k < dim) {
          rq = *reinterpret_cast<const VecN<AT, CH>*>(src + (size_t)tt * RW + k);
          rk = *reinterpret_cast<const VecN<AT, CH>*>(src + (size_t)tt * RW + DR + k);
        }
        if (ROT && k < ndec) {
          const float* cs = ca + (size_t)tt * DR;
          float fq[CH], fk[CH];
          if (rp.half && rp.pairs % CH == 0) {                 // the partners of a chunk are a chunk
            const bool hi = k >= rp.pairs;
            const int kp = hi ? k - rp.pairs : k + rp.pairs, p0 = hi ? kp : k;
            const VecN<AT, CH> wq = *reinterpret_cast<const VecN<AT, CH>*>(src + (size_t)tt * RW + kp);
            const VecN<AT, CH> wk = *reinterpret_cast<const VecN<AT, CH>*>(src + (size_t)tt * RW + DR + kp);
#pragma unroll
            for (int c = 0; c < CH; ++c) {
              const float co = cs[p0 + c], si = hi ? cs[rp.pairs + p0 + c] : -cs[rp.pairs + p0 + c];
              fq[c] = fmaf(to_f(rq.v[c]), co, to_f(wq.v[c]) * si);
              fk[c] = fmaf(to_f(rk.v[c]), co, to_f(wk.v[c]) * si);
            }
          } else {
#pragma unroll
            for (int c = 0; c < CH; ++c) {
              fq[c] = to_f(rq.v[c]); fk[c] = to_f(rk.v[c]);
              if (k + c < ndec) {
                const int kp = rp.partner(k + c);
                fq[c] = rp.turn(cs, k + c, fq[c], to_f(src[(size_t)tt * RW + kp]));
                fk[c] = rp.turn(cs, k + c, fk[c], to_f(src[(size_t)tt * RW + DR + kp]));
              }
            }
          }
#pragma unroll
          for (int c = 0; c < CH; c += 4) {
            *reinterpret_cast<float4*>(&sq[tt * DR + k + c]) = make_float4(fq[c] * qscale, fq[c + 1] * qscale, fq[c + 2] * qscale, fq[c + 3] * qscale);
            *reinterpret_cast<float4*>(&sk[tt * DR + k + c]) = make_float4(fk[c], fk[c + 1], fk[c + 2], fk[c + 3]);
          }
          continue;
        }
#pragma unroll
        for (int c = 0; c < CH; c += 4) {
          *reinterpret_cast<float4*>(&sq[tt * DR + k + c]) = make_float4(to_f(rq.v[c]) * qscale, to_f(rq.v[c + 1]) * qscale, to_f(rq.v[c + 2]) * qscale, to_f(rq.v[c + 3]) * qscale);
          *reinterpret_cast<float4*>(&sk[tt * DR + k + c]) = make_float4(to_f(rk.v[c]), to_f(rk.v[c + 1]), to_f(rk.v[c + 2]), to_f(rk.v[c + 3]));
        }
      }
      for (int i = tid; i < nb * CPB; i += 128) {
        const int tt = i / CPB, k = i % CPB;
        sv[i] = k < ncol ? to_f(src[(size_t)tt * RW + 2 * DR + k]) : 0.0f;
      }
    } else {
      for (int i = tid; i < nb * DR; i += 128) {
        const int tt = i / DR, k = i % DR;
        const size_t t = (size_t)(start + j0 + tt);
        const bool ok = k < dim;
        float q = ok ? to_f(inq[t * ld + k]) : 0.0f, kk = ok ? to_f(ink[t * ld + k]) : 0.0f;
        if (ROT) {
          if (k < ndec) {
            const int kp = rp.partner(k);
            q = rp.turn(dec + t * ldd, k, q, to_f(inq[t * ld + kp]));
            kk = rp.turn(dec + t * ldd, k, kk, to_f(ink[t * ld + kp]));
          }
        } else {
          ca[i] = ok ? dec[t * ldd + k] : 0.0f;
        }
        sq[i] = q * qscale;
        sk[i] = kk;
      }
      for (int i = tid; i < nb * CPB; i += 128) {
        const int tt = i / CPB, k = i % CPB;
        sv[i] = k < ncol ? to_f(inv[(size_t)(start + j0 + tt) * ld + k]) : 0.0f;
      }
    }
    __syncthreads();
    if (ahead && j0 + TB < cnt) fetch(j0 + TB, min(TB, cnt - j0 - TB), buf ^ 1);     // that buffer was read before the barrier above
    float* po = o + (size_t)(start + j0) * ldo + h * vdim + col;
    int tt = 0;
    for (; tt + TG <= nb; tt += TG) {
      // TG tokens without a shuffle between them, then one exchange in which every step halves the values a lane keeps
      constexpr int VT = 2 * TG;                               // value 2 u + c: token tt + u, column col + c
      float p[VT];
#pragma unroll
      for (int u = 0; u < TG; ++u) update(ca, tt + u, p + 2 * u);
      int n = VT, base = 0;
#pragma unroll
      for (int s = 16; s >= CW; s >>= 1) {
        const bool hi = (lane & s) != 0;
        if (n > 1) {
          n >>= 1;
#pragma unroll
          for (int u = 0; u < VT / 2; ++u) {
            if (u >= n) break;
            const float other = __shfl_xor_sync(0xffffffffu, hi ? p[u] : p[u + n], s);
            p[u] = (hi ? p[u + n] : p[u]) + other;
          }
          base += hi ? n : 0;
        } else {
          p[0] += __shfl_xor_sync(0xffffffffu, p[0], s);
        }
      }
      constexpr int LEFT = VT > PARTS ? VT / PARTS : 1, SAME = PARTS > VT ? PARTS / VT : 1;     // values per lane, lanes per value
      if ((part & (SAME - 1)) == 0) {
#pragma unroll
        for (int u = 0; u < LEFT; ++u) {
          const int c = (base + u) & 1;
          if (col + c < vdim) po[(size_t)(tt + (base + u) / 2) * ldo + c] = p[u];
        }
      }
    }
    for (; tt < nb; ++tt) {
      float p[2];
      update(ca, tt, p);
#pragma unroll
      for (int s = CW; s < 32; s <<= 1) {
        p[0] += __shfl_xor_sync(0xffffffffu, p[0], s);
        p[1] += __shfl_xor_sync(0xffffffffu, p[1], s);
      }
      if (part < 2 && col + part < vdim) po[(size_t)tt * ldo + part] = part ? p[1] : p[0];
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
