// The gated delta rule with one decay per head, from the raw projections to the gated read-out, over a packed batch. Everything between
// the projections is fp32: short causal convolutions, unit vectors, decays, write strengths, the dim x vdim state, norm and gate.
//
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q          per token
//
// Portions longer than a token run in three launches:
//   1. gd_prep_kernel: all tokens in parallel. Convolutions and silu, unit vectors, decays, write strengths, and for every block of 4
//      consecutive tokens of a sequence's portion what the recurrence needs to walk the block at once. With G_t the decays' product from
//      the block's start through token t and S0 the state before the block,
//        u_t = beta_t v_t - beta_t G_t (S0^T k_t) - sum_{s<t} beta_t (G_t / G_s) (k_t . k_s) u_s
//        o_t = G_t (S0^T q_t) + sum_{s<=t} (G_t / G_s) (q_t . k_s) u_s
//        S   = G_3 S0 + sum_s (G_3 / G_s) k_s u_s^T
//      so the eight contractions with S0 do not wait for one another: only a 4-step scalar chain per state column is left serial. The
//      ratios come from differences of summed log decays (all <= 0), never from quotients.
//   2. gd_scan_kernel: one CTA per (sequence, head, 32 state columns), a warp per 4 columns, a lane per dim / 32 state rows: a q / k value
//      read from shared memory serves 4 columns, and the 32 partial sums of a block (8 contractions x 4 columns) are reduced over the warp
//      by halving exchanges (31 shuffles) that leave exactly one of them in each lane.
//   3. the grouped RMS norm with gate of seqmix.cu.
// Single tokens are one launch (gd_step_kernel): one CTA per (sequence, head) reads and writes the head's state once, with both
// contractions taken from the state before the token (o = g S^T q + (k . q) u).
#include <math.h>

#include "seqmix.cuh"

namespace vy {

struct GdDev {
  const int* cu; const int* pos0; const int* slot;
  const float* q; long long ldq; const float* k; long long ldk; const float* v; long long ldv;
  const float* a; long long ld_a; const float* b; long long ld_b;
  const float* gate; long long ld_gate; int gate_act;
  const void* cwq; const void* cwk; const void* cwv; int cw_dt, taps;
  float* conv_state; int channels;   // 2 kv_heads dim + heads vdim
  const void* a_log; const void* norm; int w_dt;
  int heads, kv_heads, dim, vdim, dp, vp;   // dp, vp: dim and vdim padded to the kernels' tiles in the workspace
  float unit_eps, norm_eps;
  float* state;
  float* qn; float* kn; float* vn; float* rec; float* o;
  void* out; long long ld_out; int out_dt;
};

constexpr int GD_B = 4;          // tokens per block of the recurrence
constexpr int GD_REC = 16;       // floats per (token, head) record: [-beta G, beta, G, G_3 / G | 4 of the u chain | 4 of the o chain | G_3, pad]

// 32 values per lane -> the warp's sum of value number `lane`
__device__ __forceinline__ float reduce_scatter32(float (&v)[32], int lane) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const bool up = lane & o;
#pragma unroll
    for (int j = 0; j < o; ++j) {
      const float send = up ? v[j] : v[j + o], keep = up ? v[j + o] : v[j];
      v[j] = keep + __shfl_xor_sync(0xffffffffu, send, o);
    }
  }
  return v[0];
}

__device__ __forceinline__ float log_decay(const GdDev& d, int h, float a) {
  return fmaxf(-expf(ld_as_float(d.a_log, d.w_dt, h)) * softplusf_(a), MIN_LOG_DECAY);
}

// silu of the convolution of one channel at tokens i0 .. i0 + 3 of the portion (TP >= taps; positions before the portion from the ring)
template <int TP>
__device__ __forceinline__ void conv_block(const GdDev& d, const float* x, long long ldx, int base, int n, int i0, int pos0, const float* ring,
                                           const void* w, long long wc, float (&y)[GD_B]) {
  float xs[TP + GD_B - 1], wl[TP];
#pragma unroll
  for (int j = 0; j < TP + GD_B - 1; ++j) {
    const int i = i0 - (TP - 1) + j;
    xs[j] = 0.f;
    if (i0 - i < d.taps && i < n) {
      if (i >= 0) xs[j] = x[static_cast<long long>(base + i) * ldx];
      else if (pos0 + i >= 0) xs[j] = ring[static_cast<long long>((pos0 + i) % d.taps) * d.channels];
    }
  }
#pragma unroll
  for (int t = 0; t < TP; ++t) wl[t] = t < d.taps ? ld_as_float(w, d.cw_dt, wc * d.taps + (d.taps - 1 - t)) : 0.f;
#pragma unroll
  for (int t = 0; t < GD_B; ++t) {
    float s = 0.f;
#pragma unroll
    for (int lag = 0; lag < TP; ++lag) s = fmaf(wl[lag], xs[t + TP - 1 - lag], s);
    y[t] = i0 + t < n ? siluf_(s) : 0.f;
  }
}

// one warp per (block of 4 tokens, unit); units: the q / k heads (with the records of the heads that read them), then the value heads
template <int DR, int TP>
__global__ void __launch_bounds__(128) gd_prep_kernel(GdDev d) {
  pdl_trigger();
  pdl_wait();
  const int s = blockIdx.z, unit = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int base = d.cu[s], n = d.cu[s + 1] - base;
  const int i0 = (static_cast<int>(blockIdx.x) * 4 + warp) * GD_B;
  if (i0 >= n) return;
  const int pos0 = d.pos0[s];
  const float* ring = d.conv_state + static_cast<long long>(d.slot[s]) * d.taps * d.channels;
  const int qk_ch = d.kv_heads * d.dim;
  if (unit >= d.kv_heads) {
    const int h = unit - d.kv_heads;
    for (int c = lane; c < d.vp; c += 32) {
      float y[GD_B] = {0.f, 0.f, 0.f, 0.f};
      const long long ch = static_cast<long long>(h) * d.vdim + c;
      if (c < d.vdim) conv_block<TP>(d, d.v + ch, d.ldv, base, n, i0, pos0, ring + 2 * qk_ch + ch, d.cwv, ch, y);
#pragma unroll
      for (int t = 0; t < GD_B; ++t)
        if (i0 + t < n) d.vn[(static_cast<long long>(base + i0 + t) * d.heads + h) * d.vp + c] = y[t];
    }
    return;
  }
  float yq[DR][GD_B], yk[DR][GD_B];
#pragma unroll
  for (int r = 0; r < DR; ++r) {
    const int c = lane + 32 * r;
    const long long ch = static_cast<long long>(unit) * d.dim + c;
#pragma unroll
    for (int t = 0; t < GD_B; ++t) yq[r][t] = yk[r][t] = 0.f;
    if (c < d.dim) {
      conv_block<TP>(d, d.q + ch, d.ldq, base, n, i0, pos0, ring + ch, d.cwq, ch, yq[r]);
      conv_block<TP>(d, d.k + ch, d.ldk, base, n, i0, pos0, ring + qk_ch + ch, d.cwk, ch, yk[r]);
    }
  }
  // sums over the channels: q.q (0..3), k.k (4..7), q_t.k_s (8 + 4 t + s, all pairs), k_t.k_s for t > s (24 + t (t - 1) / 2 + s)
  float val[32];
#pragma unroll
  for (int j = 0; j < 32; ++j) val[j] = 0.f;
#pragma unroll
  for (int r = 0; r < DR; ++r) {
#pragma unroll
    for (int t = 0; t < GD_B; ++t) {
      val[t] = fmaf(yq[r][t], yq[r][t], val[t]);
      val[4 + t] = fmaf(yk[r][t], yk[r][t], val[4 + t]);
#pragma unroll
      for (int u = 0; u <= t; ++u) {
        val[8 + 4 * t + u] = fmaf(yq[r][t], yk[r][u], val[8 + 4 * t + u]);
        if (u < t) val[24 + t * (t - 1) / 2 + u] = fmaf(yk[r][t], yk[r][u], val[24 + t * (t - 1) / 2 + u]);
      }
    }
  }
  const float red = reduce_scatter32(val, lane);
  // lanes 0..3 / 4..7 turn their sums into the factors that make q (with dim^-1/2) and k unit vectors
  float inv = 1.f / sqrtf(red + d.unit_eps);
  if (lane < 4) inv *= 1.f / sqrtf(static_cast<float>(d.dim));
  float fq[GD_B], fk[GD_B];
#pragma unroll
  for (int t = 0; t < GD_B; ++t) {
    fq[t] = __shfl_sync(0xffffffffu, inv, t);
    fk[t] = __shfl_sync(0xffffffffu, inv, 4 + t);
  }
#pragma unroll
  for (int t = 0; t < GD_B; ++t) {
    if (i0 + t >= n) break;
    const long long o = (static_cast<long long>(base + i0 + t) * d.kv_heads + unit) * d.dp;
#pragma unroll
    for (int r = 0; r < DR; ++r) {
      d.qn[o + lane + 32 * r] = yq[r][t] * fq[t];
      d.kn[o + lane + 32 * r] = yk[r][t] * fk[t];
    }
  }
  // the heads' records: lane = kind 16 + 4 t + u
  const int t = (lane >> 2) & 3, u = lane & 3;
  const bool kind_o = lane >= 16;
  const float dot_q = __shfl_sync(0xffffffffu, red, 8 + 4 * t + u);
  const float dot_k = __shfl_sync(0xffffffffu, red, (24 + t * (t - 1) / 2 + u) & 31);
  const float fq_t = __shfl_sync(0xffffffffu, inv, t), fk_t = __shfl_sync(0xffffffffu, inv, 4 + t), fk_u = __shfl_sync(0xffffffffu, inv, 4 + u);
  const int rep = d.heads / d.kv_heads;
  for (int e = 0; e < rep; ++e) {
    const int h = unit * rep + e;
    const long long row_u = base + i0 + u;
    const bool has_u = i0 + u < n;
    float L = has_u ? log_decay(d, h, d.a[row_u * d.ld_a + h]) : 0.f;
    const float beta_u = has_u ? sigmoidf_(d.b[row_u * d.ld_b + h]) : 0.f;
    float x = __shfl_up_sync(0xffffffffu, L, 1, 4);
    if (u >= 1) L += x;
    x = __shfl_up_sync(0xffffffffu, L, 2, 4);
    if (u >= 2) L += x;   // L: summed log decays through token u (the same in every group of 4 lanes)
    const float Lt = __shfl_sync(0xffffffffu, L, t), LB = __shfl_sync(0xffffffffu, L, 3);
    const float beta_t = __shfl_sync(0xffffffffu, beta_u, t);
    const float ratio = u <= t ? expf(Lt - L) : 0.f;
    const float m = kind_o ? (u <= t ? ratio * dot_q * fq_t * fk_u : 0.f) : (u < t ? -beta_t * ratio * dot_k * fk_t * fk_u : 0.f);
    if (i0 + t < n) {
      float* rp = d.rec + (static_cast<long long>(base + i0 + t) * d.heads + h) * GD_REC;
      rp[4 + (kind_o ? 4 : 0) + u] = m;
      if (!kind_o && u == 0) {
        const float G = expf(Lt);
        *reinterpret_cast<float4*>(rp) = make_float4(-beta_t * G, beta_t, G, expf(LB - Lt));
        *reinterpret_cast<float4*>(rp + 12) = make_float4(expf(LB), 0.f, 0.f, 0.f);
      }
    }
  }
}

__device__ __forceinline__ void cp_async16(float* dst, const float* src, bool ok) {
  const unsigned a = static_cast<unsigned>(__cvta_generic_to_shared(dst));
  const int bytes = ok ? 16 : 0;   // 0: the destination is filled with zeros
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(a), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

constexpr int GD_CT = 16;   // tokens per shared-memory stage
constexpr int GD_T = 256;   // threads of the scan: 8 warps x 4 columns

template <int RPL>
struct GdStage {
  static constexpr int DP = 32 * RPL;
  static constexpr int floats = GD_CT * (2 * DP + 32 + GD_REC);
};

// the lane's state rows: RPL adjacent ones, or for 8 two runs of 4
template <int RPL>
__device__ __forceinline__ int gd_row(int lane, int r) { return RPL <= 4 ? lane * RPL + r : 128 * (r >> 2) + 4 * lane + (r & 3); }
template <int RPL>
__device__ __forceinline__ void gd_lane_rows(const float* p, int lane, float (&x)[RPL]) {
  if constexpr (RPL == 1) x[0] = p[lane];
  else if constexpr (RPL == 2) { const float2 v = *reinterpret_cast<const float2*>(p + 2 * lane); x[0] = v.x; x[1] = v.y; }
  else {
#pragma unroll
    for (int m = 0; m < RPL / 4; ++m) {
      const float4 v = *reinterpret_cast<const float4*>(p + 128 * m + 4 * lane);
      x[4 * m] = v.x; x[4 * m + 1] = v.y; x[4 * m + 2] = v.z; x[4 * m + 3] = v.w;
    }
  }
}

template <int RPL>
__global__ void __launch_bounds__(GD_T, RPL <= 4 ? 2 : 1) gd_scan_kernel(GdDev d) {
  pdl_trigger();
  pdl_wait();
  constexpr int DP = 32 * RPL;
  extern __shared__ __align__(16) float gd_smem[];
  __shared__ __align__(16) float us[GD_T / 32][2][GD_B * 4];
  const int s = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * 32;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int base = d.cu[s], n = d.cu[s + 1] - base;
  if (n <= 0) return;
  const int rep = d.heads / d.kv_heads, gq = h / rep;
  const int pos0 = d.pos0[s];
  const long long slot = d.slot[s];
  auto stage = [&](int b) { return gd_smem + b * GdStage<RPL>::floats; };
  auto fetch = [&](int t0, int b) {
    float* qs = stage(b);
    float* ks = qs + GD_CT * DP;
    float* vs = ks + GD_CT * DP;
    float* rs = vs + GD_CT * 32;
    for (int e = threadIdx.x; e < GD_CT * DP / 4; e += GD_T) {
      const int tt = e / (DP / 4), c = (e % (DP / 4)) * 4;
      const bool ok = t0 + tt < n;
      const long long o = (static_cast<long long>(base + (ok ? t0 + tt : 0)) * d.kv_heads + gq) * DP + c;
      cp_async16(qs + tt * DP + c, d.qn + o, ok);
      cp_async16(ks + tt * DP + c, d.kn + o, ok);
    }
    for (int e = threadIdx.x; e < GD_CT * 12; e += GD_T) {
      const int tt = e / 12, j = e % 12;
      const bool ok = t0 + tt < n;
      const long long row = (static_cast<long long>(base + (ok ? t0 + tt : 0)) * d.heads + h);
      if (j < 8) cp_async16(vs + tt * 32 + 4 * j, d.vn + row * d.vp + v0 + 4 * j, ok);
      else cp_async16(rs + tt * GD_REC + 4 * (j - 8), d.rec + row * GD_REC + 4 * (j - 8), ok);
    }
    cp_async_commit();
  };
  fetch(0, 0);
  // the portion's last inputs enter the convolution ring (the preparing launch, which read the older ones, is complete)
  if (blockIdx.x == 0) {
    float* ring = d.conv_state + slot * d.taps * d.channels;
    const int qk_ch = d.kv_heads * d.dim;
    for (int i = max(0, n - d.taps); i < n; ++i) {
      float* rp = ring + static_cast<long long>((pos0 + i) % d.taps) * d.channels;
      const long long row = base + i;
      for (int c = threadIdx.x; c < d.vdim; c += GD_T) rp[2 * qk_ch + h * d.vdim + c] = d.v[row * d.ldv + h * d.vdim + c];
      if (h % rep == 0)
        for (int c = threadIdx.x; c < d.dim; c += GD_T) {
          rp[gq * d.dim + c] = d.q[row * d.ldq + gq * d.dim + c];
          rp[qk_ch + gq * d.dim + c] = d.k[row * d.ldk + gq * d.dim + c];
        }
    }
  }
  float S[RPL][4];
  float* sp = d.state + (slot * d.heads + h) * d.dim * d.vdim;
  const int col0 = v0 + 4 * warp;
  const bool vec = d.vdim % 4 == 0;
#pragma unroll
  for (int r = 0; r < RPL; ++r) {
    const int i = gd_row<RPL>(lane, r);
#pragma unroll
    for (int e = 0; e < 4; ++e) S[r][e] = 0.f;
    if (pos0 > 0 && i < d.dim && col0 < d.vdim) {
      const float* p = sp + static_cast<long long>(i) * d.vdim + col0;
      if (vec) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        S[r][0] = x.x; S[r][1] = x.y; S[r][2] = x.z; S[r][3] = x.w;
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (col0 + e < d.vdim) S[r][e] = p[e];
      }
    }
  }
  const int lt = (lane >> 2) & 3, le = lane & 3;
  const bool kind_o = lane >= 16;
  for (int t0 = 0, b = 0; t0 < n; t0 += GD_CT, b ^= 1) {
    if (t0 + GD_CT < n) {
      fetch(t0 + GD_CT, b ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const float* qs = stage(b);
    const float* ks = qs + GD_CT * DP;
    const float* vs = ks + GD_CT * DP;
    const float* rs = vs + GD_CT * 32;
    const int nb = min(GD_CT, n - t0 + GD_B - 1) / GD_B;   // blocks of this stage (a last short one is padded with zero tokens)
    for (int blk = 0; blk < nb; ++blk) {
      const int tb = blk * GD_B;
      float kr[GD_B][RPL], val[32];
#pragma unroll
      for (int t = 0; t < GD_B; ++t) {
        float qr[RPL];
        gd_lane_rows<RPL>(ks + (tb + t) * DP, lane, kr[t]);
        gd_lane_rows<RPL>(qs + (tb + t) * DP, lane, qr);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          float x = S[0][e] * kr[t][0], y = S[0][e] * qr[0];
#pragma unroll
          for (int r = 1; r < RPL; ++r) {
            x = fmaf(S[r][e], kr[t][r], x);
            y = fmaf(S[r][e], qr[r], y);
          }
          val[4 * t + e] = x;
          val[16 + 4 * t + e] = y;
        }
      }
      const float4 r0 = *reinterpret_cast<const float4*>(rs + (tb + lt) * GD_REC);
      const float4 m = *reinterpret_cast<const float4*>(rs + (tb + lt) * GD_REC + (kind_o ? 8 : 4));
      const float gb = rs[tb * GD_REC + 12];
      const float vt = vs[(tb + lt) * 32 + 4 * warp + le];
      const float red = reduce_scatter32(val, lane);
      float acc = kind_o ? r0.z * red : fmaf(r0.x, red, r0.y * vt);
      acc = fmaf(m.x, __shfl_sync(0xffffffffu, acc, le), acc);
      acc = fmaf(m.y, __shfl_sync(0xffffffffu, acc, 4 + le), acc);
      acc = fmaf(m.z, __shfl_sync(0xffffffffu, acc, 8 + le), acc);
      acc = fmaf(m.w, __shfl_sync(0xffffffffu, acc, 12 + le), acc);
      float* ub = us[warp][blk & 1];
      if (kind_o) {
        if (t0 + tb + lt < n && col0 + le < d.vdim)
          d.o[static_cast<long long>(base + t0 + tb + lt) * d.heads * d.vdim + static_cast<long long>(h) * d.vdim + col0 + le] = acc;
      } else {
        ub[4 * lt + le] = acc * r0.w;
      }
      __syncwarp();
      float4 u4[GD_B];
#pragma unroll
      for (int t = 0; t < GD_B; ++t) u4[t] = *reinterpret_cast<const float4*>(ub + 4 * t);
#pragma unroll
      for (int r = 0; r < RPL; ++r) {
#pragma unroll
        for (int e = 0; e < 4; ++e) S[r][e] *= gb;
#pragma unroll
        for (int t = 0; t < GD_B; ++t) {
          S[r][0] = fmaf(kr[t][r], u4[t].x, S[r][0]);
          S[r][1] = fmaf(kr[t][r], u4[t].y, S[r][1]);
          S[r][2] = fmaf(kr[t][r], u4[t].z, S[r][2]);
          S[r][3] = fmaf(kr[t][r], u4[t].w, S[r][3]);
        }
      }
    }
    __syncthreads();   // the stage is refilled next
  }
#pragma unroll
  for (int r = 0; r < RPL; ++r) {
    const int i = gd_row<RPL>(lane, r);
    if (i >= d.dim || col0 >= d.vdim) continue;
    float* p = sp + static_cast<long long>(i) * d.vdim + col0;
    if (vec) *reinterpret_cast<float4*>(p) = make_float4(S[r][0], S[r][1], S[r][2], S[r][3]);
    else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (col0 + e < d.vdim) p[e] = S[r][e];
    }
  }
}

// single tokens: one CTA per (head, sequence), 8 warps; warp w holds state rows w + 8 r, lane 4 columns of a 128-column chunk (VEC:
// adjacent ones, one 16-byte access per row; else every 32nd)
constexpr int GS_T = 256, GS_MAXV = 512;

template <int RM, bool VEC>
__global__ void __launch_bounds__(GS_T, RM <= 16 ? 2 : 1) gd_step_kernel(GdDev d) {
  pdl_trigger();
  pdl_wait();
  __shared__ float qs[256], ks[256], vs[GS_MAXV], os[GS_MAXV];
  __shared__ float red[3][GS_T / 32];
  __shared__ __align__(16) float part[GS_T / 32][2][128];
  const int s = blockIdx.y, h = blockIdx.x;
  const int t = threadIdx.x, warp = t >> 5, lane = t & 31;
  const int base = d.cu[s];
  if (d.cu[s + 1] - base <= 0) return;
  const int rep = d.heads / d.kv_heads, gq = h / rep, pos = d.pos0[s];
  const long long slot = d.slot[s], row = base;
  float* sp = d.state + (slot * d.heads + h) * d.dim * d.vdim;
  auto col = [&](int c0, int e) { return c0 + (VEC ? 4 * lane + e : lane + 32 * e); };
  float S[RM][4];
  auto load_state = [&](int c0) {
#pragma unroll
    for (int r = 0; r < RM; ++r) {
      const int i = warp + 8 * r;
#pragma unroll
      for (int e = 0; e < 4; ++e) S[r][e] = 0.f;
      if (pos > 0 && i < d.dim) {
        const float* p = sp + static_cast<long long>(i) * d.vdim;
        if (VEC) {
          if (col(c0, 0) < d.vdim) {
            const float4 x = *reinterpret_cast<const float4*>(p + col(c0, 0));
            S[r][0] = x.x; S[r][1] = x.y; S[r][2] = x.z; S[r][3] = x.w;
          }
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (col(c0, e) < d.vdim) S[r][e] = p[col(c0, e)];
        }
      }
    }
  };
  load_state(0);   // in flight while the convolutions and unit vectors are made
  const int qk_ch = d.kv_heads * d.dim;
  float* ring = d.conv_state + slot * d.taps * d.channels;
  const int cur_ring = pos % d.taps;
#pragma unroll 1
  for (int c = t; c < 2 * d.dim + d.vdim; c += GS_T) {
    const int which = c < d.dim ? 0 : c < 2 * d.dim ? 1 : 2;
    const int j = which == 0 ? c : which == 1 ? c - d.dim : c - 2 * d.dim;
    const int ch = which == 2 ? h * d.vdim + j : gq * d.dim + j;            // channel of its tensor
    const int rc = which == 0 ? ch : which == 1 ? qk_ch + ch : 2 * qk_ch + ch;   // channel of the ring
    const float* x = which == 0 ? d.q + row * d.ldq : which == 1 ? d.k + row * d.ldk : d.v + row * d.ldv;
    const void* w = which == 0 ? d.cwq : which == 1 ? d.cwk : d.cwv;
    const float cur = x[ch];
    const int wo = ch * d.taps + d.taps - 1;
    float y = ld_as_float(w, d.cw_dt, wo) * cur;
    const int lags = min(d.taps - 1, pos);
    int e = cur_ring;
#pragma unroll 4
    for (int lag = 1; lag <= lags; ++lag) {
      e = e == 0 ? d.taps - 1 : e - 1;
      y = fmaf(ld_as_float(w, d.cw_dt, wo - lag), ring[e * d.channels + rc], y);
    }
    // the token's own ring entry is not one of those read above, so the CTAs of heads that share q / k do not race
    if (which == 2 || h % rep == 0) ring[cur_ring * d.channels + rc] = cur;
    (which == 0 ? qs : which == 1 ? ks : vs)[j] = siluf_(y);
  }
  __syncthreads();
  float sq = 0.f, sk = 0.f, sqk = 0.f;
  if (t < d.dim) {
    const float a = qs[t], b = ks[t];
    sq = a * a;
    sk = b * b;
    sqk = a * b;
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  sqk = warp_sum(sqk);
  if (lane == 0) { red[0][warp] = sq; red[1][warp] = sk; red[2][warp] = sqk; }
  __syncthreads();
  sq = sk = sqk = 0.f;
#pragma unroll
  for (int w = 0; w < GS_T / 32; ++w) { sq += red[0][w]; sk += red[1][w]; sqk += red[2][w]; }
  const float fq = 1.f / sqrtf(sq + d.unit_eps) / sqrtf(static_cast<float>(d.dim)), fk = 1.f / sqrtf(sk + d.unit_eps);
  const float kq = sqk * fq * fk;
  const float g = expf(log_decay(d, h, d.a[row * d.ld_a + h])), beta = sigmoidf_(d.b[row * d.ld_b + h]);
  for (int c0 = 0; c0 < d.vdim; c0 += 128) {
    if (c0 > 0) load_state(c0);
    float pr[4] = {0.f, 0.f, 0.f, 0.f}, pq[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int r = 0; r < RM; ++r) {
      const int i = warp + 8 * r;
      const float kv = i < d.dim ? ks[i] : 0.f, qv = i < d.dim ? qs[i] : 0.f;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        pr[e] = fmaf(S[r][e], kv, pr[e]);
        pq[e] = fmaf(S[r][e], qv, pq[e]);
      }
    }
    *reinterpret_cast<float4*>(&part[warp][0][4 * lane]) = make_float4(pr[0], pr[1], pr[2], pr[3]);
    *reinterpret_cast<float4*>(&part[warp][1][4 * lane]) = make_float4(pq[0], pq[1], pq[2], pq[3]);
    __syncthreads();
#pragma unroll
    for (int e = 0; e < 4; ++e) pr[e] = pq[e] = 0.f;
#pragma unroll 2
    for (int w = 0; w < GS_T / 32; ++w) {
      const float4 x = *reinterpret_cast<const float4*>(&part[w][0][4 * lane]), y = *reinterpret_cast<const float4*>(&part[w][1][4 * lane]);
      pr[0] += x.x; pr[1] += x.y; pr[2] += x.z; pr[3] += x.w;
      pq[0] += y.x; pq[1] += y.y; pq[2] += y.z; pq[3] += y.w;
    }
    float u[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = col(c0, e);
      u[e] = c < d.vdim ? beta * (vs[c] - g * fk * pr[e]) : 0.f;
      if (warp == 0 && c < d.vdim) os[c] = fmaf(g * fq, pq[e], kq * u[e]);
    }
#pragma unroll
    for (int r = 0; r < RM; ++r) {
      const int i = warp + 8 * r;
      if (i >= d.dim) continue;
      const float kv = ks[i] * fk;
      float* p = sp + static_cast<long long>(i) * d.vdim;
      float y[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] = fmaf(g, S[r][e], kv * u[e]);
      if (VEC) {
        if (col(c0, 0) < d.vdim) *reinterpret_cast<float4*>(p + col(c0, 0)) = make_float4(y[0], y[1], y[2], y[3]);
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (col(c0, e) < d.vdim) p[col(c0, e)] = y[e];
      }
    }
    __syncthreads();   // os complete (after the last chunk); part may be overwritten
  }
  float so = 0.f;
  for (int c = lane; c < d.vdim; c += 32) so = fmaf(os[c], os[c], so);
  const float inv = 1.f / sqrtf(warp_sum(so) / static_cast<float>(d.vdim) + d.norm_eps);
  for (int c = t; c < d.vdim; c += GS_T) {
    float y = os[c] * inv * ld_as_float(d.norm, d.w_dt, c);
    const long long o = static_cast<long long>(h) * d.vdim + c;
    if (d.gate) y *= apply_uact(d.gate[row * d.ld_gate + o], d.gate_act);
    st_from_float(d.out, d.out_dt, row * d.ld_out + o, y);
  }
}

static int gd_pad_dim(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }

template <int DR>
static cudaError_t launch_gd_prep(const GdDev& d, dim3 grid, cudaStream_t st) {
  return d.taps <= 4 ? launch_kernel(gd_prep_kernel<DR, 4>, grid, dim3(128), 0, st, d) : launch_kernel(gd_prep_kernel<DR, 16>, grid, dim3(128), 0, st, d);
}
template <int RPL>
static cudaError_t launch_gd_scan(const GdDev& d, int n_seqs, cudaStream_t st) {
  constexpr size_t smem = sizeof(float) * 2 * GdStage<RPL>::floats;
  if (smem > 48 * 1024) {
    static bool once = false;
    if (!once) {
      cudaError_t e = cudaFuncSetAttribute(gd_scan_kernel<RPL>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
      if (e != cudaSuccess) return e;
      once = true;
    }
  }
  return launch_kernel(gd_scan_kernel<RPL>, dim3((d.vdim + 31) / 32, d.heads, n_seqs), dim3(GD_T), smem, st, d);
}

}  // namespace vy

#define VY_NEED_DEVICE(name)                                                   \
  if (!vy_device_ok()) {                                                       \
    ::vy::set_error(name ": no sm_100 device (there is no CPU fallback)");     \
    return VY_ERR_NO_DEVICE;                                                   \
  }

extern "C" int64_t vy_gated_delta_workspace_floats(int64_t rows, int32_t max_new, int32_t heads, int32_t kv_heads, int32_t dim, int32_t vdim) {
  if (rows <= 0 || max_new <= 1 || heads <= 0 || kv_heads <= 0 || dim <= 0 || vdim <= 0) return 0;
  const int64_t dp = vy::gd_pad_dim(dim), vp = (vdim + 31) / 32 * 32;
  const int64_t o = (static_cast<int64_t>(heads) * vdim + 3) / 4 * 4;
  return rows * (2 * kv_heads * dp + heads * vp + heads * static_cast<int64_t>(vy::GD_REC) + o);
}

extern "C" int vy_gated_delta(const VyGatedDelta* p) {
  using namespace vy;
  VY_CHECK_ARG(p != nullptr, "vy_gated_delta: null params");
  VY_NEED_DEVICE("vy_gated_delta");
  VY_CHECK_ARG(p->n_seqs > 0 && p->n_seqs <= 65535 && p->max_new > 0 && p->rows > 0 && p->cu_tokens && p->pos0 && p->slot, "vy_gated_delta: bad batch");
  VY_CHECK_ARG(p->heads > 0 && p->heads <= 32767 && p->kv_heads > 0 && p->heads % p->kv_heads == 0 && p->dim > 0 && p->dim <= 256 && p->vdim > 0 &&
                   p->vdim <= GS_MAXV && p->taps >= 1 && p->taps <= 16, "vy_gated_delta: heads %d, kv_heads %d, dim %d (<= 256), vdim %d (<= %d), taps %d (1..16)",
               p->heads, p->kv_heads, p->dim, p->vdim, GS_MAXV, p->taps);
  VY_CHECK_ARG(p->q && p->k && p->v && p->a && p->b && p->conv_q && p->conv_k && p->conv_v && p->conv_state && p->a_log && p->norm && p->state && p->out &&
                   dtype_ok(p->conv_dtype) && dtype_ok(p->w_dtype) && dtype_ok(p->out_dtype), "vy_gated_delta: bad tensors");
  GdDev d;
  memset(&d, 0, sizeof(d));
  d.cu = p->cu_tokens; d.pos0 = p->pos0; d.slot = p->slot;
  d.q = p->q; d.ldq = p->ldq; d.k = p->k; d.ldk = p->ldk; d.v = p->v; d.ldv = p->ldv;
  d.a = p->a; d.ld_a = p->ld_a; d.b = p->b; d.ld_b = p->ld_b;
  d.gate = p->gate; d.ld_gate = p->ld_gate; d.gate_act = p->gate_act;
  d.cwq = p->conv_q; d.cwk = p->conv_k; d.cwv = p->conv_v; d.cw_dt = p->conv_dtype; d.taps = p->taps;
  d.conv_state = p->conv_state; d.channels = 2 * p->kv_heads * p->dim + p->heads * p->vdim;
  d.a_log = p->a_log; d.norm = p->norm; d.w_dt = p->w_dtype;
  d.heads = p->heads; d.kv_heads = p->kv_heads; d.dim = p->dim; d.vdim = p->vdim;
  d.dp = gd_pad_dim(p->dim); d.vp = (p->vdim + 31) / 32 * 32;
  d.unit_eps = p->unit_eps; d.norm_eps = p->norm_eps;
  d.state = p->state;
  d.out = p->out; d.ld_out = p->ld_out; d.out_dt = p->out_dtype;
  cudaStream_t st = static_cast<cudaStream_t>(p->stream);
  if (p->max_new == 1) {
    const dim3 grid(p->heads, p->n_seqs), block(GS_T);
    const bool vec = p->vdim % 4 == 0 && reinterpret_cast<uintptr_t>(p->state) % 16 == 0;
    cudaError_t e;
    if (p->dim <= 64) e = vec ? launch_kernel(gd_step_kernel<8, true>, grid, block, 0, st, d) : launch_kernel(gd_step_kernel<8, false>, grid, block, 0, st, d);
    else if (p->dim <= 128) e = vec ? launch_kernel(gd_step_kernel<16, true>, grid, block, 0, st, d) : launch_kernel(gd_step_kernel<16, false>, grid, block, 0, st, d);
    else e = vec ? launch_kernel(gd_step_kernel<32, true>, grid, block, 0, st, d) : launch_kernel(gd_step_kernel<32, false>, grid, block, 0, st, d);
    VY_CUDA_OK(e);
    VY_LAUNCH_OK();
    count_launch();
    return VY_OK;
  }
  VY_CHECK_ARG(p->workspace && reinterpret_cast<uintptr_t>(p->workspace) % 16 == 0 && reinterpret_cast<uintptr_t>(p->state) % 16 == 0 &&
                   p->workspace_floats >= vy_gated_delta_workspace_floats(p->rows, p->max_new, p->heads, p->kv_heads, p->dim, p->vdim),
               "vy_gated_delta: the workspace is 16-byte aligned and holds vy_gated_delta_workspace_floats(...) floats");
  d.qn = p->workspace;
  d.kn = d.qn + p->rows * p->kv_heads * d.dp;
  d.vn = d.kn + p->rows * p->kv_heads * d.dp;
  d.rec = d.vn + p->rows * p->heads * d.vp;
  d.o = d.rec + p->rows * p->heads * GD_REC;
  const dim3 grid((p->max_new + 4 * GD_B - 1) / (4 * GD_B), p->kv_heads + p->heads, p->n_seqs);
  cudaError_t e;
  switch (d.dp) {
    case 32: e = launch_gd_prep<1>(d, grid, st); break;
    case 64: e = launch_gd_prep<2>(d, grid, st); break;
    case 128: e = launch_gd_prep<4>(d, grid, st); break;
    default: e = launch_gd_prep<8>(d, grid, st); break;
  }
  VY_CUDA_OK(e);
  VY_LAUNCH_OK();
  count_launch();
  switch (d.dp) {
    case 32: e = launch_gd_scan<1>(d, p->n_seqs, st); break;
    case 64: e = launch_gd_scan<2>(d, p->n_seqs, st); break;
    case 128: e = launch_gd_scan<4>(d, p->n_seqs, st); break;
    default: e = launch_gd_scan<8>(d, p->n_seqs, st); break;
  }
  VY_CUDA_OK(e);
  VY_LAUNCH_OK();
  count_launch();
  VyRmsNorm nm;
  memset(&nm, 0, sizeof(nm));
  nm.tokens = p->rows; nm.groups = p->heads; nm.width = p->vdim;
  nm.x = d.o; nm.ldx = static_cast<int64_t>(p->heads) * p->vdim; nm.x_dtype = VY_F32;
  nm.weight = p->norm; nm.w_dtype = p->w_dtype; nm.w_mode = 1;
  nm.gate = p->gate; nm.ld_gate = p->ld_gate; nm.gate_dtype = VY_F32; nm.gate_act = p->gate_act;
  nm.eps = p->norm_eps; nm.coef = 1.f;
  nm.out = p->out; nm.ld_out = p->ld_out; nm.out_dtype = p->out_dtype;
  nm.stream = p->stream;
  return vy_rms_norm(&nm);
}
