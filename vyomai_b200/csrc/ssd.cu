// State-space recurrence with one decay per head and token (Mamba-2), from the raw projections to the gated, normed read-out, over a
// packed batch, all in fp32:
//
//   w = softplus(dt + dt_bias);   S <- exp(-exp(a_log) w) S + w b x^T;   y = S^T c + skip x;   u = y gate_act(z);   out = grouped RMS norm of u
//
// Portions longer than a token run in three launches: the short convolutions of x, b, c (ssd_conv_kernel: a thread walks a run of tokens
// of its channels with the last inputs in registers), the chunked recurrence of seqmix_tiled.cu (which also gates), the grouped norm of
// seqmix.cu. Single tokens are one launch (ssd_step_kernel): a CTA per (sequence, 1 to 4 heads of a group) reads and writes the state once; the CTA
// that finishes last in its sequence norms the whole row. The convolutions' inputs live in a ring by position (entry p mod taps, one
// entry more than the convolution looks back), so CTAs of heads that share b and c read old entries while one of them writes the new one.
#include <math.h>

#include "seqmix.cuh"

namespace vy {

struct SsdDev {
  const int* cu; const int* pos0; const int* slot;
  const float* x; long long ldx; const float* b; long long ldb; const float* c; long long ldc;
  const float* dt; long long ld_dt;
  const float* gate; long long ld_gate; int gate_act;
  const void* conv_w; const void* conv_b; int taps;
  float* ring; int channels;   // x [heads * vdim] | b [groups * dim] | c [groups * dim]
  const void* dt_bias; const void* a_log; const void* skip; const void* norm; int w_dt;
  int heads, groups, dim, vdim, inner, gn, norm_groups;
  float norm_eps;
  float* state; int* tickets;
  float* xc; long long ld_xc;   // convolved channels of all tokens (portions)
  float* u;                     // gated read-out [rows, inner]
  void* out; long long ld_out; int out_dt;
};

// the raw input of channel ch of the x | b | c row, its row stride
__device__ __forceinline__ const float* ssd_channel(const SsdDev& d, int ch, long long& ld) {
  if (ch < d.inner) { ld = d.ldx; return d.x + ch; }
  if (ch < d.inner + d.gn) { ld = d.ldb; return d.b + (ch - d.inner); }
  ld = d.ldc;
  return d.c + (ch - d.inner - d.gn);
}

constexpr int SC_T = 128, SC_TOK = 64, SC_G = 8;   // threads, tokens per CTA, tokens in flight per thread

template <int V>
__device__ __forceinline__ void ld_run(const float* p, float (&v)[V]) {
  if constexpr (V == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  } else {
    v[0] = *p;
  }
}
template <int V>
__device__ __forceinline__ void st_run(float* p, const float (&v)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}

// V channels per thread; TP: taps padded (the unused oldest ones weigh 0)
template <int TP, int V>
__global__ void __launch_bounds__(SC_T) ssd_conv_kernel(SsdDev d) {
  pdl_trigger();
  pdl_wait();
  const int ch = (static_cast<int>(blockIdx.x) * SC_T + static_cast<int>(threadIdx.x)) * V, s = blockIdx.z;
  const int base = d.cu[s], n = d.cu[s + 1] - base, i0 = static_cast<int>(blockIdx.y) * SC_TOK;
  if (ch >= d.channels || i0 >= n) return;
  const int pos0 = d.pos0[s];
  long long ld;
  const float* src = ssd_channel(d, ch, ld) + base * ld;
  float* ring = d.ring + static_cast<long long>(d.slot[s]) * d.taps * d.channels + ch;
  float w[TP][V], bias[V], xs[TP - 1 + SC_G][V];
#pragma unroll
  for (int e = 0; e < V; ++e) {
    bias[e] = d.conv_b ? ld_as_float(d.conv_b, d.w_dt, ch + e) : 0.f;
#pragma unroll
    for (int lag = 0; lag < TP; ++lag)
      w[lag][e] = lag < d.taps ? ld_as_float(d.conv_w, d.w_dt, static_cast<long long>(ch + e) * d.taps + (d.taps - 1 - lag)) : 0.f;
  }
  // xs[j]: input of token i - (TP - 1) + j; before the run's first token from the portion or, before that, from the ring
#pragma unroll
  for (int j = 0; j < TP - 1; ++j) {
    const int i = i0 - (TP - 1) + j;
#pragma unroll
    for (int e = 0; e < V; ++e) xs[j][e] = 0.f;
    if (i0 - i < d.taps) {
      if (i >= 0) ld_run<V>(src + i * ld, xs[j]);
      else if (pos0 + i >= 0) ld_run<V>(ring + static_cast<long long>((pos0 + i) % d.taps) * d.channels, xs[j]);
    }
  }
  const int i1 = min(i0 + SC_TOK, n);
  for (int i = i0; i < i1; i += SC_G) {
#pragma unroll
    for (int t = 0; t < SC_G; ++t) {
      if (i + t < i1) ld_run<V>(src + (i + t) * ld, xs[TP - 1 + t]);
      else {
#pragma unroll
        for (int e = 0; e < V; ++e) xs[TP - 1 + t][e] = 0.f;
      }
    }
#pragma unroll
    for (int t = 0; t < SC_G; ++t) {
      float y[V];
#pragma unroll
      for (int e = 0; e < V; ++e) {
        float a = bias[e];
#pragma unroll
        for (int lag = 0; lag < TP; ++lag) a = fmaf(w[lag][e], xs[t + TP - 1 - lag][e], a);
        y[e] = siluf_(a);
      }
      if (i + t < i1) st_run<V>(d.xc + static_cast<long long>(base + i + t) * d.ld_xc + ch, y);
    }
#pragma unroll
    for (int j = 0; j < TP - 1; ++j)
#pragma unroll
      for (int e = 0; e < V; ++e) xs[j][e] = xs[j + SC_G][e];
  }
  // only the first run's CTA reads the ring (a run is longer than the convolution looks back), and each thread only its own channels:
  // the same thread may now store the portion's last inputs
  if (blockIdx.y == 0) {
    for (int i = max(0, n - d.taps); i < n; ++i) {
      float v[V];
      ld_run<V>(src + i * ld, v);
      st_run<V>(ring + static_cast<long long>((pos0 + i) % d.taps) * d.channels, v);
    }
  }
}

// single tokens: one CTA per (run of `hpc` heads of one group, sequence): b and c are convolved once for the run. W state columns per
// thread (4: 16-byte accesses), Q column groups, SS_T / Q state rows at a time
constexpr int SS_T = 128, SS_B = 16, SS_H = 4;   // threads, state rows in flight per thread, most heads per CTA

// the convolved channel run of V channels (V 4: adjacent, aligned): taps from the ring, the token's own input `in`
template <int V>
__device__ __forceinline__ void ssd_conv_now(const SsdDev& d, const float* ring, int ch, int cur, int lags, const float (&in)[V], float (&y)[V]) {
#pragma unroll
  for (int e = 0; e < V; ++e) y[e] = d.conv_b ? ld_as_float(d.conv_b, d.w_dt, ch + e) : 0.f;
  if (V == 4 && d.taps == 4 && d.w_dt == VY_BF16) {   // the 4 channels' weights are 16 adjacent values
    float old[3][V];
#pragma unroll
    for (int lag = 1; lag < 4; ++lag) {
#pragma unroll
      for (int e = 0; e < V; ++e) old[lag - 1][e] = 0.f;
      if (lag <= lags) ld_run<V>(ring + ((cur - lag) & 3) * d.channels + ch, old[lag - 1]);
    }
    const uint2* wp = reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(d.conv_w) + ch * 4);
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const uint2 raw = wp[e];
      const float2 w32 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), w10 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
      y[e] = fmaf(w10.y, in[e], y[e]);
      y[e] = fmaf(w10.x, old[0][e], y[e]);
      y[e] = fmaf(w32.y, old[1][e], y[e]);
      y[e] = fmaf(w32.x, old[2][e], y[e]);
    }
  } else {
    const int wo = ch * d.taps + d.taps - 1;
#pragma unroll
    for (int e = 0; e < V; ++e) y[e] = fmaf(ld_as_float(d.conv_w, d.w_dt, wo + e * d.taps), in[e], y[e]);
    int r = cur;
    for (int lag = 1; lag <= lags; ++lag) {
      r = r == 0 ? d.taps - 1 : r - 1;
      float old[V];
      ld_run<V>(ring + r * d.channels + ch, old);
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = fmaf(ld_as_float(d.conv_w, d.w_dt, wo + e * d.taps - lag), old[e], y[e]);
    }
  }
#pragma unroll
  for (int e = 0; e < V; ++e) y[e] = siluf_(y[e]);
}

// RB > 0: the even geometry (16-byte columns, a power of two of column groups, RB adjacent rows per thread with nothing left over):
// consecutive blocks of rows, across the run's heads, stream through the registers without a bounds check
template <int W, int V, int RB>
__global__ void __launch_bounds__(SS_T, 4) ssd_step_kernel(SsdDev d, int hpc) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ __align__(16) float ss_smem[];
  float* part = ss_smem;                          // [2][SS_T * W]: the partial sums of this head and of the one before
  float* bs = part + 2 * SS_T * W;                // [dim], each row padded to a multiple of 4
  float* cs = bs + (d.dim + 3) / 4 * 4;           // [dim]
  float* xs = cs + (d.dim + 3) / 4 * 4;           // [hpc * vdim]
  float* zs = xs + (hpc * d.vdim + 3) / 4 * 4;    // [hpc * vdim] the gate's factors
  __shared__ float red[SS_T / 32];
  __shared__ float w_s[SS_H], decay_s[SS_H], skip_s[SS_H];
  __shared__ int last_s;
  const int s = blockIdx.y, h0 = blockIdx.x * hpc;
  const int t = threadIdx.x, warp = t >> 5, lane = t & 31;
  const int base = d.cu[s];
  if (d.cu[s + 1] - base <= 0) return;
  const int pos = d.pos0[s];
  const long long slot = d.slot[s], row = base;
  const int Q = (d.vdim + W - 1) / W, Qc = min(Q, SS_T), R = SS_T / Qc;
  const int rt = t / Qc, qt = t - rt * Qc;
  // lanes Qc apart hold the same columns when Qc is a power of two: their sums meet in registers, one partial row per warp is left
  const bool folded = Qc <= 32 && (Qc & (Qc - 1)) == 0;
  const bool one_pass = Q <= Qc && d.dim <= R * SS_B;   // a thread's registers hold its whole share of a head's state
  float* sp = d.state + (slot * d.heads + h0) * d.dim * d.vdim;
  constexpr int NS = RB > 0 ? RB : SS_B;
  float S[NS][W];
  float* sr = sp + rt * RB * d.vdim + qt * W;   // RB > 0: the thread's first row of the current block
  auto load_row = [&](float (&v)[W], const float* from, int q, int i) {
#pragma unroll
    for (int e = 0; e < W; ++e) v[e] = 0.f;
    if (pos > 0 && rt < R && q < Q && i < d.dim) ld_run<W>(from + i * d.vdim + q * W, v);
  };
  if constexpr (RB > 0) {   // in flight while the convolutions are made
    if (pos > 0) {
#pragma unroll
      for (int k = 0; k < NS; ++k) ld_run<W>(sr + k * d.vdim, S[k]);
    } else {
#pragma unroll
      for (int k = 0; k < NS; ++k)
#pragma unroll
        for (int e = 0; e < W; ++e) S[k][e] = 0.f;
    }
  } else {
#pragma unroll
    for (int k = 0; k < NS; ++k) load_row(S[k], sp, qt, rt + R * k);
  }
  {
    float* ring = d.ring + slot * d.taps * d.channels;
    const int rep = d.heads / d.groups, g = h0 / rep, cur = pos % d.taps, lags = min(d.taps - 1, pos), nx = hpc * d.vdim;
    const bool keeps_bc = h0 == g * rep;   // this CTA's input of b and c enters the ring
#pragma unroll 1
    for (int j = V * t; j < nx + 2 * d.dim; j += V * SS_T) {
      const bool is_x = j < nx, is_b = !is_x && j < nx + d.dim;
      const int jj = is_x ? j : is_b ? j - nx : j - nx - d.dim;
      const int ch = is_x ? h0 * d.vdim + jj : (is_b ? d.inner : d.inner + d.gn) + g * d.dim + jj;
      const float* src = is_x ? d.x + row * d.ldx + h0 * d.vdim : is_b ? d.b + row * d.ldb + g * d.dim : d.c + row * d.ldc + g * d.dim;
      float in[V], y[V];
      ld_run<V>(src + jj, in);
      ssd_conv_now<V>(d, ring, ch, cur, lags, in, y);
      // the token's own ring entry is not one of those read
      if (is_x || keeps_bc) st_run<V>(ring + cur * d.channels + ch, in);
      st_run<V>((is_x ? xs : is_b ? bs : cs) + jj, y);
    }
    for (int j = V * t; j < nx; j += V * SS_T) {
      float z[V];
      if (d.gate) ld_run<V>(d.gate + row * d.ld_gate + h0 * d.vdim + j, z);
#pragma unroll
      for (int e = 0; e < V; ++e) zs[j + e] = d.gate ? apply_uact(z[e], d.gate_act) : 1.f;
    }
    if (t >= SS_T - hpc) {
      const int k = SS_T - 1 - t, h = h0 + k;
      const float w = softplusf_(d.dt[row * d.ld_dt + h] + ld_as_float(d.dt_bias, d.w_dt, h));
      w_s[k] = w;
      decay_s[k] = expf(fmaxf(-expf(ld_as_float(d.a_log, d.w_dt, h)) * w, MIN_LOG_DECAY));
      skip_s[k] = ld_as_float(d.skip, d.w_dt, h);
    }
  }
  __syncthreads();
  int buf = 0;
  for (int hh = 0; hh < hpc; ++hh, sp += d.dim * d.vdim) {
    const float w = w_s[hh], decay = decay_s[hh], skip = skip_s[hh];
    const float* xh = xs + hh * d.vdim;
    const long long oh = static_cast<long long>(h0 + hh) * d.vdim;
    for (int q0 = 0; q0 < Q; q0 += Qc, buf ^= 1) {
      const int q = q0 + qt;
      const bool on = rt < R && q < Q;
      float wx[W], acc[W];
#pragma unroll
      for (int e = 0; e < W; ++e) {
        wx[e] = on ? w * xh[q * W + e] : 0.f;
        acc[e] = 0.f;
      }
      auto update = [&](float (&v)[W], int i) {
        if (!on || i >= d.dim) return;
        const float bv = bs[i], cv = cs[i];
#pragma unroll
        for (int e = 0; e < W; ++e) {
          v[e] = fmaf(decay, v[e], bv * wx[e]);
          acc[e] = fmaf(v[e], cv, acc[e]);
        }
        st_run<W>(sp + i * d.vdim + q * W, v);
      };
      if constexpr (RB > 0) {
        const int blocks = d.dim / (R * RB);
        for (int b = 0; b < blocks; ++b) {
          const bool more = pos > 0 && (b + 1 < blocks || hh + 1 < hpc);
          const float* bb = bs + (b * R + rt) * RB;
          const float* cb = cs + (b * R + rt) * RB;
          float* nx = sr + R * RB * d.vdim;   // the next block of rows (of this head or the next): takes the registers as they come free
#pragma unroll
          for (int k4 = 0; k4 < RB; k4 += 4) {
            const float4 b4 = f4(bb + k4), c4 = f4(cb + k4);
            const float bv[4] = {b4.x, b4.y, b4.z, b4.w}, cv[4] = {c4.x, c4.y, c4.z, c4.w};
#pragma unroll
            for (int k = 0; k < 4; ++k) {
#pragma unroll
              for (int e = 0; e < W; ++e) {
                S[k4 + k][e] = fmaf(decay, S[k4 + k][e], bv[k] * wx[e]);
                acc[e] = fmaf(S[k4 + k][e], cv[k], acc[e]);
              }
              st_run<W>(sr + (k4 + k) * d.vdim, S[k4 + k]);
            }
            if (more) {
#pragma unroll
              for (int k = 0; k < 4; ++k) ld_run<W>(nx + (k4 + k) * d.vdim, S[k4 + k]);
            } else {
#pragma unroll
              for (int k = 0; k < 4; ++k)
#pragma unroll
                for (int e = 0; e < W; ++e) S[k4 + k][e] = 0.f;
            }
          }
          sr = nx;
        }
      } else if (one_pass) {
        const bool more = hh + 1 < hpc;
#pragma unroll
        for (int k = 0; k < NS; ++k) {
          const int i = rt + R * k;
          update(S[k], i);
          if (more) load_row(S[k], sp + d.dim * d.vdim, q, i);   // the next head's row takes the register
        }
      } else {
        for (int k0 = 0; k0 * R < d.dim; k0 += NS) {
#pragma unroll
          for (int k = 0; k < NS; ++k)
            if (hh > 0 || q0 > 0 || k0 > 0) load_row(S[k], sp, q, rt + R * (k0 + k));
#pragma unroll
          for (int k = 0; k < NS; ++k) update(S[k], rt + R * (k0 + k));
        }
      }
      float* pb = part + buf * SS_T * W;
      const int prow = Qc * W;   // columns of one partial row
      if (folded) {
        for (int o = 16; o >= Qc; o >>= 1)
#pragma unroll
          for (int e = 0; e < W; ++e) acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], o);
        if (lane < Qc) st_run<W>(pb + warp * prow + lane * W, acc);
      } else {
        st_run<W>(pb + t * W, acc);
      }
      __syncthreads();   // the other buffer is free again: its readers passed the barrier before this one's writers did
      for (int j = t; j < prow; j += SS_T) {
        const int col = q0 * W + j;
        if (col >= d.vdim) continue;
        float y = skip * xh[col];
        if (folded) {
#pragma unroll
          for (int r = 0; r < SS_T / 32; ++r) y += pb[r * prow + j];
        } else {
          for (int r = 0; r < R; ++r) y += pb[r * prow + j];
        }
        d.u[row * d.inner + oh + col] = y * zs[hh * d.vdim + col];
      }
    }
  }
  // the last CTA of the sequence norms the row: `wpg` warps per group of columns, as many groups at a time as the CTA has warps for
  __threadfence();
  __syncthreads();
  if (t == 0) last_s = atomicAdd(d.tickets + slot, 1) == static_cast<int>(gridDim.x) - 1;
  __syncthreads();
  if (!last_s) return;
  if (t == 0) d.tickets[slot] = 0;
  __threadfence();
  constexpr int NW = SS_T / 32, NB = 16;   // warps; columns a lane has in flight
  const int gw = d.inner / d.norm_groups, at_once = min(d.norm_groups, NW), wpg = NW / at_once;
  const int own = warp / wpg, first = (warp - own * wpg) * 32 + lane, step = 32 * wpg;
  for (int g0 = 0; g0 < d.norm_groups; g0 += at_once) {
    const bool on = own < at_once && g0 + own < d.norm_groups;
    const int c0 = (g0 + own) * gw;
    const float* ur = d.u + row * d.inner + c0;
    float v[NB], ss = 0.f;
    auto fetch = [&](int b) {
#pragma unroll
      for (int k = 0; k < NB; ++k) {
        const int c = first + (b + k) * step;
        v[k] = on && c < gw ? __ldcg(ur + c) : 0.f;
      }
    };
    const int blocks = (gw + step * NB - 1) / (step * NB);   // one for rows of up to NB columns per lane: read once
    for (int b = 0; b < blocks; ++b) {
      fetch(b * NB);
#pragma unroll
      for (int k = 0; k < NB; ++k) ss = fmaf(v[k], v[k], ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = 0.f;
    for (int k = 0; k < wpg; ++k) ss += red[min(own * wpg + k, NW - 1)];
    const float inv = 1.f / sqrtf(ss / static_cast<float>(gw) + d.norm_eps);
    for (int b = 0; b < blocks; ++b) {
      if (blocks > 1) fetch(b * NB);
      float nw[NB];
#pragma unroll
      for (int k = 0; k < NB; ++k) {
        const int c = first + (b * NB + k) * step;
        nw[k] = on && c < gw ? ld_as_float(d.norm, d.w_dt, c0 + c) : 0.f;
      }
#pragma unroll
      for (int k = 0; k < NB; ++k) {
        const int c = first + (b * NB + k) * step;
        if (on && c < gw) st_from_float(d.out, d.out_dt, row * d.ld_out + c0 + c, v[k] * inv * nw[k]);
      }
    }
    __syncthreads();
  }
}

}  // namespace vy

#define VY_NEED_DEVICE(name)                                                   \
  if (!vy_device_ok()) {                                                       \
    ::vy::set_error(name ": no sm_100 device (there is no CPU fallback)");     \
    return VY_ERR_NO_DEVICE;                                                   \
  }

static int64_t up4(int64_t n) { return (n + 3) / 4 * 4; }

extern "C" int64_t vy_ssd_workspace_floats(int64_t rows, int32_t n_seqs, int32_t max_new, int32_t heads, int32_t groups, int32_t dim, int32_t vdim) {
  if (rows <= 0 || n_seqs <= 0 || max_new <= 0 || heads <= 0 || groups <= 0 || dim <= 0 || vdim <= 0) return 0;
  const int64_t inner = static_cast<int64_t>(heads) * vdim, channels = inner + 2LL * groups * dim;
  return up4(rows * inner) + (max_new > 1 ? rows * up4(channels) : 0);
}

extern "C" int vy_ssd(const VySsd* p) {
  using namespace vy;
  VY_CHECK_ARG(p != nullptr, "vy_ssd: null params");
  VY_NEED_DEVICE("vy_ssd");
  VY_CHECK_ARG(p->n_seqs > 0 && p->n_seqs <= 65535 && p->max_new > 0 && p->rows > 0 && p->cu_tokens && p->pos0 && p->slot, "vy_ssd: bad batch");
  VY_CHECK_ARG(p->heads > 0 && p->heads <= 65535 && p->groups > 0 && p->heads % p->groups == 0 && p->dim > 0 && p->dim <= 256 && p->vdim > 0 && p->vdim <= 1024 &&
                   p->taps >= 1 && p->taps <= 16, "vy_ssd: heads %d, groups %d, dim %d (<= 256), vdim %d (<= 1024), taps %d (1..16)", p->heads, p->groups, p->dim,
               p->vdim, p->taps);
  const long long inner = static_cast<long long>(p->heads) * p->vdim, gn = static_cast<long long>(p->groups) * p->dim;
  VY_CHECK_ARG(p->norm_groups > 0 && inner % p->norm_groups == 0 && inner + 2 * gn < (1 << 24), "vy_ssd: %d norm groups must divide %lld columns", p->norm_groups, inner);
  VY_CHECK_ARG(p->x && p->b && p->c && p->dt && p->conv_w && p->conv_state && p->dt_bias && p->a_log && p->skip && p->norm && p->state && p->tickets && p->out &&
                   dtype_ok(p->w_dtype) && dtype_ok(p->out_dtype), "vy_ssd: bad tensors");
  VY_CHECK_ARG(p->workspace && reinterpret_cast<uintptr_t>(p->workspace) % 16 == 0 && reinterpret_cast<uintptr_t>(p->state) % 16 == 0 &&
                   p->workspace_floats >= vy_ssd_workspace_floats(p->rows, p->n_seqs, p->max_new, p->heads, p->groups, p->dim, p->vdim),
               "vy_ssd: the workspace is 16-byte aligned and holds vy_ssd_workspace_floats(...) floats");
  SsdDev d;
  memset(&d, 0, sizeof(d));
  d.cu = p->cu_tokens; d.pos0 = p->pos0; d.slot = p->slot;
  d.x = p->x; d.ldx = p->ldx; d.b = p->b; d.ldb = p->ldb; d.c = p->c; d.ldc = p->ldc; d.dt = p->dt; d.ld_dt = p->ld_dt;
  d.gate = p->gate; d.ld_gate = p->ld_gate; d.gate_act = p->gate_act;
  d.conv_w = p->conv_w; d.conv_b = p->conv_b; d.taps = p->taps;
  d.ring = p->conv_state; d.channels = static_cast<int>(inner + 2 * gn);
  d.dt_bias = p->dt_bias; d.a_log = p->a_log; d.skip = p->skip; d.norm = p->norm; d.w_dt = p->w_dtype;
  d.heads = p->heads; d.groups = p->groups; d.dim = p->dim; d.vdim = p->vdim; d.inner = static_cast<int>(inner); d.gn = static_cast<int>(gn);
  d.norm_groups = p->norm_groups; d.norm_eps = p->norm_eps;
  d.state = p->state; d.tickets = p->tickets;
  d.u = p->workspace;
  d.xc = d.u + up4(p->rows * inner); d.ld_xc = up4(d.channels);
  d.out = p->out; d.ld_out = p->ld_out; d.out_dt = p->out_dtype;
  cudaStream_t st = static_cast<cudaStream_t>(p->stream);
  const auto al = [](const void* q, long long ld) { return reinterpret_cast<uintptr_t>(q) % 16 == 0 && ld % 4 == 0; };
  // runs of 4 adjacent channels: each belongs to one of x, b, c, and every row of inputs and ring is aligned
  const bool cvec = d.inner % 4 == 0 && d.gn % 4 == 0 && al(d.x, d.ldx) && al(d.b, d.ldb) && al(d.c, d.ldc) && al(d.ring, d.channels);
  if (p->max_new == 1) {
    const bool vec = p->vdim % 4 == 0;
    // several heads of a group per CTA while that still leaves three CTAs for every SM
    const int rep = p->heads / p->groups;
    int hpc = 1;
    while (hpc < SS_H && rep % (2 * hpc) == 0 && static_cast<long long>(p->heads / (2 * hpc)) * p->n_seqs >= 3LL * num_sms()) hpc *= 2;
    const dim3 grid(p->heads / hpc, p->n_seqs);
    const size_t smem = sizeof(float) * ((vec ? 8 : 2) * SS_T + 2 * ((p->dim + 3) / 4 * 4) + 2 * ((hpc * p->vdim + 3) / 4 * 4));
    const bool cvec4 = cvec && (!d.gate || al(d.gate, d.ld_gate)) && p->vdim % 4 == 0 && p->dim % 4 == 0 && reinterpret_cast<uintptr_t>(p->conv_w) % 8 == 0;
    const int q = p->vdim / 4, r = q >= 1 && q <= 32 ? SS_T / q : 0;
    const bool even = cvec4 && q >= 1 && q <= 32 && (q & (q - 1)) == 0;
    const auto go = [&](auto kernel) { return launch_kernel(kernel, grid, dim3(SS_T), smem, st, d, hpc); };
    VY_CUDA_OK(even && p->dim % (16 * r) == 0 ? go(ssd_step_kernel<4, 4, 16>) : even && p->dim % (8 * r) == 0 ? go(ssd_step_kernel<4, 4, 8>)
               : even && p->dim % (4 * r) == 0 ? go(ssd_step_kernel<4, 4, 4>) : cvec4 ? go(ssd_step_kernel<4, 4, 0>) : vec ? go(ssd_step_kernel<4, 1, 0>) : go(ssd_step_kernel<1, 1, 0>));
    VY_LAUNCH_OK();
    count_launch();
    return VY_OK;
  }
  VY_CHECK_ARG((p->max_new + SC_TOK - 1) / SC_TOK <= 65535, "vy_ssd: too many tokens per sequence");
  const int per = SC_T * (cvec ? 4 : 1);
  const dim3 cgrid((d.channels + per - 1) / per, (p->max_new + SC_TOK - 1) / SC_TOK, p->n_seqs);
  if (p->taps <= 4) VY_CUDA_OK(cvec ? launch_kernel(ssd_conv_kernel<4, 4>, cgrid, dim3(SC_T), 0, st, d) : launch_kernel(ssd_conv_kernel<4, 1>, cgrid, dim3(SC_T), 0, st, d));
  else VY_CUDA_OK(cvec ? launch_kernel(ssd_conv_kernel<16, 4>, cgrid, dim3(SC_T), 0, st, d) : launch_kernel(ssd_conv_kernel<16, 1>, cgrid, dim3(SC_T), 0, st, d));
  VY_LAUNCH_OK();
  count_launch();
  RecDev r;
  memset(&r, 0, sizeof(r));
  r.cu = d.cu; r.pos0 = d.pos0; r.slot = d.slot;
  r.v = d.xc; r.ldv = d.ld_xc; r.k = d.xc + inner; r.ldk = d.ld_xc; r.q = d.xc + inner + gn; r.ldq = d.ld_xc; r.in_dt = VY_F32;
  r.dt = d.dt; r.ld_dt = d.ld_dt; r.dt_bias = d.dt_bias; r.a_log = d.a_log; r.a_log_dt = d.w_dt; r.skip = d.skip;
  r.gate = d.gate; r.ld_gate = d.ld_gate; r.gate_act = d.gate_act;
  r.heads = p->heads; r.kv_heads = p->groups; r.dim = p->dim; r.vdim = p->vdim;
  r.state = d.state;
  r.out = d.u; r.ld_out = inner; r.out_dt = VY_F32;
  VY_CUDA_OK(launch_ssd_chunked(r, p->n_seqs, st));
  VY_LAUNCH_OK();
  count_launch();
  VyRmsNorm nm;
  memset(&nm, 0, sizeof(nm));
  nm.tokens = p->rows; nm.groups = p->norm_groups; nm.width = static_cast<int32_t>(inner / p->norm_groups);
  nm.x = d.u; nm.ldx = inner; nm.x_dtype = VY_F32;
  nm.weight = p->norm; nm.w_dtype = p->w_dtype; nm.w_mode = 1; nm.w_full = 1;
  nm.eps = p->norm_eps; nm.coef = 1.f;
  nm.out = p->out; nm.ld_out = p->ld_out; nm.out_dtype = p->out_dtype;
  nm.stream = p->stream;
  return vy_rms_norm(&nm);
}
