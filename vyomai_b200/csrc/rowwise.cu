// Row-wise pieces over packed rows. vy_sandwich_norm: a sublayer's result normed, added to the residual, and the sum normed for the next
// sublayer (values in registers between the passes). vy_glu: the gated feed-forward's activation. vy_poly_norm: a polynomial of the row's normalised powers,
//   out = a N(z) + b N(z^2) + c3 N(z^3) + e,   N(u) = u / sqrt(mean(u^2) + eps) over the row,
// with all statistics and the polynomial in fp32. One CTA per row: the row is read once into shared memory while the sums of
// z^2, z^4 and z^6 are taken, then written from there.
#include <math.h>

#include "seqmix.cuh"

namespace vy {

struct PolyDev {
  long long rows; int width;
  const void* x; long long ldx; int x_dt;
  float a, b, c3, e, eps;
  void* out; long long ld_out; int out_dt;
};

template <int T>
__global__ void __launch_bounds__(T) poly_norm_kernel(PolyDev d) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ __align__(16) float pn_row[];
  __shared__ float part[3][T / 32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (long long r = blockIdx.x; r < d.rows; r += gridDim.x) {
    const long long xo = r * d.ldx;
    float s2 = 0.f, s4 = 0.f, s6 = 0.f;
    for (int c = threadIdx.x; c < d.width; c += T) {
      const float z = ld_as_float(d.x, d.x_dt, xo + c);
      pn_row[c] = z;
      const float z2 = z * z, z4 = z2 * z2;
      s2 += z2;
      s4 += z4;
      s6 = fmaf(z4, z2, s6);
    }
    s2 = warp_sum(s2);
    s4 = warp_sum(s4);
    s6 = warp_sum(s6);
    __syncthreads();   // the previous row's readers of `part` are done
    if (lane == 0) { part[0][warp] = s2; part[1][warp] = s4; part[2][warp] = s6; }
    __syncthreads();
    s2 = s4 = s6 = 0.f;
#pragma unroll
    for (int w = 0; w < T / 32; ++w) { s2 += part[0][w]; s4 += part[1][w]; s6 += part[2][w]; }
    const float n = static_cast<float>(d.width);
    const float k1 = d.a / sqrtf(s2 / n + d.eps), k2 = d.b / sqrtf(s4 / n + d.eps), k3 = d.c3 / sqrtf(s6 / n + d.eps);
    const long long oo = r * d.ld_out;
    for (int c = threadIdx.x; c < d.width; c += T) {
      const float z = pn_row[c];
      st_from_float(d.out, d.out_dt, oo + c, fmaf(z, fmaf(z, fmaf(z, k3, k2), k1), d.e));
    }
  }
}

// ---- sandwich norm ----------------------------------------------------------------------------------------------------------
struct SandDev {
  long long rows; int width;
  const int* row_index;
  const float* x; long long ldx; const float* y; long long ldy;
  const void* w1; const void* b1; const void* w2; const void* b2; int w_dt;
  int kind;   // VY_CLOSE_LAYER, or RMS norms with the weight as it is / stored around zero
  const void* u; long long ld_u; int u_dt; const float* u_coef;   // y + u_coef[row] * u is what is normed (u null: y)
  float eps;
  float* xo; long long ld_xo;
  void* copy; long long ld_copy; int copy_dt;
  void* out; long long ld_out; int out_dt;
};

// sum over the TPR threads of a row (a warp, or whole warps of the CTA: every thread of the CTA takes part)
template <int TPR>
__device__ __forceinline__ float row_sum(float v, float* part, int lr, int lt) {
  v = warp_sum(v);
  if constexpr (TPR > 32) {
    __syncthreads();   // part may still be read from the previous reduction
    if ((lt & 31) == 0) part[lr * (TPR / 32) + (lt >> 5)] = v;
    __syncthreads();
    v = 0.f;
#pragma unroll
    for (int w = 0; w < TPR / 32; ++w) v += part[lr * (TPR / 32) + w];
  }
  return v;
}

// v <- layer norm (or RMS norm, d.kind) of the row's values (entries past the width stay out of the statistics)
template <int TPR, int NC, bool VEC>
__device__ __forceinline__ void norm_row(float (&v)[NC], const SandDev& d, const void* w, const void* b, float* part, int lr, int lt) {
  auto col = [&](int i) { return VEC ? 4 * lt + (i >> 2) * 4 * TPR + (i & 3) : lt + i * TPR; };
  float mean = 0.f;
  if (d.kind == VY_CLOSE_LAYER) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NC; ++i) s += v[i];
    mean = row_sum<TPR>(s, part, lr, lt) / static_cast<float>(d.width);
  }
  const float w_add = d.kind == VY_CLOSE_RMS_CENTRED ? 1.f : 0.f;
  float q = 0.f;
#pragma unroll
  for (int i = 0; i < NC; ++i) {
    const float u = col(i) < d.width ? v[i] - mean : 0.f;
    v[i] = u;
    q = fmaf(u, u, q);
  }
  const float inv = 1.f / sqrtf(row_sum<TPR>(q, part, lr, lt) / static_cast<float>(d.width) + d.eps);
  if (VEC && d.w_dt == VY_BF16 && w && b) {   // four adjacent columns: one 8-byte load of each
#pragma unroll
    for (int i = 0; i < NC; i += 4) {
      if (col(i) >= d.width) continue;
      const uint2 wr = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(w) + col(i));
      const uint2 br = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(b) + col(i));
      const __nv_bfloat162* wp = reinterpret_cast<const __nv_bfloat162*>(&wr);
      const __nv_bfloat162* bp = reinterpret_cast<const __nv_bfloat162*>(&br);
      const float2 w0 = __bfloat1622float2(wp[0]), w1 = __bfloat1622float2(wp[1]), b0 = __bfloat1622float2(bp[0]), b1 = __bfloat1622float2(bp[1]);
      v[i] = fmaf(v[i] * inv, w0.x, b0.x);
      v[i + 1] = fmaf(v[i + 1] * inv, w0.y, b0.y);
      v[i + 2] = fmaf(v[i + 2] * inv, w1.x, b1.x);
      v[i + 3] = fmaf(v[i + 3] * inv, w1.y, b1.y);
    }
  } else if (VEC && d.w_dt == VY_BF16 && w) {
#pragma unroll
    for (int i = 0; i < NC; i += 4) {
      if (col(i) >= d.width) continue;
      const uint2 wr = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(w) + col(i));
      const __nv_bfloat162* wp = reinterpret_cast<const __nv_bfloat162*>(&wr);
      const float2 w0 = __bfloat1622float2(wp[0]), w1 = __bfloat1622float2(wp[1]);
      v[i] *= inv * (w_add + w0.x);
      v[i + 1] *= inv * (w_add + w0.y);
      v[i + 2] *= inv * (w_add + w1.x);
      v[i + 3] *= inv * (w_add + w1.y);
      if (b)
#pragma unroll
        for (int e = 0; e < 4; ++e) v[i + e] += ld_as_float(b, d.w_dt, col(i) + e);
    }
  } else {
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = col(i);
      if (c >= d.width) continue;
      float z = v[i] * inv;
      if (w) z *= w_add + ld_as_float(w, d.w_dt, c);
      if (b) z += ld_as_float(b, d.w_dt, c);
      v[i] = z;
    }
  }
}

template <int TPR, int NC, bool VEC>
__device__ __forceinline__ void store_row(void* p, int dt, long long o, const float (&v)[NC], int width, int lt) {
  if constexpr (VEC) {
#pragma unroll
    for (int i = 0; i < NC; i += 4) {
      const int c = 4 * lt + (i >> 2) * 4 * TPR;
      if (c >= width) continue;
      if (dt == VY_F32) *reinterpret_cast<float4*>(reinterpret_cast<float*>(p) + o + c) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
      else {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(v[i], v[i + 1]), hi = __floats2bfloat162_rn(v[i + 2], v[i + 3]);
        uint2 pk;
        pk.x = *reinterpret_cast<const unsigned*>(&lo);
        pk.y = *reinterpret_cast<const unsigned*>(&hi);
        *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(p) + o + c) = pk;
      }
    }
  } else {
#pragma unroll
    for (int i = 0; i < NC; ++i)
      if (lt + i * TPR < width) st_from_float(p, dt, o + lt + i * TPR, v[i]);
  }
}

// TPR threads per row; VEC: 16-byte accesses (4 adjacent columns per group)
template <int TPR, int NC, bool VEC>
__global__ void __launch_bounds__(TPR < 256 ? 256 : TPR) sandwich_norm_kernel(SandDev d) {
  pdl_trigger();
  pdl_wait();
  constexpr int RPB = TPR < 256 ? 256 / TPR : 1;
  __shared__ float part[RPB * (TPR / 32)];
  const int lr = threadIdx.x / TPR, lt = threadIdx.x % TPR;
  const long long r = static_cast<long long>(blockIdx.x) * RPB + lr;
  const bool live = r < d.rows;
  const long long st = live ? (d.row_index ? d.row_index[r] : r) : 0;
  auto load = [&](const float* p, float (&v)[NC]) {
#pragma unroll
    for (int i = 0; i < NC; i += (VEC ? 4 : 1)) {
      if constexpr (VEC) {
        const int c = 4 * lt + (i >> 2) * 4 * TPR;
        float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
        if (live && c < d.width) f = *reinterpret_cast<const float4*>(p + c);
        v[i] = f.x; v[i + 1] = f.y; v[i + 2] = f.z; v[i + 3] = f.w;
      } else {
        const int c = lt + i * TPR;
        v[i] = live && c < d.width ? p[c] : 0.f;
      }
    }
  };
  float xv[NC], yv[NC];
  load(d.x + st * d.ldx, xv);
  if (d.y) {
    load(d.y + st * d.ldy, yv);
    if (d.u) {
      const float uc = live ? d.u_coef[st] : 0.f;
      if (uc != 0.f) {   // a zero weight leaves the row unread
#pragma unroll
        for (int i = 0; i < NC; ++i) {
          const int c = VEC ? 4 * lt + (i >> 2) * 4 * TPR + (i & 3) : lt + i * TPR;
          if (c < d.width) yv[i] = fmaf(uc, ld_as_float(d.u, d.u_dt, st * d.ld_u + c), yv[i]);
        }
      }
    }
    norm_row<TPR, NC, VEC>(yv, d, d.w1, d.b1, part, lr, lt);
#pragma unroll
    for (int i = 0; i < NC; ++i) xv[i] += yv[i];
  }
  if (live && d.xo) store_row<TPR, NC, VEC>(d.xo, VY_F32, r * d.ld_xo, xv, d.width, lt);
  if (live && d.copy) store_row<TPR, NC, VEC>(d.copy, d.copy_dt, r * d.ld_copy, xv, d.width, lt);
  if (!d.out) return;
  norm_row<TPR, NC, VEC>(xv, d, d.w2, d.b2, part, lr, lt);
  if (live) store_row<TPR, NC, VEC>(d.out, d.out_dt, r * d.ld_out, xv, d.width, lt);
}

template <int TPR, int NC>
static cudaError_t launch_sandwich(const SandDev& d, bool vec, cudaStream_t st) {
  constexpr int RPB = TPR < 256 ? 256 / TPR : 1;
  const dim3 grid(static_cast<unsigned>((d.rows + RPB - 1) / RPB)), block(TPR < 256 ? 256 : TPR);
  return vec ? launch_kernel(sandwich_norm_kernel<TPR, NC, true>, grid, block, 0, st, d) : launch_kernel(sandwich_norm_kernel<TPR, NC, false>, grid, block, 0, st, d);
}

// ---- gated activation over interleaved columns ---------------------------------------------------------------------------------
template <bool VEC>
__global__ void __launch_bounds__(256) glu_kernel(long long rows, int ff, const void* x, long long ldx, int x_dt, int act, void* out, long long ld_out, int out_dt) {
  pdl_trigger();
  pdl_wait();
  const long long r = blockIdx.x;
  if (VEC) {   // four outputs per thread from 8 adjacent columns
    for (int c = (blockIdx.y * 256 + threadIdx.x) * 4; c < ff; c += gridDim.y * 1024) {
      float z[8], y[4];
      ld8_as_float(x, x_dt, r * ldx + 2 * c, z);
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] = apply_uact(z[2 * e], act) * z[2 * e + 1];
      if (out_dt == VY_F32) *reinterpret_cast<float4*>(reinterpret_cast<float*>(out) + r * ld_out + c) = make_float4(y[0], y[1], y[2], y[3]);
      else {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(y[0], y[1]), hi = __floats2bfloat162_rn(y[2], y[3]);
        uint2 pk;
        pk.x = *reinterpret_cast<const unsigned*>(&lo);
        pk.y = *reinterpret_cast<const unsigned*>(&hi);
        *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(out) + r * ld_out + c) = pk;
      }
    }
    return;
  }
  for (int c = blockIdx.y * 256 + threadIdx.x; c < ff; c += gridDim.y * 256)
    st_from_float(out, out_dt, r * ld_out + c, apply_uact(ld_as_float(x, x_dt, r * ldx + 2 * c), act) * ld_as_float(x, x_dt, r * ldx + 2 * c + 1));
}

}  // namespace vy

#define VY_NEED_DEVICE(name)                                                   \
  if (!vy_device_ok()) {                                                       \
    ::vy::set_error(name ": no sm_100 device (there is no CPU fallback)");     \
    return VY_ERR_NO_DEVICE;                                                   \
  }

extern "C" int vy_poly_norm(const VyPolyNorm* p) {
  using namespace vy;
  VY_CHECK_ARG(p != nullptr, "vy_poly_norm: null params");
  VY_NEED_DEVICE("vy_poly_norm");
  VY_CHECK_ARG(p->rows > 0 && p->width > 0 && p->width <= 49152, "vy_poly_norm: rows %lld, width %d (<= 49152)", static_cast<long long>(p->rows), p->width);
  VY_CHECK_ARG(p->x && p->out && dtype_ok(p->x_dtype) && dtype_ok(p->out_dtype), "vy_poly_norm: bad tensors");
  PolyDev d;
  d.rows = p->rows; d.width = p->width;
  d.x = p->x; d.ldx = p->ldx; d.x_dt = p->x_dtype;
  d.a = p->a; d.b = p->b; d.c3 = p->c3; d.e = p->e; d.eps = p->eps;
  d.out = p->out; d.ld_out = p->ld_out; d.out_dt = p->out_dtype;
  const size_t smem = sizeof(float) * p->width;
  cudaStream_t st = static_cast<cudaStream_t>(p->stream);
  const unsigned blocks = static_cast<unsigned>(p->rows < 1048576 ? p->rows : 1048576);
  if (p->width <= 1024) {
    VY_CUDA_OK(launch_kernel(poly_norm_kernel<128>, dim3(blocks), dim3(128), smem, st, d));
  } else {
    static size_t allowed = 48 * 1024;
    if (smem > allowed) {
      VY_CUDA_OK(cudaFuncSetAttribute(poly_norm_kernel<512>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
      allowed = smem;
    }
    VY_CUDA_OK(launch_kernel(poly_norm_kernel<512>, dim3(blocks), dim3(512), smem, st, d));
  }
  VY_LAUNCH_OK();
  count_launch();
  return VY_OK;
}

extern "C" int vy_sandwich_norm(const VySandwichNorm* p) {
  using namespace vy;
  VY_CHECK_ARG(p != nullptr, "vy_sandwich_norm: null params");
  VY_NEED_DEVICE("vy_sandwich_norm");
  VY_CHECK_ARG(p->rows > 0 && p->rows <= 2147483647LL && p->width > 0 && p->width <= 16384, "vy_sandwich_norm: rows %lld, width %d (<= 16384)",
               static_cast<long long>(p->rows), p->width);
  VY_CHECK_ARG(p->x && (p->x_out || p->copy || p->out) && ((!p->w1 && !p->b1 && !p->w2 && !p->b2) || dtype_ok(p->w_dtype)) && (!p->copy || dtype_ok(p->copy_dtype)) &&
                   (!p->out || dtype_ok(p->out_dtype)), "vy_sandwich_norm: bad tensors");
  VY_CHECK_ARG(!p->row_index || p->x_out != p->x, "vy_sandwich_norm: gathered rows do not go back in place");
  SandDev d;
  d.rows = p->rows; d.width = p->width; d.row_index = p->row_index;
  d.x = p->x; d.ldx = p->ldx; d.y = p->y; d.ldy = p->ldy;
  d.w1 = p->w1; d.b1 = p->b1; d.w2 = p->w2; d.b2 = p->b2; d.w_dt = p->w_dtype; d.eps = p->eps;
  VY_CHECK_ARG(p->norm_kind >= VY_CLOSE_LAYER && p->norm_kind <= VY_CLOSE_RMS_CENTRED && (p->norm_kind == VY_CLOSE_LAYER || (!p->b1 && !p->b2)),
               "vy_sandwich_norm: norm kind %d (RMS norms take no bias)", p->norm_kind);
  VY_CHECK_ARG(!p->u || (p->y && p->u_coef && dtype_ok(p->u_dtype)), "vy_sandwich_norm: a second result needs the first, its dtype and its weights");
  d.kind = p->norm_kind;
  d.u = p->u; d.ld_u = p->ld_u; d.u_dt = p->u_dtype; d.u_coef = p->u_coef;
  d.xo = p->x_out; d.ld_xo = p->ld_x_out;
  d.copy = p->copy; d.ld_copy = p->ld_copy; d.copy_dt = p->copy_dtype;
  d.out = p->out; d.ld_out = p->ld_out; d.out_dt = p->out_dtype;
  const auto ok = [](const void* q, long long ld, int dt) { return !q || (ld % 4 == 0 && reinterpret_cast<uintptr_t>(q) % (dt == VY_F32 ? 16 : 8) == 0); };
  const auto okw = [&](const void* q) { return ok(q, 0, p->w_dtype); };
  const bool vec = p->width % 4 == 0 && ok(p->x, p->ldx, VY_F32) && ok(p->y, p->ldy, VY_F32) && ok(p->x_out, p->ld_x_out, VY_F32) &&
                   ok(p->copy, p->ld_copy, p->copy_dtype) && ok(p->out, p->ld_out, p->out_dtype) && okw(p->w1) && okw(p->b1) && okw(p->w2) && okw(p->b2);
  cudaStream_t st = static_cast<cudaStream_t>(p->stream);
  cudaError_t e;
  if (p->width <= 256) e = launch_sandwich<32, 8>(d, vec, st);
  else if (p->width <= 1024) e = launch_sandwich<128, 8>(d, vec, st);
  else if (p->width <= 2048) e = launch_sandwich<256, 8>(d, vec, st);
  else if (p->width <= 4096) e = launch_sandwich<512, 8>(d, vec, st);
  else if (p->width <= 8192) e = launch_sandwich<1024, 8>(d, vec, st);
  else e = launch_sandwich<1024, 16>(d, vec, st);
  VY_CUDA_OK(e);
  VY_LAUNCH_OK();
  count_launch();
  return VY_OK;
}

extern "C" int vy_glu(int64_t rows, int32_t ff, const void* x, int64_t ldx, int32_t x_dtype, int32_t act, void* out, int64_t ld_out, int32_t out_dtype,
                      void* stream) {
  using namespace vy;
  VY_NEED_DEVICE("vy_glu");
  VY_CHECK_ARG(rows > 0 && rows <= 2147483647LL && ff > 0 && ff <= (1 << 29) && x && out && dtype_ok(x_dtype) && dtype_ok(out_dtype), "vy_glu: bad arguments");
  const auto al = [](const void* q, size_t a) { return reinterpret_cast<uintptr_t>(q) % a == 0; };
  const bool vec = ff % 4 == 0 && ldx % 8 == 0 && ld_out % 4 == 0 && al(x, 16) && al(out, out_dtype == VY_F32 ? 16 : 8);
  const int per = vec ? 1024 : 256;
  int gy = (ff + per - 1) / per;
  if (gy > 64) gy = 64;
  const dim3 grid(static_cast<unsigned>(rows), gy);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  VY_CUDA_OK(vec ? launch_kernel(glu_kernel<true>, grid, dim3(256), 0, st, rows, ff, x, ldx, x_dtype, act, out, ld_out, out_dtype)
                 : launch_kernel(glu_kernel<false>, grid, dim3(256), 0, st, rows, ff, x, ldx, x_dtype, act, out, ld_out, out_dtype));
  VY_LAUNCH_OK();
  count_launch();
  return VY_OK;
}
