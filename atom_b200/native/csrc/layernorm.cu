// Layer norm with weight and bias on the 32-bit residual stream, fused with what is added to the stream before it:
//   LN(x; w, b) = (x - mean(x)) / sqrt(mean((x - mean(x))^2) + eps) * w + b
//   r = residual[row]                                             (delta null)
//   r = residual[row] + dscale * delta[row]                       (wd null)
//   r = residual[row] + dscale * LN(delta[row] (+ dbias); wd, bd, eps_d)      a sub-block whose output passes a norm of
//                                                                 its own before it enters the stream
//   residual[row] = r  (unless rows are picked);   out = LN(r; w, b, eps)
// With `rows` given only those rows are normalised and written densely (the gather of the rows whose logits are
// wanted).  All arithmetic is 32-bit; the variance is the mean of squared deviations, formed in a pass of its own
// over numbers that stay on chip.  delta and out have the activation type.
#include "common.cuh"

namespace atom {

struct LayerNormArgs {
  const void* w;        // [H] weight and bias of the norm that reads the stream
  const void* b;
  int w_dtype;
  float eps;
  const void* wd;       // [H] weight and bias of the norm that delta passes (null: none)
  const void* bd;
  float eps_d;
  const void* dbias;    // [H] added to delta before its norm (null: none); all vectors have type w_dtype
  float dscale;
  const int* rows;
  int H;
};

__device__ __forceinline__ float ln_rstd(float sum_sq_dev, int H, float eps) { return rsqrtf(sum_sq_dev / (float)H + eps); }

// Any size, both precisions; the row's numbers wait in shared memory between the passes.
template <typename TA>
__global__ void add_layernorm_kernel(TA* __restrict__ out, float* __restrict__ residual, const TA* __restrict__ delta,
                                     const LayerNormArgs p) {
  atom::pdl_trigger();
  atom::pdl_wait();
  extern __shared__ float ln_row[];
  __shared__ float scratch[32];
  const int r = blockIdx.x, H = p.H;
  const int64_t src = p.rows ? p.rows[r] : r;
  float* res = residual + src * H;
  const TA* d = delta ? delta + src * H : nullptr;
  float mean_d = 0.f, rstd_d = 1.f;
  const bool normed = d && p.wd;
  if (normed) {
    float s = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
      float v = to_float(d[i]);
      if (p.dbias) v += load_as_float(p.dbias, p.w_dtype, i);
      ln_row[i] = v;
      s += v;
    }
    mean_d = block_sum(s, scratch) / (float)H;
    s = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
      const float v = ln_row[i] - mean_d;
      s = fmaf(v, v, s);
    }
    rstd_d = ln_rstd(block_sum(s, scratch), H, p.eps_d);
  }
  float s = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    float v = res[i];
    if (normed)
      v += p.dscale * ((ln_row[i] - mean_d) * rstd_d * load_as_float(p.wd, p.w_dtype, i) + load_as_float(p.bd, p.w_dtype, i));
    else if (d)
      v += p.dscale * (to_float(d[i]) + (p.dbias ? load_as_float(p.dbias, p.w_dtype, i) : 0.f));
    if (d && !p.rows) res[i] = v;
    ln_row[i] = v;
    s += v;
  }
  const float mean = block_sum(s, scratch) / (float)H;
  s = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    const float v = ln_row[i] - mean;
    s = fmaf(v, v, s);
  }
  const float rstd = ln_rstd(block_sum(s, scratch), H, p.eps);
  TA* o = out + (int64_t)r * H;
  for (int i = threadIdx.x; i < H; i += blockDim.x)
    o[i] = from_float<TA>((ln_row[i] - mean) * rstd * load_as_float(p.w, p.w_dtype, i) + load_as_float(p.b, p.w_dtype, i));
}

__device__ __forceinline__ void ln_load8(const void* w, int dtype, int64_t i, float (&o)[8]) {
  if (dtype == ATOM_F32) {
    const float4 a = *reinterpret_cast<const float4*>((const float*)w + i);
    const float4 b = *reinterpret_cast<const float4*>((const float*)w + i + 4);
    o[0] = a.x; o[1] = a.y; o[2] = a.z; o[3] = a.w; o[4] = b.x; o[5] = b.y; o[6] = b.z; o[7] = b.w;
  } else {
    const uint4 q = *reinterpret_cast<const uint4*>((const __nv_bfloat16*)w + i);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&q);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 f = __bfloat1622float2(h[e]);
      o[2 * e] = f.x;
      o[2 * e + 1] = f.y;
    }
  }
}

// A block's sum with a scratch row of its own for every sum of the kernel, so that one barrier is enough.
__device__ __forceinline__ float block_sum_once(float v, float* scratch) {
  const int lane = threadIdx.x & 31, warps = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  if (lane == 0) scratch[threadIdx.x >> 5] = v;
  __syncthreads();
  return warp_sum(lane < warps ? scratch[lane] : 0.f);
}
// Mean of the row and sum of squared deviations from it.
template <int NV>
__device__ __forceinline__ void row_moments(const float (&v)[NV][8], int H, float* sums, float& mean, float& m2) {
  float s = 0.f;
#pragma unroll
  for (int k = 0; k < NV; ++k)
    if ((int)(threadIdx.x + k * blockDim.x) * 8 < H) {
#pragma unroll
      for (int e = 0; e < 8; ++e) s += v[k][e];
    }
  mean = block_sum_once(s, sums) / (float)H;
  s = 0.f;
#pragma unroll
  for (int k = 0; k < NV; ++k)
    if ((int)(threadIdx.x + k * blockDim.x) * 8 < H) {
#pragma unroll
      for (int e = 0; e < 8; ++e) s = fmaf(v[k][e] - mean, v[k][e] - mean, s);
    }
  m2 = block_sum_once(s, sums + 32);
}

// bfloat16 rows of a multiple of 8 numbers, at most 8 * NV * blockDim: a thread keeps its 8 * NV numbers in registers,
// so that every array is read once and written once, 16 bytes at a time.  A CTA takes row after row; with NV == 1 it keeps
// the weights in registers over its rows, and they are on their way before the wait, since they do not depend on the
// kernel in front of this one.
template <int NV>
__global__ void __launch_bounds__(1024)
add_layernorm_bf16_vec_kernel(__nv_bfloat16* __restrict__ out, float* __restrict__ residual,
                              const __nv_bfloat16* __restrict__ delta, const LayerNormArgs p, int n_rows) {
  atom::pdl_trigger();
  __shared__ float scratch[2][4][32];      // (two rows in turn: a row's sums may still be read when the next begins)
  constexpr bool AHEAD = NV == 1;
  const int H = p.H;
  const bool normed = delta && p.wd;
  float w1[8], b1[8], w2[8], b2[8];
  if (AHEAD && threadIdx.x * 8 < H) {
    if (normed) {
      ln_load8(p.wd, p.w_dtype, threadIdx.x * 8, w1);
      ln_load8(p.bd, p.w_dtype, threadIdx.x * 8, b1);
    }
    ln_load8(p.w, p.w_dtype, threadIdx.x * 8, w2);
    ln_load8(p.b, p.w_dtype, threadIdx.x * 8, b2);
  }
  atom::pdl_wait();
  for (int r = blockIdx.x, odd = 0; r < n_rows; r += gridDim.x, odd ^= 1) {
    float(*sums)[32] = scratch[odd];
    const int64_t src = p.rows ? p.rows[r] : r;
    float* res = residual + src * H;
    float v[NV][8], rv[NV][8];
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8;
      if (i < H) {
        ln_load8(res, ATOM_F32, i, rv[k]);
        if (delta) {
          ln_load8(delta, ATOM_BF16, src * H + i, v[k]);
          if (p.dbias) {
            float bv[8];
            ln_load8(p.dbias, p.w_dtype, i, bv);
#pragma unroll
            for (int e = 0; e < 8; ++e) v[k][e] += bv[e];
          }
        }
      }
    }
    if (normed) {
      float mean, m2;
      row_moments<NV>(v, H, sums[0], mean, m2);
      const float rstd = ln_rstd(m2, H, p.eps_d);
#pragma unroll
      for (int k = 0; k < NV; ++k) {
        const int i = (threadIdx.x + k * blockDim.x) * 8;
        if (i < H) {
          if (!AHEAD) {
            ln_load8(p.wd, p.w_dtype, i, w1);
            ln_load8(p.bd, p.w_dtype, i, b1);
          }
#pragma unroll
          for (int e = 0; e < 8; ++e) v[k][e] = (v[k][e] - mean) * rstd * w1[e] + b1[e];
        }
      }
    }
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8;
      if (i < H && delta) {
#pragma unroll
        for (int e = 0; e < 8; ++e) rv[k][e] += p.dscale * v[k][e];
        if (!p.rows) {
          *reinterpret_cast<float4*>(res + i) = make_float4(rv[k][0], rv[k][1], rv[k][2], rv[k][3]);
          *reinterpret_cast<float4*>(res + i + 4) = make_float4(rv[k][4], rv[k][5], rv[k][6], rv[k][7]);
        }
      }
    }
    float mean, m2;
    row_moments<NV>(rv, H, sums[2], mean, m2);
    const float rstd = ln_rstd(m2, H, p.eps);
    __nv_bfloat16* o = out + (int64_t)r * H;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int i = (threadIdx.x + k * blockDim.x) * 8;
      if (i < H) {
        if (!AHEAD) {
          ln_load8(p.w, p.w_dtype, i, w2);
          ln_load8(p.b, p.w_dtype, i, b2);
        }
        uint4 q;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&q);
#pragma unroll
        for (int e = 0; e < 4; ++e)
          h[e] = __floats2bfloat162_rn((rv[k][2 * e] - mean) * rstd * w2[2 * e] + b2[2 * e],
                                       (rv[k][2 * e + 1] - mean) * rstd * w2[2 * e + 1] + b2[2 * e + 1]);
        *reinterpret_cast<uint4*>(o + i) = q;
      }
    }
  }
}

// y = LN(x (+ xbias); w, b) of dense rows of the activation type.
template <typename TA>
__global__ void layernorm_kernel(TA* __restrict__ y, const TA* __restrict__ x, const void* __restrict__ xbias,
                                 const void* __restrict__ w, const void* __restrict__ b, int w_dtype, float eps, int H) {
  atom::pdl_trigger();
  atom::pdl_wait();
  extern __shared__ float ln_row[];
  __shared__ float scratch[32];
  const TA* xr = x + (int64_t)blockIdx.x * H;
  float s = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    const float v = to_float(xr[i]) + (xbias ? load_as_float(xbias, w_dtype, i) : 0.f);
    ln_row[i] = v;
    s += v;
  }
  const float mean = block_sum(s, scratch) / (float)H;
  s = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    const float v = ln_row[i] - mean;
    s = fmaf(v, v, s);
  }
  const float rstd = ln_rstd(block_sum(s, scratch), H, eps);
  TA* yr = y + (int64_t)blockIdx.x * H;
  for (int i = threadIdx.x; i < H; i += blockDim.x)
    yr[i] = from_float<TA>((ln_row[i] - mean) * rstd * load_as_float(w, w_dtype, i) + load_as_float(b, w_dtype, i));
}

static inline int ln_threads(int H) { return H >= 2048 ? 512 : (H >= 512 ? 256 : 128); }
constexpr int kLnMaxRow = 12 * 1024 - 64;      // a row waits in shared memory, beside the reductions' numbers

}  // namespace atom

// The vectors w, b, wd, bd, dbias have one type (w_dtype).
ATOM_EXPORT int atom_add_layernorm(void* out, int act_dtype, float* residual, const void* delta, const void* dbias,
                                   const void* wd, const void* bd, float eps_d, float dscale, const void* w,
                                   const void* b, int w_dtype, float eps, const int* rows, int n_rows, int H,
                                   cudaStream_t stream) {
  using namespace atom;
  if (n_rows <= 0) return ATOM_OK;
  if (H <= 0 || !w || !b || (wd && !bd) || (w_dtype != ATOM_F32 && w_dtype != ATOM_BF16)) return ATOM_ERR_ARG;
  LayerNormArgs p{w, b, w_dtype, eps, wd, bd, eps_d, dbias, dscale, rows, H};
  auto al = [](const void* q) { return ((uintptr_t)q % 16) == 0; };
  if (act_dtype == ATOM_BF16 && H % 8 == 0 && H <= 8 * 2 * 1024 && al(out) && al(residual) && al(delta) && al(w) && al(b) && al(wd) && al(bd) &&
      al(dbias)) {
    const int vecs = H / 8;
    auto threads = [&](int nv) { return (((vecs + nv - 1) / nv + 31) / 32) * 32; };
    const int nv = vecs <= 1024 ? 1 : 2, th = threads(nv);
    const int grid = min(n_rows, 148 * max(1, 1024 / th));      // (64 registers a thread)
    if (nv == 1)
      launch_pdl(add_layernorm_bf16_vec_kernel<1>, dim3(grid), dim3(th), 0, stream, (__nv_bfloat16*)out, residual,
                 (const __nv_bfloat16*)delta, p, n_rows);
    else
      launch_pdl(add_layernorm_bf16_vec_kernel<2>, dim3(grid), dim3(th), 0, stream, (__nv_bfloat16*)out, residual,
                 (const __nv_bfloat16*)delta, p, n_rows);
    return check_launch();
  }
  if (H > kLnMaxRow) return ATOM_ERR_ARG;
  const size_t smem = sizeof(float) * (size_t)H;
  if (act_dtype == ATOM_F32)
    launch_pdl(add_layernorm_kernel<float>, dim3(n_rows), dim3(ln_threads(H)), smem, stream, (float*)out, residual,
               (const float*)delta, p);
  else if (act_dtype == ATOM_BF16)
    launch_pdl(add_layernorm_kernel<__nv_bfloat16>, dim3(n_rows), dim3(ln_threads(H)), smem, stream, (__nv_bfloat16*)out,
               residual, (const __nv_bfloat16*)delta, p);
  else
    return ATOM_ERR_ARG;
  return check_launch();
}

ATOM_EXPORT int atom_layernorm(void* y, const void* x, int act_dtype, const void* xbias, const void* w, const void* b,
                               int w_dtype, float eps, int n_rows, int H, cudaStream_t stream) {
  using namespace atom;
  if (n_rows <= 0) return ATOM_OK;
  if (H <= 0 || H > kLnMaxRow || (w_dtype != ATOM_F32 && w_dtype != ATOM_BF16)) return ATOM_ERR_ARG;
  const size_t smem = sizeof(float) * (size_t)H;
  if (act_dtype == ATOM_F32)
    launch_pdl(layernorm_kernel<float>, dim3(n_rows), dim3(ln_threads(H)), smem, stream, (float*)y, (const float*)x, xbias,
               w, b, w_dtype, eps, H);
  else if (act_dtype == ATOM_BF16)
    launch_pdl(layernorm_kernel<__nv_bfloat16>, dim3(n_rows), dim3(ln_threads(H)), smem, stream, (__nv_bfloat16*)y,
               (const __nv_bfloat16*)x, xbias, w, b, w_dtype, eps, H);
  else
    return ATOM_ERR_ARG;
  return check_launch();
}
