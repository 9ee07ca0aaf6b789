// Dynamic tanh (Zhu et al. 2025, "Transformers without Normalization") on the 32-bit residual stream, fused with what is
// added to the stream before it:
//   r = residual[row] (+ d0[row]) (+ d1[row]);   residual[row] = r  (unless rows are picked)
//   out = tanh(alpha * r) * w + b
// d0 and d1 are the outputs of two sub-blocks that run side by side (either may be null).  With `rows` given only those
// rows are read and written densely (the gather of the rows whose logits are wanted).  All arithmetic is 32-bit; d0, d1
// and out have the activation type, w and b a type of their own.
#include "common.cuh"

namespace atom {

struct DynamicTanhArgs {
  const void* w;
  const void* b;
  int w_dtype;
  float alpha;
  const int* rows;
  int H;
};

template <typename TA>
__global__ void add_dynamic_tanh_kernel(TA* __restrict__ out, float* __restrict__ residual, const TA* __restrict__ d0,
                                        const TA* __restrict__ d1, const DynamicTanhArgs p) {
  atom::pdl_trigger();
  atom::pdl_wait();
  const int r = blockIdx.x, H = p.H;
  const int64_t src = (int64_t)(p.rows ? p.rows[r] : r) * H;
  for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < H; i += gridDim.y * blockDim.x) {
    float v = residual[src + i];
    if (d0) v += to_float(d0[src + i]);
    if (d1) v += to_float(d1[src + i]);
    if ((d0 || d1) && !p.rows) residual[src + i] = v;
    out[(int64_t)r * H + i] =
        from_float<TA>(fmaf(tanhf(p.alpha * v), load_as_float(p.w, p.w_dtype, i), load_as_float(p.b, p.w_dtype, i)));
  }
}

__device__ __forceinline__ void dyt_load8(const __nv_bfloat16* p, float (&o)[8]) {
  const uint4 q = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&q);
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const float2 f = __bfloat1622float2(h[e]);
    o[2 * e] = f.x;
    o[2 * e + 1] = f.y;
  }
}

// bfloat16 activations and weights, H in steps of 8: a thread 8 numbers, 16 bytes at a time.
__global__ void __launch_bounds__(128)
add_dynamic_tanh_vec_kernel(__nv_bfloat16* __restrict__ out, float* __restrict__ residual,
                            const __nv_bfloat16* __restrict__ d0, const __nv_bfloat16* __restrict__ d1,
                            const DynamicTanhArgs p) {
  atom::pdl_trigger();
  const int H = p.H;
  const int i = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
  float w[8], b[8];
  if (i < H) {                                         // (weights: nothing of the step writes them)
    dyt_load8((const __nv_bfloat16*)p.w + i, w);
    dyt_load8((const __nv_bfloat16*)p.b + i, b);
  }
  atom::pdl_wait();
  if (i >= H) return;
  const int r = blockIdx.x;
  const int64_t src = (int64_t)(p.rows ? p.rows[r] : r) * H + i;
  float v[8];
  const float4 lo = *reinterpret_cast<const float4*>(residual + src);
  const float4 hi = *reinterpret_cast<const float4*>(residual + src + 4);
  v[0] = lo.x; v[1] = lo.y; v[2] = lo.z; v[3] = lo.w; v[4] = hi.x; v[5] = hi.y; v[6] = hi.z; v[7] = hi.w;
  if (d0) {
    float d[8];
    dyt_load8(d0 + src, d);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] += d[e];
  }
  if (d1) {
    float d[8];
    dyt_load8(d1 + src, d);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] += d[e];
  }
  if ((d0 || d1) && !p.rows) {
    *reinterpret_cast<float4*>(residual + src) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(residual + src + 4) = make_float4(v[4], v[5], v[6], v[7]);
  }
  uint4 packed;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&packed);
#pragma unroll
  for (int e = 0; e < 4; ++e)
    h[e] = __floats2bfloat162_rn(fmaf(tanhf(p.alpha * v[2 * e]), w[2 * e], b[2 * e]),
                                 fmaf(tanhf(p.alpha * v[2 * e + 1]), w[2 * e + 1], b[2 * e + 1]));
  *reinterpret_cast<uint4*>(out + (int64_t)r * H + i) = packed;
}

}  // namespace atom

ATOM_EXPORT int atom_add_dynamic_tanh(void* out, int dtype, float* residual, const void* d0, const void* d1, const void* w,
                                      const void* b, int w_dtype, float alpha, const int* rows, int n, int H,
                                      cudaStream_t stream) {
  if (n <= 0) return ATOM_OK;
  if (H <= 0 || (w_dtype != ATOM_F32 && w_dtype != ATOM_BF16)) return ATOM_ERR_ARG;
  const atom::DynamicTanhArgs p{w, b, w_dtype, alpha, rows, H};
  const uintptr_t all = (uintptr_t)out | (uintptr_t)residual | (uintptr_t)d0 | (uintptr_t)d1 | (uintptr_t)w | (uintptr_t)b;
  if (dtype == ATOM_BF16 && w_dtype == ATOM_BF16 && H % 8 == 0 && (all % 16) == 0) {
    const int groups = H / 8;
    const int threads = groups >= 128 ? 128 : ((groups + 31) / 32) * 32;
    atom::launch_pdl(atom::add_dynamic_tanh_vec_kernel, dim3(n, (groups + threads - 1) / threads), dim3(threads), 0, stream,
                     (__nv_bfloat16*)out, residual, (const __nv_bfloat16*)d0, (const __nv_bfloat16*)d1, p);
    return atom::check_launch();
  }
  const int cols = (H + 255) / 256;
  const dim3 grid(n, cols > 64 ? 64 : cols);
  if (dtype == ATOM_F32)
    atom::launch_pdl(atom::add_dynamic_tanh_kernel<float>, grid, dim3(256), 0, stream, (float*)out, residual,
                     (const float*)d0, (const float*)d1, p);
  else if (dtype == ATOM_BF16)
    atom::launch_pdl(atom::add_dynamic_tanh_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, (__nv_bfloat16*)out, residual,
                     (const __nv_bfloat16*)d0, (const __nv_bfloat16*)d1, p);
  else
    return ATOM_ERR_ARG;
  return atom::check_launch();
}
