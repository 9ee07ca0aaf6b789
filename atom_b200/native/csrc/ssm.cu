// State-space duality (Mamba-2): a matrix state per head with one decay per head and token.
//
//   ssm_conv_kernel       [x | B | C]: y_t[c] = silu(sum_j w[c, j] * u_(t - taps + 1 + j)[c] + b[c]), with rows before the
//                         step's first token of a request from the request's convolution state (its last taps - 1
//                         projected rows), which the same kernel brings up to date (up to 8 taps; more: the state is
//                         updated by conv_state_update_kernel afterwards).  A thread owns two channels over a strip of
//                         16 rows of one request; the strip of a request's first rows holds all rows that read the
//                         state, so the thread that read it may write it.
//                         The blocks of the last grid row do the work of ssm_step_kernel for the strip's rows.
//   ssm_step_kernel       dt = softplus(raw + dt_bias), la = -exp(A_log) * dt   per (token, head), 32-bit
//   ssm_scan_kernel       S_t = exp(la_t) S_(t-1) + dt_t B_t x_t^T;   y_t = S_t^T C_t + D x_t
//   ssm_gate_norm_kernel  y <- (y * silu(z)) / rms over each of `parts` equal parts * w (* a constant)
// State, decays, dt and every sum are 32-bit.  Head h reads B and C of group h / (heads / groups).
//
// The scan: every column of the state runs by itself, so a CTA owns (a run of a request's rows, a head, 32 value
// columns): a thread holds a quarter of one column's N numbers in registers, the four quarters of a column sit in
// neighbouring lanes.  The recurrence is linear in S, so a request's rows are cut into runs of `run` rows:
//   mode 1  every run from S = 0: its sum, and the logarithm of the product of its decays, to scratch
//   prefix  per request and state element, over the runs in order: the scratch takes the state the run begins with, the
//           slot the state after the step
//   mode 2  every run from its beginning: the outputs
// and a step of few rows walks each request once (mode 0: slot in, outputs, slot out).
// (ssm_tc.cu: the runs' sums and outputs on the tensor cores, for bfloat16.)
#include "common.cuh"

namespace atom {

constexpr int kSsmThreads = 128;
constexpr int kSsmCols = 32;       // value columns per CTA
constexpr int kSsmStage = 16;      // rows staged in shared memory at a time
constexpr int kSsmStrip = 16;      // rows of a convolution strip

// Run slot x -> request and run: requests take ceil(len / run) slots one after another.
__device__ __forceinline__ bool ssm_find_run(int x, const int* __restrict__ cu_q, int num_seqs, int run, int& s, int& r) {
  int acc = 0;
  for (s = 0; s < num_seqs; ++s) {
    const int n_runs = (cu_q[s + 1] - cu_q[s] + run - 1) / run;
    if (x < acc + n_runs) {
      r = x - acc;
      return true;
    }
    acc += n_runs;
  }
  return false;
}

__device__ __forceinline__ float ssm_silu(float z) { return z / (1.f + expf(-z)); }

// Two neighbouring channels at a time; `two`: both exist and the pair is aligned.
template <typename T>
__device__ __forceinline__ float2 load_pair(const T* p, bool two) {
  return make_float2(to_float(p[0]), two ? to_float(p[1]) : 0.f);
}
template <>
__device__ __forceinline__ float2 load_pair<__nv_bfloat16>(const __nv_bfloat16* p, bool two) {
  if (two && ((uintptr_t)p & 3) == 0) return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
  return make_float2(__bfloat162float(p[0]), two ? __bfloat162float(p[1]) : 0.f);
}
template <typename T>
__device__ __forceinline__ void store_pair(T* p, float2 v, bool two) {
  p[0] = from_float<T>(v.x);
  if (two) p[1] = from_float<T>(v.y);
}
template <>
__device__ __forceinline__ void store_pair<__nv_bfloat16>(__nv_bfloat16* p, float2 v, bool two) {
  if (two && ((uintptr_t)p & 3) == 0) {
    *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y);
  } else {
    p[0] = __float2bfloat16_rn(v.x);
    if (two) p[1] = __float2bfloat16_rn(v.y);
  }
}

// dt = softplus(raw + dt_bias), la = -exp(A_log) dt of one (token, head).
struct StepArgs {
  float* dt;                   // [T, H]
  float* la;
  const void* raw;             // rows of the projection (their own stride), activation type
  const void* dt_bias;
  const void* a_log;
  int H;
};
template <typename T>
__device__ __forceinline__ void ssm_step_at(const StepArgs& p, int64_t ld, int w_dtype, int64_t t, int h) {
  const float v = to_float(((const T*)p.raw)[t * ld + h]) + load_as_float(p.dt_bias, w_dtype, h);
  const float d = fmaxf(v, 0.f) + log1pf(expf(-fabsf(v)));
  p.dt[t * p.H + h] = d;
  p.la[t * p.H + h] = -expf(load_as_float(p.a_log, w_dtype, h)) * d;
}

// u [T, C] dense; xbc: rows of the projection (stride ld); state [slots, TAPS - 1, C].
template <typename T, int TAPS>
__global__ void __launch_bounds__(128)
ssm_conv_kernel(T* __restrict__ u, const T* __restrict__ xbc, int64_t ld, const void* __restrict__ w,
                const void* __restrict__ b, int w_dtype, T* __restrict__ state, const int* __restrict__ cu_q,
                const int* __restrict__ state_slots, int num_seqs, int C, int write_state, const StepArgs steps) {
  atom::pdl_trigger();
  atom::pdl_wait();
  int s, r;
  if (!ssm_find_run(blockIdx.x, cu_q, num_seqs, kSsmStrip, s, r)) return;
  if (blockIdx.y == gridDim.y - 1) {
    const int ta = cu_q[s] + r * kSsmStrip, n = min(cu_q[s + 1] - ta, kSsmStrip);
    for (int e = threadIdx.x; e < n * steps.H; e += blockDim.x)
      ssm_step_at<T>(steps, ld, w_dtype, ta + e / steps.H, e % steps.H);
    return;
  }
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * 2;
  if (c >= C) return;
  const bool two = c + 1 < C;
  const int first = cu_q[s], end = cu_q[s + 1];
  const int t0 = first + r * kSsmStrip, t1 = min(end, t0 + kSsmStrip);
  float2 wk[TAPS], in[TAPS];                 // in[TAPS - 1]: the present row; in[0]: the oldest
#pragma unroll
  for (int j = 0; j < TAPS; ++j)
    wk[j] = make_float2(load_as_float(w, w_dtype, (int64_t)c * TAPS + j),
                        two ? load_as_float(w, w_dtype, (int64_t)(c + 1) * TAPS + j) : 0.f);
  const float2 bias = make_float2(load_as_float(b, w_dtype, c), two ? load_as_float(b, w_dtype, c + 1) : 0.f);
  T* st = TAPS > 1 ? state + (int64_t)state_slots[s] * (TAPS - 1) * C + c : nullptr;
#pragma unroll
  for (int j = 0; j < TAPS - 1; ++j) {
    const int tp = t0 - (TAPS - 1) + j;
    in[j + 1] = tp >= first ? load_pair(xbc + (int64_t)tp * ld + c, two)
                            : load_pair(st + (int64_t)(TAPS - 1 - (first - tp)) * C, two);
  }
  if (TAPS > 1 && r == 0 && write_state) {
    // the request's last TAPS - 1 rows after this step: rows of the step, or of the state as it was
    const int len = end - first;
    float2 keep[TAPS];
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) {
      const int src = len - (TAPS - 1) + j;      // a row of the step (>= 0) or, counted from its end, of the old state
      if (src >= 0) {
        keep[j] = load_pair(xbc + (int64_t)(first + src) * ld + c, two);
      } else {
        keep[j] = make_float2(0.f, 0.f);
#pragma unroll
        for (int q = 0; q < TAPS - 1; ++q)
          if (q == TAPS - 1 + src) keep[j] = in[q + 1];      // (in strip 0 the window holds the old state's rows)
      }
    }
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) store_pair(st + (int64_t)j * C, keep[j], two);
  }
  for (int t = t0; t < t1; ++t) {
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) in[j] = in[j + 1];
    in[TAPS - 1] = load_pair(xbc + (int64_t)t * ld + c, two);
    float2 y = make_float2(0.f, 0.f);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      y.x = fmaf(wk[j].x, in[j].x, y.x);
      y.y = fmaf(wk[j].y, in[j].y, y.y);
    }
    store_pair(u + (int64_t)t * C + c, make_float2(ssm_silu(y.x + bias.x), ssm_silu(y.y + bias.y)), two);
  }
}

// Any number of taps; the state is only read.
template <typename T>
__global__ void ssm_conv_any_kernel(T* __restrict__ u, const T* __restrict__ xbc, int64_t ld, const void* __restrict__ w,
                                    const void* __restrict__ b, int w_dtype, const T* __restrict__ state, int taps,
                                    const int* __restrict__ seq_of_token, const int* __restrict__ cu_q,
                                    const int* __restrict__ state_slots, int C) {
  atom::pdl_trigger();
  atom::pdl_wait();
  const int t = blockIdx.x, s = seq_of_token[t];
  if (s < 0) return;
  const int first = cu_q[s];
  const T* st = state + (int64_t)state_slots[s] * (taps - 1) * C;
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x) {
    float y = 0.f;
    for (int j = 0; j < taps; ++j) {
      const int tp = t - taps + 1 + j;
      const float v = tp >= first ? to_float(xbc[(int64_t)tp * ld + c]) : to_float(st[(int64_t)(taps - 1 - (first - tp)) * C + c]);
      y = fmaf(load_as_float(w, w_dtype, (int64_t)c * taps + j), v, y);
    }
    u[(int64_t)t * C + c] = from_float<T>(ssm_silu(y + load_as_float(b, w_dtype, c)));
  }
}

template <typename T>
__global__ void ssm_step_kernel(const StepArgs steps, int64_t ld, int w_dtype, int64_t total) {
  atom::pdl_trigger();
  atom::pdl_wait();
  const int64_t e = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (e >= total) return;
  ssm_step_at<T>(steps, ld, w_dtype, e / steps.H, (int)(e % steps.H));
}

// Row n of register m of a thread of slice 0..3: runs of four in a row (one 16-byte load each).
__device__ __forceinline__ int ssm_row(int slice, int m) { return (slice + 4 * (m / 4)) * 4 + (m % 4); }

// u rows: [x (H P) | B (G N) | C (G N)], dense (C_all numbers).  dt, la [T, H].  out [T, H P] float.
// state [slots, H, N, P]; sB [run slots, H, N, P]; sA [run slots, H].
template <typename T, int KPT, int MODE>
__global__ void __launch_bounds__(kSsmThreads)
ssm_scan_kernel(float* __restrict__ out, const T* __restrict__ u, const float* __restrict__ dt, const float* __restrict__ la,
                const void* __restrict__ D, int d_dtype, float* __restrict__ state, float* __restrict__ sB,
                float* __restrict__ sA, const int* __restrict__ cu_q, const int* __restrict__ state_slots, int num_seqs,
                int H, int G, int N, int P, int run, int write_state) {
  atom::pdl_trigger();
  atom::pdl_wait();
  constexpr int NP = 4 * KPT;
  extern __shared__ __align__(16) float ssm_smem[];
  float* b_s = ssm_smem;                       // [stage][NP]
  float* c_s = b_s + kSsmStage * NP;           // [stage][NP]
  float* x_s = c_s + kSsmStage * NP;           // [stage][cols]
  __shared__ float a_s[kSsmStage], d_s[kSsmStage];
  int s, r = 0;
  if (MODE == 0) {
    s = blockIdx.x;
    if (s >= num_seqs) return;
  } else if (!ssm_find_run(blockIdx.x, cu_q, num_seqs, run, s, r)) {
    return;
  }
  const int hd = blockIdx.y, col0 = blockIdx.z * kSsmCols;
  const int g = hd / (H / G);
  const int t0 = cu_q[s] + r * run;
  const int t1 = MODE == 0 ? cu_q[s + 1] : min(cu_q[s + 1], t0 + run);
  if (t1 <= t0) return;
  const int col = threadIdx.x >> 2, slice = threadIdx.x & 3;
  const int j = col0 + col;
  const int64_t ldu = (int64_t)H * P + 2 * (int64_t)G * N;
  float* S_g = state + (((int64_t)state_slots[s] * H + hd) * N) * P;
  float* B_g = sB ? sB + (((int64_t)blockIdx.x * H + hd) * N) * P : nullptr;
  float S[KPT];
#pragma unroll
  for (int m = 0; m < KPT; ++m) {
    const int n = ssm_row(slice, m);
    if (MODE == 1 || n >= N || j >= P) S[m] = 0.f;
    else S[m] = MODE == 0 ? S_g[(int64_t)n * P + j] : B_g[(int64_t)n * P + j];
  }
  const float Dh = MODE == 1 ? 0.f : load_as_float(D, d_dtype, hd);
  float la_sum = 0.f;
  for (int c0 = t0; c0 < t1; c0 += kSsmStage) {
    const int n_rows = min(kSsmStage, t1 - c0);
    for (int e = threadIdx.x; e < n_rows * NP; e += kSsmThreads) {
      const int row = e / NP, i = e - row * NP;
      float bb = 0.f, cc = 0.f;
      if (i < N) {
        const T* ur = u + (int64_t)(c0 + row) * ldu + (int64_t)H * P + (int64_t)g * N + i;
        bb = to_float(ur[0]);
        if (MODE != 1) cc = to_float(ur[(int64_t)G * N]);
      }
      b_s[e] = bb;
      if (MODE != 1) c_s[e] = cc;
    }
    for (int e = threadIdx.x; e < n_rows * kSsmCols; e += kSsmThreads) {
      const int row = e / kSsmCols, c = e - row * kSsmCols;
      x_s[e] = col0 + c < P ? to_float(u[(int64_t)(c0 + row) * ldu + (int64_t)hd * P + col0 + c]) : 0.f;
    }
    if (threadIdx.x < n_rows) {
      const int64_t at = (int64_t)(c0 + threadIdx.x) * H + hd;
      a_s[threadIdx.x] = expf(la[at]);
      d_s[threadIdx.x] = dt[at];
    }
    __syncthreads();
    for (int row = 0; row < n_rows; ++row) {
      const float x = x_s[row * kSsmCols + col];
      const float a = a_s[row], xd = x * d_s[row];
      float acc0 = 0.f, acc1 = 0.f;
#pragma unroll
      for (int m4 = 0; m4 < KPT / 4; ++m4) {
        const int at = row * NP + (slice + 4 * m4) * 4;
        const float4 b4 = *reinterpret_cast<const float4*>(b_s + at);
        S[4 * m4] = fmaf(a, S[4 * m4], b4.x * xd);
        S[4 * m4 + 1] = fmaf(a, S[4 * m4 + 1], b4.y * xd);
        S[4 * m4 + 2] = fmaf(a, S[4 * m4 + 2], b4.z * xd);
        S[4 * m4 + 3] = fmaf(a, S[4 * m4 + 3], b4.w * xd);
        if (MODE != 1) {
          const float4 c4 = *reinterpret_cast<const float4*>(c_s + at);
          acc0 = fmaf(c4.x, S[4 * m4], acc0);
          acc1 = fmaf(c4.y, S[4 * m4 + 1], acc1);
          acc0 = fmaf(c4.z, S[4 * m4 + 2], acc0);
          acc1 = fmaf(c4.w, S[4 * m4 + 3], acc1);
        }
      }
      if (MODE != 1) {
        float acc = acc0 + acc1;
        acc += __shfl_xor_sync(0xffffffffu, acc, 1);
        acc += __shfl_xor_sync(0xffffffffu, acc, 2);
        if (slice == 0 && j < P) out[(int64_t)(c0 + row) * H * P + (int64_t)hd * P + j] = fmaf(Dh, x, acc);
      }
    }
    if (MODE == 1 && blockIdx.z == 0 && threadIdx.x == 0)
      for (int row = 0; row < n_rows; ++row) la_sum += la[(int64_t)(c0 + row) * H + hd];
    __syncthreads();
  }
  if ((MODE == 0 && !write_state) || MODE == 2) return;
  float* dst = MODE == 0 ? S_g : B_g;
#pragma unroll
  for (int m = 0; m < KPT; ++m) {
    const int n = ssm_row(slice, m);
    if (n < N && j < P) dst[(int64_t)n * P + j] = S[m];
  }
  if (MODE == 1 && blockIdx.z == 0 && threadIdx.x == 0) sA[(int64_t)blockIdx.x * H + hd] = la_sum;
}

// Per request and state element, over the request's runs in order: sB[run] <- the state the run begins with, and the
// slot takes the state after the last run.  sA: logarithms of the runs' decays.
__global__ void ssm_prefix_kernel(float* __restrict__ state, float* __restrict__ sB, const float* __restrict__ sA,
                                  const int* __restrict__ cu_q, const int* __restrict__ state_slots, int H, int mat,
                                  int run, int write_state) {
  atom::pdl_trigger();
  atom::pdl_wait();
  const int s = blockIdx.x, hd = blockIdx.y;
  const int len = cu_q[s + 1] - cu_q[s];
  if (len <= 0) return;
  int x0 = 0;
  for (int p = 0; p < s; ++p) x0 += (cu_q[p + 1] - cu_q[p] + run - 1) / run;
  const int n_runs = (len + run - 1) / run;
  float* S_g = state + ((int64_t)state_slots[s] * H + hd) * mat;
  constexpr int kAhead = 16;             // the runs' sums do not depend on S: sixteen loads are under way together
  for (int e = blockIdx.z * blockDim.x + threadIdx.x; e < mat; e += gridDim.z * blockDim.x) {
    float S = S_g[e];
    for (int r0 = 0; r0 < n_runs; r0 += kAhead) {
      float b[kAhead];
#pragma unroll
      for (int q = 0; q < kAhead; ++q)
        b[q] = r0 + q < n_runs ? sB[((int64_t)(x0 + r0 + q) * H + hd) * mat + e] : 0.f;
#pragma unroll
      for (int q = 0; q < kAhead; ++q)
        if (r0 + q < n_runs) {
          sB[((int64_t)(x0 + r0 + q) * H + hd) * mat + e] = S;
          S = fmaf(expf(sA[(int64_t)(x0 + r0 + q) * H + hd]), S, b[q]);
        }
    }
    if (write_state) S_g[e] = S;
  }
}

// y [T, n] float; z: rows of the projection (stride ldz); out rows at stride ldo.  A CTA per (token, part).
template <typename T>
__global__ void ssm_gate_norm_kernel(T* __restrict__ out, int64_t ldo, const float* __restrict__ y, const T* __restrict__ z,
                                     int64_t ldz, const void* __restrict__ w, int w_dtype, int n, int parts, float eps,
                                     float mul, const int* __restrict__ seq_of_token) {
  atom::pdl_trigger();
  atom::pdl_wait();
  __shared__ float scratch[32];
  extern __shared__ float gated[];
  const int t = blockIdx.x;
  if (seq_of_token[t] < 0) return;
  const int len = n / parts, i0 = blockIdx.y * len;
  float ss = 0.f;
  for (int i = threadIdx.x; i < len; i += blockDim.x) {
    const float v = y[(int64_t)t * n + i0 + i] * ssm_silu(to_float(z[(int64_t)t * ldz + i0 + i]));
    gated[i] = v;
    ss = fmaf(v, v, ss);
  }
  ss = block_sum(ss, scratch);
  const float f = rsqrtf(ss / (float)len + eps);
  for (int i = threadIdx.x; i < len; i += blockDim.x)
    out[(int64_t)t * ldo + i0 + i] = from_float<T>(gated[i] * f * load_as_float(w, w_dtype, i0 + i) * mul);
}

// The same for bfloat16 parts of a multiple of 8 numbers, 16 bytes at a time; at most 8 * NV * blockDim numbers a part,
// which wait in registers.
template <int NV>
__global__ void ssm_gate_norm_bf16_vec_kernel(__nv_bfloat16* __restrict__ out, int64_t ldo, const float* __restrict__ y,
                                              const __nv_bfloat16* __restrict__ z, int64_t ldz,
                                              const __nv_bfloat16* __restrict__ w, int n, int parts, float eps, float mul,
                                              const int* __restrict__ seq_of_token) {
  atom::pdl_trigger();
  atom::pdl_wait();
  __shared__ float scratch[32];
  const int t = blockIdx.x;
  if (seq_of_token[t] < 0) return;
  const int len = n / parts, i0 = blockIdx.y * len;
  float v[NV][8], ss = 0.f;
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = (threadIdx.x + k * blockDim.x) * 8;
    if (i < len) {
      const float4 a = *reinterpret_cast<const float4*>(y + (int64_t)t * n + i0 + i);
      const float4 b = *reinterpret_cast<const float4*>(y + (int64_t)t * n + i0 + i + 4);
      const uint4 raw = *reinterpret_cast<const uint4*>(z + (int64_t)t * ldz + i0 + i);
      const __nv_bfloat16* zv = reinterpret_cast<const __nv_bfloat16*>(&raw);
      v[k][0] = a.x; v[k][1] = a.y; v[k][2] = a.z; v[k][3] = a.w;
      v[k][4] = b.x; v[k][5] = b.y; v[k][6] = b.z; v[k][7] = b.w;
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        v[k][e] *= ssm_silu(__bfloat162float(zv[e]));
        ss = fmaf(v[k][e], v[k][e], ss);
      }
    }
  }
  ss = block_sum(ss, scratch);
  const float f = rsqrtf(ss / (float)len + eps);
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = (threadIdx.x + k * blockDim.x) * 8;
    if (i < len) {
      const uint4 raw = *reinterpret_cast<const uint4*>(w + i0 + i);
      const __nv_bfloat16* wv = reinterpret_cast<const __nv_bfloat16*>(&raw);
      uint4 q;
      __nv_bfloat162* h2 = reinterpret_cast<__nv_bfloat162*>(&q);
#pragma unroll
      for (int e = 0; e < 4; ++e)
        h2[e] = __floats2bfloat162_rn(v[k][2 * e] * f * __bfloat162float(wv[2 * e]) * mul,
                                      v[k][2 * e + 1] * f * __bfloat162float(wv[2 * e + 1]) * mul);
      *reinterpret_cast<uint4*>(out + (int64_t)t * ldo + i0 + i) = q;
    }
  }
}

template <typename T>
static int ssm_conv_launch(T* u, const T* xbc, int64_t ld, const void* w, const void* b, int w_dtype, T* state, int taps,
                           const int* seq_of_token, const int* cu_q, const int* state_slots, int num_seqs, int rows, int C,
                           int write_state, const StepArgs& steps, cudaStream_t stream) {
  const dim3 grid((rows + kSsmStrip - 1) / kSsmStrip + num_seqs, (C + 255) / 256 + 1);
#define ATOM_SC(N)                                                                                                  \
  case N:                                                                                                           \
    launch_pdl(ssm_conv_kernel<T, N>, grid, dim3(128), 0, stream, u, xbc, ld, w, b, w_dtype, state, cu_q, state_slots, \
               num_seqs, C, write_state, steps);                                                                    \
    break;
  switch (taps) {
    ATOM_SC(1) ATOM_SC(2) ATOM_SC(3) ATOM_SC(4) ATOM_SC(5) ATOM_SC(6) ATOM_SC(7) ATOM_SC(8)
    default:
      launch_pdl(ssm_conv_any_kernel<T>, dim3(rows, (C + 255) / 256), dim3(256), 0, stream, u, xbc, ld, w, b, w_dtype,
                 (const T*)state, taps, seq_of_token, cu_q, state_slots, C);
      const int64_t total = (int64_t)rows * steps.H;
      launch_pdl(ssm_step_kernel<T>, dim3((unsigned)((total + 127) / 128)), dim3(128), 0, stream, steps, ld, w_dtype, total);
  }
#undef ATOM_SC
  return check_launch();
}

template <typename T, int KPT>
static int ssm_scan_launch(float* out, const T* u, const float* dt, const float* la, const void* D, int d_dtype,
                           float* state, float* sB, float* sA, const int* cu_q, const int* state_slots, int num_seqs,
                           int rows, int H, int G, int N, int P, int run, int write_state, cudaStream_t stream) {
  const size_t smem = sizeof(float) * (size_t)kSsmStage * (2 * 4 * KPT + kSsmCols);
  const int cols = (P + kSsmCols - 1) / kSsmCols;
  if (run <= 0) {
    launch_pdl(ssm_scan_kernel<T, KPT, 0>, dim3(num_seqs, H, cols), dim3(kSsmThreads), smem, stream, out, u, dt, la, D,
               d_dtype, state, (float*)nullptr, (float*)nullptr, cu_q, state_slots, num_seqs, H, G, N, P, 0, write_state);
    return check_launch();
  }
  const int slots = (rows + run - 1) / run + num_seqs;
  launch_pdl(ssm_scan_kernel<T, KPT, 1>, dim3(slots, H, cols), dim3(kSsmThreads), smem, stream, out, u, dt, la, D, d_dtype,
             state, sB, sA, cu_q, state_slots, num_seqs, H, G, N, P, run, write_state);
  const int eb = (N * P + 255) / 256;
  launch_pdl(ssm_prefix_kernel, dim3(num_seqs, H, eb > 64 ? 64 : eb), dim3(256), 0, stream, state, sB, (const float*)sA,
             cu_q, state_slots, H, N * P, run, write_state);
  launch_pdl(ssm_scan_kernel<T, KPT, 2>, dim3(slots, H, cols), dim3(kSsmThreads), smem, stream, out, u, dt, la, D, d_dtype,
             state, sB, sA, cu_q, state_slots, num_seqs, H, G, N, P, run, write_state);
  return check_launch();
}

template <typename T>
static int ssm_scan_dispatch(float* out, const T* u, const float* dt, const float* la, const void* D, int d_dtype,
                             float* state, float* sB, float* sA, const int* cu_q, const int* state_slots, int num_seqs,
                             int rows, int H, int G, int N, int P, int run, int write_state, cudaStream_t stream) {
#define ATOM_SSM(K)                                                                                                    \
  if (N <= 4 * K)                                                                                                      \
    return ssm_scan_launch<T, K>(out, u, dt, la, D, d_dtype, state, sB, sA, cu_q, state_slots, num_seqs, rows, H, G, N, P, \
                                 run, write_state, stream);
  ATOM_SSM(4)
  ATOM_SSM(8)
  ATOM_SSM(16)
  ATOM_SSM(32)
  ATOM_SSM(64)
#undef ATOM_SSM
  return ATOM_ERR_ARG;
}

}  // namespace atom

ATOM_EXPORT int atom_ssm_supports(int N, int P) { return N > 0 && N <= 256 && P > 0 ? 1 : 0; }

// Whether the convolution with so many taps also brings its state up to date (and is one launch).
ATOM_EXPORT int atom_ssm_conv_updates_state(int taps) { return taps <= 8 ? 1 : 0; }

// The convolution, and dt and la [T, H] of the same rows: raw lies in rows of the same stride ld; dt_bias, a_log [H] have
// w's type.
ATOM_EXPORT int atom_ssm_conv(void* u, const void* xbc, int dtype, int64_t ld, const void* w, const void* b, int w_dtype,
                              void* state, int taps, const int* seq_of_token, const int* cu_q, const int* state_slots,
                              int num_seqs, int T, int C, int write_state, float* dt, float* la, const void* raw,
                              const void* dt_bias, const void* a_log, int H, cudaStream_t stream) {
  if (T <= 0 || num_seqs <= 0) return ATOM_OK;
  const atom::StepArgs steps{dt, la, raw, dt_bias, a_log, H};
  if (C <= 0 || H <= 0 || !dt || !la || !raw || taps < 1 || taps > 64 || (taps > 1 && !state)) return ATOM_ERR_ARG;
  if (dtype == ATOM_F32)
    return atom::ssm_conv_launch<float>((float*)u, (const float*)xbc, ld, w, b, w_dtype, (float*)state, taps, seq_of_token,
                                        cu_q, state_slots, num_seqs, T, C, write_state, steps, stream);
  if (dtype == ATOM_BF16)
    return atom::ssm_conv_launch<__nv_bfloat16>((__nv_bfloat16*)u, (const __nv_bfloat16*)xbc, ld, w, b, w_dtype,
                                                (__nv_bfloat16*)state, taps, seq_of_token, cu_q, state_slots, num_seqs, T,
                                                C, write_state, steps, stream);
  return ATOM_ERR_ARG;
}

// run 0: every request is walked once.  Otherwise sB holds (ceil(T / run) + num_seqs) * H * N * P floats and sA
// (ceil(T / run) + num_seqs) * H.
ATOM_EXPORT int atom_ssm_scan(float* out, const void* u, int dtype, const float* dt, const float* la, const void* D,
                              int d_dtype, float* state, float* sB, float* sA, const int* cu_q, const int* state_slots,
                              int num_seqs, int T, int H, int G, int N, int P, int run, int write_state,
                              cudaStream_t stream) {
  if (T <= 0 || num_seqs <= 0) return ATOM_OK;
  if (!atom_ssm_supports(N, P) || H <= 0 || H > 65535 || G <= 0 || H % G || (run > 0 && (!sB || !sA)) || num_seqs > 65535)
    return ATOM_ERR_ARG;
  if (dtype == ATOM_F32)
    return atom::ssm_scan_dispatch<float>(out, (const float*)u, dt, la, D, d_dtype, state, sB, sA, cu_q, state_slots,
                                          num_seqs, T, H, G, N, P, run, write_state, stream);
  if (dtype == ATOM_BF16)
    return atom::ssm_scan_dispatch<__nv_bfloat16>(out, (const __nv_bfloat16*)u, dt, la, D, d_dtype, state, sB, sA, cu_q,
                                                  state_slots, num_seqs, T, H, G, N, P, run, write_state, stream);
  return ATOM_ERR_ARG;
}

// The middle of the three launches over runs: ssm_prefix_kernel alone (ssm_tc.cu has the other two).
ATOM_EXPORT int atom_ssm_prefix(float* state, float* sB, const float* sA, const int* cu_q, const int* state_slots,
                                int num_seqs, int H, int N, int P, int run, int write_state, cudaStream_t stream) {
  if (num_seqs <= 0) return ATOM_OK;
  if (H <= 0 || H > 65535 || N <= 0 || P <= 0 || run <= 0 || num_seqs > 65535) return ATOM_ERR_ARG;
  const int eb = (N * P + 255) / 256;
  atom::launch_pdl(atom::ssm_prefix_kernel, dim3(num_seqs, H, eb > 64 ? 64 : eb), dim3(256), 0, stream, state, sB, sA, cu_q,
                   state_slots, H, N * P, run, write_state);
  return atom::check_launch();
}

ATOM_EXPORT int atom_ssm_gate_norm(void* out, int dtype, int64_t ldo, const float* y, const void* z, int64_t ldz,
                                   const void* w, int w_dtype, int T, int n, int parts, float eps, float mul,
                                   const int* seq_of_token, cudaStream_t stream) {
  if (T <= 0) return ATOM_OK;
  if (n <= 0 || parts <= 0 || n % parts || parts > 65535 || n / parts > 11 * 1024) return ATOM_ERR_ARG;
  const int len = n / parts;
  const int threads = len >= 1024 ? 256 : (len >= 256 ? 128 : (len > 32 ? 64 : 32));
  auto al = [](const void* q) { return ((uintptr_t)q % 16) == 0; };
  if (dtype == ATOM_BF16 && w_dtype == ATOM_BF16 && len % 8 == 0 && len <= 8 * 1024 && ldo % 8 == 0 && ldz % 8 == 0 && al(out) &&
      al(y) && al(z) && al(w)) {
    const int vecs = len / 8, th = vecs <= 512 ? ((vecs + 31) / 32) * 32 : ((vecs / 2 + 32) / 32) * 32;
    if (vecs <= 512)
      atom::launch_pdl(atom::ssm_gate_norm_bf16_vec_kernel<1>, dim3(T, parts), dim3(th), 0, stream, (__nv_bfloat16*)out, ldo, y,
                       (const __nv_bfloat16*)z, ldz, (const __nv_bfloat16*)w, n, parts, eps, mul, seq_of_token);
    else
      atom::launch_pdl(atom::ssm_gate_norm_bf16_vec_kernel<2>, dim3(T, parts), dim3(th), 0, stream, (__nv_bfloat16*)out, ldo, y,
                       (const __nv_bfloat16*)z, ldz, (const __nv_bfloat16*)w, n, parts, eps, mul, seq_of_token);
    return atom::check_launch();
  }
  const size_t smem = sizeof(float) * (size_t)len;
  if (dtype == ATOM_F32)
    atom::launch_pdl(atom::ssm_gate_norm_kernel<float>, dim3(T, parts), dim3(threads), smem, stream, (float*)out, ldo, y,
                     (const float*)z, ldz, w, w_dtype, n, parts, eps, mul, seq_of_token);
  else if (dtype == ATOM_BF16)
    atom::launch_pdl(atom::ssm_gate_norm_kernel<__nv_bfloat16>, dim3(T, parts), dim3(threads), smem, stream,
                     (__nv_bfloat16*)out, ldo, y, (const __nv_bfloat16*)z, ldz, w, w_dtype, n, parts, eps, mul, seq_of_token);
  else
    return ATOM_ERR_ARG;
  return atom::check_launch();
}
