// Gated delta rule with a decay per key channel (Kimi Linear's form of the delta rule of Yang et al. 2024, "Gated Delta
// Networks"): per value head, with unit keys and queries,
//   S <- diag(g_t) S;   u_t = beta_t (v_t - S^T k_t);   S <- S + k_t u_t^T;   o_t = S^T q_t
//
//   delta_prepare_kernel  per token, channels [q (G dk) | k (G dk) | v (H dv)]:
//                           u_t[c] = silu(sum_j w[c, j] * in_(t - taps + 1 + j)[c])   rows before the step's first token of
//                             a request from its convolution state (the last taps - 1 projected rows, only read here)
//                           rn[t] = factors that make every q and k head a unit vector, 1 / sqrt(sum u^2 + eps), the
//                             queries' times q_scale (the factor is 32-bit; u stays in the activation type)
//                           la[t] = -exp(A_log) * softplus(z + dt_bias) * log2(e)   in place of z, per head and key channel
//                           beta[t] = sigmoid(raw)   per head
//   delta_scan_kernel     the recurrence over every request's rows, the state (32-bit) carried in the request's slot.
//                         Every column of the state runs by itself: a CTA owns (a request, a head, 128 / LPC value columns),
//                         LPC neighbouring lanes share a column's key channels and hold them in registers.  Four more warps
//                         bring the next rows into shared memory (unit vectors and decays formed on the way) while
//                         the four compute warps walk the present ones.
//   delta_step_kernel     a step in which every request brings one row, everything from the projected rows to the gated
//                         output in one kernel: a CTA per (request, head), four lanes to a column of the state.  With as
//                         many q/k heads as heads it also brings the convolution's rows up to date (every channel is then
//                         one CTA's).
// Head h reads q and k head h / (H / G).
#include "common.cuh"

namespace atom {

constexpr float kDrLog2e = 1.4426950408889634f;

__device__ __forceinline__ float dr_silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float dr_silu_fast(float z) { return __fdividef(z, 1.f + __expf(-z)); }      // (before a rounding to bfloat16)
__device__ __forceinline__ float dr_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

struct DeltaPrep {
  void* u;                 // [T, C] dense, activation type
  float* rn;               // [T, 2 G]: the queries' factors, then the keys'
  const void* x;           // [T, C] rows at stride ldx
  int64_t ldx;
  const void* w;           // [C, taps]
  int w_dtype, taps;
  const void* state;       // [slots, taps - 1, C]
  float* z;                // [T, H dk] dense: in the raw decay inputs, out the decays' base-2 logarithms
  const void* A_log;       // [H]
  const void* dt_bias;     // [H dk]
  int v_dtype;             // of A_log and dt_bias
  const void* beta_in;     // [T, H] rows at stride ldb, activation type
  int64_t ldb;
  float* beta;             // [T, H]
  const int* seq_of_token;
  const int* cu_q;
  const int* state_slots;
  int G, H, dk, dv;
  float q_scale, unit_eps;
};

__device__ __forceinline__ void delta_decays4(const DeltaPrep& p, float* z, int i, const __nv_bfloat16* bias) {
  float4 v = *reinterpret_cast<const float4*>(z + i);
  const uint2 q = *reinterpret_cast<const uint2*>(bias + i);
  const float2 b0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.x));
  const float2 b1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.y));
  const float a = -expf(load_as_float(p.A_log, p.v_dtype, i / p.dk)) * kDrLog2e;
  v.x = a * dr_softplus(v.x + b0.x);
  v.y = a * dr_softplus(v.y + b0.y);
  v.z = a * dr_softplus(v.z + b1.x);
  v.w = a * dr_softplus(v.w + b1.y);
  *reinterpret_cast<float4*>(z + i) = v;
}

template <typename T>
__device__ __forceinline__ void delta_decays(const DeltaPrep& p, int t) {
  const int n = p.H * p.dk;
  float* z = p.z + (int64_t)t * n;
  if (p.dk % 4 == 0 && p.v_dtype == ATOM_BF16 && (((uintptr_t)p.z | (uintptr_t)p.dt_bias) % 16) == 0) {
    for (int i = threadIdx.x * 4; i < n; i += blockDim.x * 4) delta_decays4(p, z, i, (const __nv_bfloat16*)p.dt_bias);
  } else {
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
      const float a = expf(load_as_float(p.A_log, p.v_dtype, i / p.dk));
      z[i] = -a * kDrLog2e * dr_softplus(z[i] + load_as_float(p.dt_bias, p.v_dtype, i));
    }
  }
  for (int h = threadIdx.x; h < p.H; h += blockDim.x) {
    const float b = to_float(((const T*)p.beta_in)[(int64_t)t * p.ldb + h]);
    p.beta[(int64_t)t * p.H + h] = 1.f / (1.f + expf(-b));
  }
}

// Any sizes, both precisions.  dynamic shared memory: 2 G dk floats (the squares' summands).
template <typename T>
__global__ void __launch_bounds__(256) delta_prepare_kernel(const DeltaPrep p) {
  atom::pdl_trigger();
  atom::pdl_wait();
  extern __shared__ float dp_qk[];
  const int t = blockIdx.x, s = p.seq_of_token[t];
  if (s < 0) return;
  const int first = p.cu_q[s], qk = 2 * p.G * p.dk, C = qk + p.H * p.dv;
  const T* x = (const T*)p.x;
  const T* st = p.taps > 1 ? (const T*)p.state + (int64_t)p.state_slots[s] * (p.taps - 1) * C : nullptr;
  T* u = (T*)p.u + (int64_t)t * C;
  for (int c = threadIdx.x; c < C; c += blockDim.x) {
    float y = 0.f;
    for (int j = 0; j < p.taps; ++j) {
      const int tp = t - p.taps + 1 + j;
      const float v = tp >= first ? to_float(x[(int64_t)tp * p.ldx + c])
                                  : to_float(st[(int64_t)(p.taps - 1 - (first - tp)) * C + c]);
      y = fmaf(load_as_float(p.w, p.w_dtype, (int64_t)c * p.taps + j), v, y);
    }
    const T o = from_float<T>(dr_silu(y));
    u[c] = o;
    if (c < qk) dp_qk[c] = to_float(o);
  }
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int n = warp; n < 2 * p.G; n += blockDim.x >> 5) {
    float ss = 0.f;
    for (int i = lane; i < p.dk; i += 32) ss = fmaf(dp_qk[n * p.dk + i], dp_qk[n * p.dk + i], ss);
    ss = warp_sum(ss);
    if (lane == 0) p.rn[(int64_t)t * 2 * p.G + n] = rsqrtf(ss + p.unit_eps) * (n < p.G ? p.q_scale : 1.f);
  }
  delta_decays<T>(p, t);
}

// bfloat16 rows and taps, dk and dv in steps of 8: a thread 8 channels, 16 bytes at a time.
// dynamic shared memory: 2 G dk / 8 floats.
template <int TAPS>
__global__ void __launch_bounds__(256) delta_prepare_vec_kernel(const DeltaPrep p) {
  atom::pdl_trigger();
  atom::pdl_wait();
  extern __shared__ float dp_part[];
  const int t = blockIdx.x, s = p.seq_of_token[t];
  if (s < 0) return;
  const int first = p.cu_q[s], qk = 2 * p.G * p.dk, C = qk + p.H * p.dv;
  const __nv_bfloat16* x = (const __nv_bfloat16*)p.x;
  const __nv_bfloat16* st =
      TAPS > 1 ? (const __nv_bfloat16*)p.state + (int64_t)p.state_slots[s] * (TAPS - 1) * C : nullptr;
  for (int g = threadIdx.x; g < C / 8; g += blockDim.x) {
    const int c = g * 8;
    uint4 wraw[TAPS];                                  // the 8 channels' taps: 8 * TAPS numbers in a row
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
      wraw[j] = *reinterpret_cast<const uint4*>((const __nv_bfloat16*)p.w + (int64_t)c * TAPS + j * 8);
    const __nv_bfloat16* wv = reinterpret_cast<const __nv_bfloat16*>(wraw);
    float y[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) y[e] = 0.f;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const int tp = t - TAPS + 1 + j;
      const uint4 raw = tp >= first ? *reinterpret_cast<const uint4*>(x + (int64_t)tp * p.ldx + c)
                                    : *reinterpret_cast<const uint4*>(st + (int64_t)(TAPS - 1 - (first - tp)) * C + c);
      const __nv_bfloat16* xv = reinterpret_cast<const __nv_bfloat16*>(&raw);
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] = fmaf(__bfloat162float(wv[e * TAPS + j]), __bfloat162float(xv[e]), y[e]);
    }
    uint4 packed;
    __nv_bfloat162* h2 = reinterpret_cast<__nv_bfloat162*>(&packed);
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      h2[e] = __floats2bfloat162_rn(dr_silu_fast(y[2 * e]), dr_silu_fast(y[2 * e + 1]));
      const float2 f = __bfloat1622float2(h2[e]);
      ss = fmaf(f.x, f.x, fmaf(f.y, f.y, ss));
    }
    *reinterpret_cast<uint4*>((__nv_bfloat16*)p.u + (int64_t)t * C + c) = packed;
    if (c < qk) dp_part[g] = ss;
  }
  __syncthreads();
  const int per = p.dk / 8;
  for (int n = threadIdx.x; n < 2 * p.G; n += blockDim.x) {
    float ss = 0.f;
    for (int i = 0; i < per; ++i) ss += dp_part[n * per + i];
    p.rn[(int64_t)t * 2 * p.G + n] = rsqrtf(ss + p.unit_eps) * (n < p.G ? p.q_scale : 1.f);
  }
  delta_decays<__nv_bfloat16>(p, t);
}

// ------------------------------------------------------------------ the recurrence, row by row

constexpr int kDrCompute = 128, kDrStagers = 128;      // threads
constexpr int kDrRows = 8;                             // rows staged at a time, in two buffers

struct DeltaScan {
  float* out;              // [T, H dv] dense
  const void* u;           // [T, C] dense: q | k | v
  const float* rn;         // [T, 2 G]
  const float* la;         // [T, H dk]: base-2 logarithms of the decays
  const float* beta;       // [T, H]
  float* state;            // [slots, H, dk, dv]
  const int* cu_q;
  const int* state_slots;
  int num_seqs, G, H, dk, dv, write_state;
};

__device__ __forceinline__ float4 dr_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 dr_load4(const __nv_bfloat16* p) {
  const uint2 q = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ float4 dr_scale4(float4 v, float f) { return make_float4(v.x * f, v.y * f, v.z * f, v.w * f); }

__device__ __forceinline__ float dr_ex2(float x) {
  float y;
  asm("ex2.approx.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// Key channel of register m of a lane of slice 0 .. LPC-1: runs of four channels in a row (one 16-byte load each).
template <int LPC>
__device__ __forceinline__ int dr_channel(int slice, int m) { return (slice + LPC * (m / 4)) * 4 + (m % 4); }

template <typename T, int KPT, int LPC>
__global__ void __launch_bounds__(kDrCompute + kDrStagers) delta_scan_kernel(const DeltaScan p) {
  atom::pdl_trigger();
  atom::pdl_wait();
  constexpr int DKP = LPC * KPT, COLS = kDrCompute / LPC;
  constexpr int BUF = kDrRows * (3 * DKP + COLS) + kDrRows;
  extern __shared__ __align__(16) float dr_smem[];       // two buffers of [q | k | decay] rows, v rows, beta
  const int s = blockIdx.x, hd = blockIdx.y, col0 = blockIdx.z * COLS;
  const int t0 = p.cu_q[s], t1 = p.cu_q[s + 1];
  if (t1 <= t0) return;
  const int dk = p.dk, dv = p.dv, G = p.G, H = p.H;
  const int C = 2 * G * dk + H * dv, g = hd / (H / G);
  const T* u = (const T*)p.u;
  const bool vec = dk % 4 == 0 && C % 4 == 0 && ((uintptr_t)p.u % 16) == 0 && ((uintptr_t)p.la % 16) == 0;

  auto stage = [&](int c0, float* buf, int tid, int nthreads) {
    const int n = min(kDrRows, t1 - c0);
    float* q_s = buf;
    float* k_s = q_s + kDrRows * DKP;
    float* a_s = k_s + kDrRows * DKP;
    float* v_s = a_s + kDrRows * DKP;
    float* b_s = v_s + kDrRows * COLS;
    if (vec) {                                            // four channels at a time
      constexpr int Q = DKP / 4;
#pragma unroll 4
      for (int e = tid; e < n * Q; e += nthreads) {
        const int row = e / Q, i = (e - row * Q) * 4;
        const int64_t t = c0 + row;
        float4 qq = make_float4(0.f, 0.f, 0.f, 0.f), kk = qq, aa = make_float4(1.f, 1.f, 1.f, 1.f);
        if (i < dk) {
          qq = dr_scale4(dr_load4(u + t * C + g * dk + i), p.rn[t * 2 * G + g]);
          kk = dr_scale4(dr_load4(u + t * C + (G + g) * dk + i), p.rn[t * 2 * G + G + g]);
          aa = dr_load4(p.la + (t * H + hd) * dk + i);
          aa = make_float4(dr_ex2(aa.x), dr_ex2(aa.y), dr_ex2(aa.z), dr_ex2(aa.w));
        }
        *reinterpret_cast<float4*>(q_s + row * DKP + i) = qq;
        *reinterpret_cast<float4*>(k_s + row * DKP + i) = kk;
        *reinterpret_cast<float4*>(a_s + row * DKP + i) = aa;
      }
    } else {
      for (int e = tid; e < n * DKP; e += nthreads) {
        const int row = e / DKP, i = e - row * DKP;
        const int64_t t = c0 + row;
        float qq = 0.f, kk = 0.f, aa = 1.f;
        if (i < dk) {
          qq = to_float(u[t * C + g * dk + i]) * p.rn[t * 2 * G + g];
          kk = to_float(u[t * C + (G + g) * dk + i]) * p.rn[t * 2 * G + G + g];
          aa = dr_ex2(p.la[(t * H + hd) * dk + i]);
        }
        q_s[e] = qq;
        k_s[e] = kk;
        a_s[e] = aa;
      }
    }
    for (int e = tid; e < n * COLS; e += nthreads) {
      const int row = e / COLS, c = e - row * COLS;
      v_s[e] = col0 + c < dv ? to_float(u[(int64_t)(c0 + row) * C + 2 * G * dk + hd * dv + col0 + c]) : 0.f;
    }
    for (int e = tid; e < n; e += nthreads) b_s[e] = p.beta[(int64_t)(c0 + e) * H + hd];
  };

  stage(t0, dr_smem, threadIdx.x, kDrCompute + kDrStagers);
  __syncthreads();
  if (threadIdx.x >= kDrCompute) {                       // the staging warps: always one buffer ahead
    int b = 1;
    for (int c0 = t0; c0 < t1; c0 += kDrRows, b ^= 1) {
      if (c0 + kDrRows < t1) stage(c0 + kDrRows, dr_smem + b * BUF, threadIdx.x - kDrCompute, kDrStagers);
      __syncthreads();
    }
    return;
  }
  const int col = threadIdx.x / LPC, slice = threadIdx.x % LPC;
  const int j = col0 + col;
  float* S_g = p.state + ((int64_t)p.state_slots[s] * H + hd) * dk * dv;
  float S[KPT];
#pragma unroll
  for (int m = 0; m < KPT; ++m) {
    const int ch = dr_channel<LPC>(slice, m);
    S[m] = (ch < dk && j < dv) ? S_g[(int64_t)ch * dv + j] : 0.f;
  }
  int b = 0;
  for (int c0 = t0; c0 < t1; c0 += kDrRows, b ^= 1) {
    const int n = min(kDrRows, t1 - c0);
    const float* q_s = dr_smem + b * BUF;
    const float* k_s = q_s + kDrRows * DKP;
    const float* a_s = k_s + kDrRows * DKP;
    const float* v_s = a_s + kDrRows * DKP;
    const float* b_s = v_s + kDrRows * COLS;
    for (int row = 0; row < n; ++row) {
      const int base = row * DKP + slice * 4;
      float k[KPT];
      float p0 = 0.f, p1 = 0.f, p2 = 0.f, p3 = 0.f;
#pragma unroll
      for (int m4 = 0; m4 < KPT / 4; ++m4) {
        const float4 a4 = *reinterpret_cast<const float4*>(a_s + base + m4 * 4 * LPC);
        const float4 k4 = *reinterpret_cast<const float4*>(k_s + base + m4 * 4 * LPC);
        S[4 * m4] *= a4.x;
        S[4 * m4 + 1] *= a4.y;
        S[4 * m4 + 2] *= a4.z;
        S[4 * m4 + 3] *= a4.w;
        k[4 * m4] = k4.x;
        k[4 * m4 + 1] = k4.y;
        k[4 * m4 + 2] = k4.z;
        k[4 * m4 + 3] = k4.w;
        p0 = fmaf(S[4 * m4], k4.x, p0);
        p1 = fmaf(S[4 * m4 + 1], k4.y, p1);
        p2 = fmaf(S[4 * m4 + 2], k4.z, p2);
        p3 = fmaf(S[4 * m4 + 3], k4.w, p3);
      }
      float pk = (p0 + p1) + (p2 + p3);
#pragma unroll
      for (int o = 1; o < LPC; o <<= 1) pk += __shfl_xor_sync(0xffffffffu, pk, o);
      const float uu = b_s[row] * (v_s[row * COLS + col] - pk);
      p0 = p1 = p2 = p3 = 0.f;
#pragma unroll
      for (int m4 = 0; m4 < KPT / 4; ++m4) {
        const float4 q4 = *reinterpret_cast<const float4*>(q_s + base + m4 * 4 * LPC);
        S[4 * m4] = fmaf(k[4 * m4], uu, S[4 * m4]);
        S[4 * m4 + 1] = fmaf(k[4 * m4 + 1], uu, S[4 * m4 + 1]);
        S[4 * m4 + 2] = fmaf(k[4 * m4 + 2], uu, S[4 * m4 + 2]);
        S[4 * m4 + 3] = fmaf(k[4 * m4 + 3], uu, S[4 * m4 + 3]);
        p0 = fmaf(S[4 * m4], q4.x, p0);
        p1 = fmaf(S[4 * m4 + 1], q4.y, p1);
        p2 = fmaf(S[4 * m4 + 2], q4.z, p2);
        p3 = fmaf(S[4 * m4 + 3], q4.w, p3);
      }
      float pq = (p0 + p1) + (p2 + p3);
#pragma unroll
      for (int o = 1; o < LPC; o <<= 1) pq += __shfl_xor_sync(0xffffffffu, pq, o);
      if (slice == 0 && j < dv) p.out[((int64_t)(c0 + row) * H + hd) * dv + j] = pq;
    }
    __syncthreads();
  }
  if (!p.write_state) return;
#pragma unroll
  for (int m = 0; m < KPT; ++m) {
    const int ch = dr_channel<LPC>(slice, m);
    if (ch < dk && j < dv) S_g[(int64_t)ch * dv + j] = S[m];
  }
}

// ------------------------------------------------------------------ one row per request

struct DeltaStep {
  DeltaPrep in;            // (u, rn and beta are not used; z holds the raw decay inputs; state is brought up to date)
  float* S;                // [slots, H, dk, dv]
  void* y;                 // [T, H dv] rows at stride ldy
  int64_t ldy;
  const void* gate;        // [T, H dv] rows at stride ldg
  int64_t ldg;
  const void* norm;        // [dv]
  int norm_dtype;
  float norm_eps, y_scale;
  int write_state;
};

template <typename T, int KPT>
__global__ void __launch_bounds__(512) delta_step_kernel(const DeltaStep d) {
  atom::pdl_trigger();
  atom::pdl_wait();
  constexpr int DKP = 4 * KPT;
  __shared__ __align__(16) float q_s[DKP], k_s[DKP], a_s[DKP];
  __shared__ float v_s[128], f_s[2], scratch[32];
  const DeltaPrep& p = d.in;
  const int s = blockIdx.x, hd = blockIdx.y, tid = threadIdx.x;
  const int t = p.cu_q[s];
  if (p.cu_q[s + 1] - t <= 0) return;
  const int dk = p.dk, dv = p.dv, G = p.G, H = p.H, g = hd / (H / G);
  const int C = 2 * G * dk + H * dv, slot = p.state_slots[s];
  const int col = tid >> 2, slice = tid & 3;
  float* S_g = d.S + ((int64_t)slot * H + hd) * dk * dv;
  float S[KPT];
#pragma unroll
  for (int m = 0; m < KPT; ++m) {
    const int ch = dr_channel<4>(slice, m);
    S[m] = (ch < dk && col < dv) ? S_g[(int64_t)ch * dv + col] : 0.f;
  }
  T* st = p.taps > 1 ? (T*)p.state + (int64_t)slot * (p.taps - 1) * C : nullptr;
  const bool shift = st && d.write_state && H == G;
  for (int e = tid; e < 2 * dk + dv; e += blockDim.x) {
    const int c = e < dk ? g * dk + e : (e < 2 * dk ? (G + g) * dk + e - dk : 2 * G * dk + hd * dv + e - 2 * dk);
    const T now = ((const T*)p.x)[(int64_t)t * p.ldx + c];
    float y = 0.f;
    for (int j = 0; j < p.taps - 1; ++j) {
      const T old = st[(int64_t)j * C + c];
      y = fmaf(load_as_float(p.w, p.w_dtype, (int64_t)c * p.taps + j), to_float(old), y);
      if (shift && j > 0) st[(int64_t)(j - 1) * C + c] = old;
    }
    if (shift) st[(int64_t)(p.taps - 2) * C + c] = now;
    y = fmaf(load_as_float(p.w, p.w_dtype, (int64_t)c * p.taps + p.taps - 1), to_float(now), y);
    const float o = to_float(from_float<T>(dr_silu(y)));
    if (e < dk) q_s[e] = o;
    else if (e < 2 * dk) k_s[e - dk] = o;
    else v_s[e - 2 * dk] = o;
  }
  for (int i = tid; i < DKP; i += blockDim.x) {
    float a = 1.f;
    if (i < dk) {
      const int64_t at = (int64_t)hd * dk + i;
      const float A = expf(load_as_float(p.A_log, p.v_dtype, hd));
      a = dr_ex2(-A * kDrLog2e * dr_softplus(p.z[(int64_t)t * H * dk + at] + load_as_float(p.dt_bias, p.v_dtype, at)));
    } else {
      q_s[i] = k_s[i] = 0.f;
    }
    a_s[i] = a;
  }
  const float beta = 1.f / (1.f + expf(-to_float(((const T*)p.beta_in)[(int64_t)t * p.ldb + hd])));
  __syncthreads();
  const int warp = tid >> 5, lane = tid & 31, warps = blockDim.x >> 5;
  for (int n = warp; n < 2; n += warps) {
    const float* x = n ? k_s : q_s;
    float ss = 0.f;
    for (int i = lane; i < dk; i += 32) ss = fmaf(x[i], x[i], ss);
    ss = warp_sum(ss);
    if (lane == 0) f_s[n] = rsqrtf(ss + p.unit_eps) * (n ? 1.f : p.q_scale);
  }
  __syncthreads();
  const float fq = f_s[0], fk = f_s[1];
  float p0 = 0.f, p1 = 0.f, p2 = 0.f, p3 = 0.f;
#pragma unroll
  for (int m4 = 0; m4 < KPT / 4; ++m4) {
    const float4 a4 = *reinterpret_cast<const float4*>(a_s + slice * 4 + m4 * 16);
    const float4 k4 = *reinterpret_cast<const float4*>(k_s + slice * 4 + m4 * 16);
    S[4 * m4] *= a4.x;
    S[4 * m4 + 1] *= a4.y;
    S[4 * m4 + 2] *= a4.z;
    S[4 * m4 + 3] *= a4.w;
    p0 = fmaf(S[4 * m4], k4.x, p0);
    p1 = fmaf(S[4 * m4 + 1], k4.y, p1);
    p2 = fmaf(S[4 * m4 + 2], k4.z, p2);
    p3 = fmaf(S[4 * m4 + 3], k4.w, p3);
  }
  float pk = ((p0 + p1) + (p2 + p3)) * fk;
  pk += __shfl_xor_sync(0xffffffffu, pk, 1);
  pk += __shfl_xor_sync(0xffffffffu, pk, 2);
  const float ku = col < dv ? beta * (v_s[col] - pk) * fk : 0.f;
  p0 = p1 = p2 = p3 = 0.f;
#pragma unroll
  for (int m4 = 0; m4 < KPT / 4; ++m4) {
    const float4 k4 = *reinterpret_cast<const float4*>(k_s + slice * 4 + m4 * 16);
    const float4 q4 = *reinterpret_cast<const float4*>(q_s + slice * 4 + m4 * 16);
    S[4 * m4] = fmaf(k4.x, ku, S[4 * m4]);
    S[4 * m4 + 1] = fmaf(k4.y, ku, S[4 * m4 + 1]);
    S[4 * m4 + 2] = fmaf(k4.z, ku, S[4 * m4 + 2]);
    S[4 * m4 + 3] = fmaf(k4.w, ku, S[4 * m4 + 3]);
    p0 = fmaf(S[4 * m4], q4.x, p0);
    p1 = fmaf(S[4 * m4 + 1], q4.y, p1);
    p2 = fmaf(S[4 * m4 + 2], q4.z, p2);
    p3 = fmaf(S[4 * m4 + 3], q4.w, p3);
  }
  float o = ((p0 + p1) + (p2 + p3)) * fq;
  o += __shfl_xor_sync(0xffffffffu, o, 1);
  o += __shfl_xor_sync(0xffffffffu, o, 2);
  if (d.write_state) {
#pragma unroll
    for (int m = 0; m < KPT; ++m) {
      const int ch = dr_channel<4>(slice, m);
      if (ch < dk && col < dv) S_g[(int64_t)ch * dv + col] = S[m];
    }
  }
  const bool own = slice == 0 && col < dv;
  const float ss = block_sum(own ? o * o : 0.f, scratch);
  if (own) {
    const float z = to_float(((const T*)d.gate)[(int64_t)t * d.ldg + (int64_t)hd * dv + col]);
    ((T*)d.y)[(int64_t)t * d.ldy + (int64_t)hd * dv + col] =
        from_float<T>(o * rsqrtf(ss / (float)dv + d.norm_eps) * d.y_scale * load_as_float(d.norm, d.norm_dtype, col) /
                      (1.f + expf(-z)));
  }
}

template <typename T>
static int launch_delta_step(const DeltaStep& d, int num_seqs, cudaStream_t stream) {
  const dim3 grid(num_seqs, d.in.H), block((d.in.dv + 7) / 8 * 32);
  const int dk = d.in.dk;
  if (dk <= 32) launch_pdl(delta_step_kernel<T, 8>, grid, block, 0, stream, d);
  else if (dk <= 64) launch_pdl(delta_step_kernel<T, 16>, grid, block, 0, stream, d);
  else if (dk <= 96) launch_pdl(delta_step_kernel<T, 24>, grid, block, 0, stream, d);
  else launch_pdl(delta_step_kernel<T, 32>, grid, block, 0, stream, d);
  return check_launch();
}

template <typename T, int KPT, int LPC>
static int launch_delta_scan(const DeltaScan& p, cudaStream_t stream) {
  constexpr int DKP = LPC * KPT, COLS = kDrCompute / LPC;
  const size_t smem = sizeof(float) * 2 * (size_t)(kDrRows * (3 * DKP + COLS) + kDrRows);
  if (smem > 48 * 1024 &&
      cudaFuncSetAttribute(delta_scan_kernel<T, KPT, LPC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return ATOM_ERR_LAUNCH;
  launch_pdl(delta_scan_kernel<T, KPT, LPC>, dim3(p.num_seqs, p.H, (p.dv + COLS - 1) / COLS), dim3(kDrCompute + kDrStagers),
             smem, stream, p);
  return check_launch();
}

template <typename T>
static int dispatch_delta_scan(const DeltaScan& p, int lanes, cudaStream_t stream) {
  const int dk = p.dk;
  if (lanes == 8) {
    if (dk <= 32) return launch_delta_scan<T, 4, 8>(p, stream);
    if (dk <= 64) return launch_delta_scan<T, 8, 8>(p, stream);
    if (dk <= 96) return launch_delta_scan<T, 12, 8>(p, stream);
    if (dk <= 128) return launch_delta_scan<T, 16, 8>(p, stream);
    if (dk <= 192) return launch_delta_scan<T, 24, 8>(p, stream);
    if (dk <= 256) return launch_delta_scan<T, 32, 8>(p, stream);
    return ATOM_ERR_ARG;
  }
  if (dk <= 16) return launch_delta_scan<T, 4, 4>(p, stream);
  if (dk <= 32) return launch_delta_scan<T, 8, 4>(p, stream);
  if (dk <= 64) return launch_delta_scan<T, 16, 4>(p, stream);
  if (dk <= 96) return launch_delta_scan<T, 24, 4>(p, stream);
  if (dk <= 128) return launch_delta_scan<T, 32, 4>(p, stream);
  return ATOM_ERR_ARG;
}

}  // namespace atom

ATOM_EXPORT int atom_delta_supports(int dk, int dv) { return dk > 0 && dk <= 256 && dv > 0 ? 1 : 0; }

ATOM_EXPORT int atom_delta_step_supports(int dk, int dv) { return dk > 0 && dk <= 128 && dv > 0 && dv <= 128 ? 1 : 0; }

ATOM_EXPORT int atom_delta_step(void* y, int64_t ldy, const void* x, int dtype, int64_t ldx, const void* w, int w_dtype,
                                int taps, void* state, const float* z, const void* A_log, const void* dt_bias, int v_dtype,
                                const void* beta_in, int64_t ldb, const void* gate, int64_t ldg, const void* norm,
                                int norm_dtype, float norm_eps, float y_scale, float* S, const int* cu_q,
                                const int* state_slots, int num_seqs, int G, int H, int dk, int dv, float q_scale,
                                float unit_eps, int write_state, cudaStream_t stream) {
  if (num_seqs <= 0) return ATOM_OK;
  if (!atom_delta_step_supports(dk, dv) || G <= 0 || H <= 0 || H % G || H > 65535 || taps < 1 || (taps > 1 && !state) ||
      (w_dtype != ATOM_F32 && w_dtype != ATOM_BF16) || (v_dtype != ATOM_F32 && v_dtype != ATOM_BF16) ||
      (norm_dtype != ATOM_F32 && norm_dtype != ATOM_BF16))
    return ATOM_ERR_ARG;
  const atom::DeltaPrep in{nullptr, nullptr, x,   ldx,     w,       w_dtype, taps,        state, const_cast<float*>(z), A_log,
                           dt_bias, v_dtype, beta_in, ldb, nullptr, nullptr, cu_q, state_slots, G, H, dk, dv, q_scale, unit_eps};
  const atom::DeltaStep d{in, S, y, ldy, gate, ldg, norm, norm_dtype, norm_eps, y_scale, write_state};
  if (dtype == ATOM_F32) return atom::launch_delta_step<float>(d, num_seqs, stream);
  if (dtype == ATOM_BF16) return atom::launch_delta_step<__nv_bfloat16>(d, num_seqs, stream);
  return ATOM_ERR_ARG;
}

ATOM_EXPORT int atom_delta_prepare(void* u, float* rn, const void* x, int dtype, int64_t ldx, const void* w, int w_dtype,
                                   int taps, const void* state, float* z, const void* A_log, const void* dt_bias,
                                   int v_dtype, const void* beta_in, int64_t ldb, float* beta, const int* seq_of_token,
                                   const int* cu_q, const int* state_slots, int T, int G, int H, int dk, int dv,
                                   float q_scale, float unit_eps, cudaStream_t stream) {
  if (T <= 0) return ATOM_OK;
  if (G <= 0 || H <= 0 || H % G || dk <= 0 || dv <= 0 || taps < 1 || (taps > 1 && !state) ||
      (w_dtype != ATOM_F32 && w_dtype != ATOM_BF16) || (v_dtype != ATOM_F32 && v_dtype != ATOM_BF16))
    return ATOM_ERR_ARG;
  const atom::DeltaPrep p{u,  rn,  x,    ldx,          w,    w_dtype,     taps, state, z,  A_log, dt_bias, v_dtype, beta_in,
                          ldb, beta, seq_of_token, cu_q, state_slots, G,    H,     dk, dv,    q_scale, unit_eps};
  const uintptr_t all = (uintptr_t)u | (uintptr_t)x | (uintptr_t)w | (uintptr_t)state;
  if (dtype == ATOM_BF16 && w_dtype == ATOM_BF16 && dk % 8 == 0 && dv % 8 == 0 && ldx % 8 == 0 && taps <= 8 && all % 16 == 0 &&
      (size_t)G * dk <= 48 * 1024) {
    const size_t smem = sizeof(float) * (2 * (size_t)G * dk / 8);
#define ATOM_DP(N) \
  case N: atom::launch_pdl(atom::delta_prepare_vec_kernel<N>, dim3(T), dim3(256), smem, stream, p); break
    switch (taps) {
      ATOM_DP(1);
      ATOM_DP(2);
      ATOM_DP(3);
      ATOM_DP(4);
      ATOM_DP(5);
      ATOM_DP(6);
      ATOM_DP(7);
      ATOM_DP(8);
    }
#undef ATOM_DP
    return atom::check_launch();
  }
  const size_t smem = sizeof(float) * 2 * (size_t)G * dk;
  if (smem > 200 * 1024) return ATOM_ERR_ARG;
  if (dtype == ATOM_F32) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(atom::delta_prepare_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    atom::launch_pdl(atom::delta_prepare_kernel<float>, dim3(T), dim3(256), smem, stream, p);
  } else if (dtype == ATOM_BF16) {
    if (smem > 48 * 1024)
      cudaFuncSetAttribute(atom::delta_prepare_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    atom::launch_pdl(atom::delta_prepare_kernel<__nv_bfloat16>, dim3(T), dim3(256), smem, stream, p);
  } else {
    return ATOM_ERR_ARG;
  }
  return atom::check_launch();
}

// lanes: lanes that share a column of the state, 4 (dk up to 128) or 8.
ATOM_EXPORT int atom_delta_scan(float* out, const void* u, int dtype, const float* rn, const float* la, const float* beta,
                                float* state, const int* cu_q, const int* state_slots, int num_seqs, int T, int G, int H,
                                int dk, int dv, int lanes, int write_state, cudaStream_t stream) {
  if (T <= 0 || num_seqs <= 0) return ATOM_OK;
  if (!atom_delta_supports(dk, dv) || G <= 0 || H <= 0 || H % G || H > 65535 || (lanes != 4 && lanes != 8)) return ATOM_ERR_ARG;
  const atom::DeltaScan p{out, u, rn, la, beta, state, cu_q, state_slots, num_seqs, G, H, dk, dv, write_state};
  if (dtype == ATOM_F32) return atom::dispatch_delta_scan<float>(p, lanes, stream);
  if (dtype == ATOM_BF16) return atom::dispatch_delta_scan<__nv_bfloat16>(p, lanes, stream);
  return ATOM_ERR_ARG;
}
