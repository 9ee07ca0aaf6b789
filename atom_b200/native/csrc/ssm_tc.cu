// The recurrence of ssm.cu in bfloat16 on the tensor cores, for steps that bring more than a few rows of a request:
// rows are cut into chunks of 64, and with c_t the sum of the logarithms of the decays up to row t of a chunk,
//   chunk sum   B = sum_s exp(c_end - c_s) dt_s B_s x_s^T                                (ssm_chunk_sum_kernel)
//   prefix      the state every chunk begins with, over the chunks in order              (ssm.cu: ssm_prefix_kernel)
//   outputs     y_t = exp(c_t) S_begin^T C_t + sum_(s <= t) (C_t . B_s) exp(c_t - c_s) dt_s x_s + D x_t
//                                                                                        (ssm_chunk_out_kernel)
// x, B and C are bfloat16 already, so the products C_t . B_s are exact with 32-bit sums.  Every 32-bit operand (the
// weighted x of the chunk sum, the state, the weights of the last sum) enters its product as THREE bfloat16 numbers,
// hi + mid + lo, which hold all 24 bits of its mantissa; the sums are 32-bit.  The c are summed in 64-bit and kept as
// two 32-bit numbers, so that a difference c_t - c_s is as exact as its own size allows.
//
// A CTA of 4 warps owns (a chunk, a head, 64 value columns).  Sizes: N and P multiples of 8, N up to 256; what a tile
// has beyond them is zero.
#include "common.cuh"

namespace atom {
namespace ssmtc {

constexpr int L = 64, PT = 64, THREADS = 128;
constexpr int LDP = PT + 8;                       // bf16 elements per row of 64 columns in shared memory

__device__ __forceinline__ void ldm_x4(uint32_t (&r)[4], const void* smem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void ldm_x4_trans(uint32_t (&r)[4], const void* smem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, "
      "{%0,%1,%2,%3};\n"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(void* smem, const void* gmem, bool valid) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  const int n = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(s), "l"(gmem), "r"(n));
}
__device__ __forceinline__ uint32_t pack2(__nv_bfloat16 a, __nv_bfloat16 b) {
  return (uint32_t)__bfloat16_as_ushort(a) | ((uint32_t)__bfloat16_as_ushort(b) << 16);
}
// x = h + m + l, each a bfloat16 number.
__device__ __forceinline__ void split3(float x, __nv_bfloat16& h, __nv_bfloat16& m, __nv_bfloat16& l) {
  h = __float2bfloat16_rn(x);
  const float r = x - __bfloat162float(h);
  m = __float2bfloat16_rn(r);
  l = __float2bfloat16_rn(r - __bfloat162float(m));
}

// Chunk x -> request and chunk number: requests take ceil(len / L) chunks one after another.
__device__ __forceinline__ bool find_chunk(int x, const int* __restrict__ cu_q, int num_seqs, int& s, int& r) {
  int acc = 0;
  for (s = 0; s < num_seqs; ++s) {
    const int n = (cu_q[s + 1] - cu_q[s] + L - 1) / L;
    if (x < acc + n) {
      r = x - acc;
      return true;
    }
    acc += n;
  }
  return false;
}

struct Chunk {
  float hi[L], lo[L];       // c_t = hi + lo
  float dt[L];
};

// By the first warp: c and dt of the chunk's rows (rows beyond `rows`: c stays, dt = 0).
__device__ __forceinline__ void load_chunk(Chunk& c, const float* __restrict__ dt, const float* __restrict__ la, int t0,
                                           int rows, int H, int h) {
  if (threadIdx.x >= 32) return;
  const int lane = threadIdx.x, i = 2 * lane;
  const int64_t at = (int64_t)(t0 + i) * H + h;
  const double a = i < rows ? (double)la[at] : 0.0, b = i + 1 < rows ? (double)la[at + H] : 0.0;
  double sum = a + b;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const double up = __shfl_up_sync(0xffffffffu, sum, o);
    if (lane >= o) sum += up;
  }
  const double c1 = sum, c0 = sum - b;
  c.hi[i] = (float)c0;
  c.lo[i] = (float)(c0 - (double)(float)c0);
  c.hi[i + 1] = (float)c1;
  c.lo[i + 1] = (float)(c1 - (double)(float)c1);
  c.dt[i] = i < rows ? dt[at] : 0.f;
  c.dt[i + 1] = i + 1 < rows ? dt[at + H] : 0.f;
}

// N columns of rows t0 .. t0 + 63 (zeros beyond `rows`) into shared memory rows of ld elements; Np: N rounded up to 16.
__device__ __forceinline__ void load_rows(__nv_bfloat16* dst, int ld, const __nv_bfloat16* __restrict__ src, int64_t lds,
                                          int rows, int n, int np) {
  const int pieces = np / 8;
  for (int e = threadIdx.x; e < L * pieces; e += THREADS) {
    const int r = e / pieces, c = (e - r * pieces) * 8;
    const bool valid = r < rows && c < n;
    cp_async16(dst + r * ld + c, src + (valid ? (int64_t)r * lds + c : 0), valid);
  }
}

struct Params {
  const __nv_bfloat16* u;      // rows [x (H P) | B (G N) | C (G N)], dense
  const float* dt;
  const float* la;
  const float* D;              // [H]
  float* out;                  // [T, H P]
  float* sB;                   // [chunks, H, N, P]
  float* sA;                   // [chunks, H]
  const int* cu_q;
  int num_seqs, H, G, N, P;
};

__global__ void __launch_bounds__(THREADS) ssm_chunk_sum_kernel(const Params p) {
  atom::pdl_trigger();
  atom::pdl_wait();
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __shared__ Chunk ch;
  int s, r;
  if (!find_chunk(blockIdx.x, p.cu_q, p.num_seqs, s, r)) return;
  const int h = blockIdx.y, p0 = blockIdx.z * PT, g = h / (p.H / p.G);
  const int t0 = p.cu_q[s] + r * L, rows = min(L, p.cu_q[s + 1] - t0);
  const int np = (p.N + 15) & ~15, ldn = np + 8;
  const int64_t ldu = (int64_t)p.H * p.P + 2 * (int64_t)p.G * p.N;
  __nv_bfloat16* Bs = reinterpret_cast<__nv_bfloat16*>(smem_raw);       // [L][ldn]
  __nv_bfloat16* Xw = Bs + L * ldn;                                        // [3][L][LDP]
  const __nv_bfloat16* ub = p.u + (int64_t)t0 * ldu;
  load_rows(Bs, ldn, ub + (int64_t)p.H * p.P + (int64_t)g * p.N, ldu, rows, p.N, np);
  asm volatile("cp.async.commit_group;\n" ::);
  load_chunk(ch, p.dt, p.la, t0, rows, p.H, h);
  __syncthreads();
  const float end_hi = ch.hi[L - 1], end_lo = ch.lo[L - 1];
  for (int e = threadIdx.x; e < L * (PT / 8); e += THREADS) {
    const int row = e / (PT / 8), c = (e % (PT / 8)) * 8;
    uint4 raw = make_uint4(0u, 0u, 0u, 0u);
    if (row < rows && p0 + c < p.P)
      raw = *reinterpret_cast<const uint4*>(ub + (int64_t)row * ldu + (int64_t)h * p.P + p0 + c);
    const __nv_bfloat16* xv = reinterpret_cast<const __nv_bfloat16*>(&raw);
    const float w = ch.dt[row] * expf((end_hi - ch.hi[row]) + (end_lo - ch.lo[row]));
    uint4 o[3];
    __nv_bfloat16* o0 = reinterpret_cast<__nv_bfloat16*>(&o[0]);
    __nv_bfloat16* o1 = reinterpret_cast<__nv_bfloat16*>(&o[1]);
    __nv_bfloat16* o2 = reinterpret_cast<__nv_bfloat16*>(&o[2]);
#pragma unroll
    for (int i = 0; i < 8; ++i) split3(w * __bfloat162float(xv[i]), o0[i], o1[i], o2[i]);
#pragma unroll
    for (int k = 0; k < 3; ++k) *reinterpret_cast<uint4*>(Xw + (k * L + row) * LDP + c) = o[k];
  }
  asm volatile("cp.async.wait_group 0;\n" ::);
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* dst = p.sB + (((int64_t)blockIdx.x * p.H + h) * p.N) * p.P;
  for (int mt = warp; mt * 16 < np; mt += 4) {
    float acc[PT / 8][4];
#pragma unroll
    for (int i = 0; i < PT / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < L / 16; ++kk) {
      uint32_t a[4];      // rows of the product are state rows n, its inner dimension the chunk's rows: B^T
      ldm_x4_trans(a, Bs + (kk * 16 + (lane >> 4) * 8 + (lane & 7)) * ldn + mt * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int k = 2; k >= 0; --k) {
#pragma unroll
        for (int q = 0; q < PT / 16; ++q) {
          uint32_t b[4];
          ldm_x4_trans(b, Xw + (k * L + kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * LDP + q * 16 + (lane >> 4) * 8);
          mma_bf16(acc[2 * q], a, b[0], b[1]);
          mma_bf16(acc[2 * q + 1], a, b[2], b[3]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < PT / 8; ++i) {
      const int c = p0 + i * 8 + (lane & 3) * 2;
      if (c >= p.P) continue;
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const int n = mt * 16 + (lane >> 2) + 8 * k;
        if (n < p.N) *reinterpret_cast<float2*>(dst + (int64_t)n * p.P + c) = make_float2(acc[i][2 * k], acc[i][2 * k + 1]);
      }
    }
  }
  if (blockIdx.z == 0 && threadIdx.x == 0) p.sA[(int64_t)blockIdx.x * p.H + h] = end_hi;
}

__global__ void __launch_bounds__(THREADS) ssm_chunk_out_kernel(const Params p) {
  atom::pdl_trigger();
  atom::pdl_wait();
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __shared__ Chunk ch;
  int s, r;
  if (!find_chunk(blockIdx.x, p.cu_q, p.num_seqs, s, r)) return;
  const int h = blockIdx.y, p0 = blockIdx.z * PT, g = h / (p.H / p.G);
  const int t0 = p.cu_q[s] + r * L, rows = min(L, p.cu_q[s + 1] - t0);
  const int np = (p.N + 15) & ~15, ldn = np + 8;
  const int64_t ldu = (int64_t)p.H * p.P + 2 * (int64_t)p.G * p.N;
  __nv_bfloat16* Cs = reinterpret_cast<__nv_bfloat16*>(smem_raw);       // [L][ldn]
  __nv_bfloat16* Bs = Cs + L * ldn;                                        // [L][ldn]
  __nv_bfloat16* Xs = Bs + L * ldn;                                        // [L][LDP]
  __nv_bfloat16* Ss = Xs + L * LDP;                                        // [3][np][LDP]
  const __nv_bfloat16* ub = p.u + (int64_t)t0 * ldu;
  const __nv_bfloat16* uB = ub + (int64_t)p.H * p.P + (int64_t)g * p.N;
  load_rows(Cs, ldn, uB + (int64_t)p.G * p.N, ldu, rows, p.N, np);
  load_rows(Bs, ldn, uB, ldu, rows, p.N, np);
  load_rows(Xs, LDP, ub + (int64_t)h * p.P + p0, ldu, rows, min(PT, p.P - p0), PT);
  asm volatile("cp.async.commit_group;\n" ::);
  load_chunk(ch, p.dt, p.la, t0, rows, p.H, h);
  const float* S = p.sB + (((int64_t)blockIdx.x * p.H + h) * p.N) * p.P + p0;
  for (int e = threadIdx.x; e < np * (PT / 4); e += THREADS) {
    const int n = e / (PT / 4), c = (e % (PT / 4)) * 4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (n < p.N && p0 + c < p.P) v = *reinterpret_cast<const float4*>(S + (int64_t)n * p.P + c);
    __nv_bfloat16 a[3][4];
    split3(v.x, a[0][0], a[1][0], a[2][0]);
    split3(v.y, a[0][1], a[1][1], a[2][1]);
    split3(v.z, a[0][2], a[1][2], a[2][2]);
    split3(v.w, a[0][3], a[1][3], a[2][3]);
#pragma unroll
    for (int k = 0; k < 3; ++k)
      *reinterpret_cast<uint2*>(Ss + (k * np + n) * LDP + c) = make_uint2(pack2(a[k][0], a[k][1]), pack2(a[k][2], a[k][3]));
  }
  asm volatile("cp.async.wait_group 0;\n" ::);
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (warp * 16 >= rows) return;
  float o[PT / 8][4], sc[L / 8][4];
#pragma unroll
  for (int i = 0; i < PT / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
#pragma unroll
  for (int i = 0; i < L / 8; ++i) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = 0.f;
  // C . S_begin, and the products C_t . B_s of the chunk's rows up to this warp's
  for (int kk = 0; kk < np / 16; ++kk) {
    uint32_t a[4];
    ldm_x4(a, Cs + (warp * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * ldn + kk * 16 + (lane >> 4) * 8);
#pragma unroll
    for (int k = 2; k >= 0; --k) {
#pragma unroll
      for (int q = 0; q < PT / 16; ++q) {
        uint32_t b[4];
        ldm_x4_trans(b, Ss + (k * np + kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * LDP + q * 16 + (lane >> 4) * 8);
        mma_bf16(o[2 * q], a, b[0], b[1]);
        mma_bf16(o[2 * q + 1], a, b[2], b[3]);
      }
    }
#pragma unroll
    for (int q = 0; q < L / 16; ++q) {
      if (q > warp) break;
      uint32_t b[4];
      ldm_x4(b, Bs + (q * 16 + (lane >> 4) * 8 + (lane & 7)) * ldn + kk * 16 + ((lane >> 3) & 1) * 8);
      mma_bf16(sc[2 * q], a, b[0], b[1]);
      mma_bf16(sc[2 * q + 1], a, b[2], b[3]);
    }
  }
  const int ta = warp * 16 + (lane >> 2), tb = ta + 8;
  const float ha = ch.hi[ta], la = ch.lo[ta], hb = ch.hi[tb], lb = ch.lo[tb];
  const float ea = expf(ha), eb = expf(hb);
#pragma unroll
  for (int i = 0; i < PT / 8; ++i) {
    o[i][0] *= ea;
    o[i][1] *= ea;
    o[i][2] *= eb;
    o[i][3] *= eb;
  }
  // (C_t . B_s) exp(c_t - c_s) dt_s for s <= t, times x
#pragma unroll
  for (int ks = 0; ks < L / 16; ++ks) {
    if (ks > warp) break;
    uint32_t w[3][4];
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int nt = 2 * ks + half;
      __nv_bfloat16 v[3][4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int col = nt * 8 + (lane & 3) * 2 + (e & 1);
        const int row = e < 2 ? ta : tb;
        const float d = e < 2 ? (ha - ch.hi[col]) + (la - ch.lo[col]) : (hb - ch.hi[col]) + (lb - ch.lo[col]);
        const float x = col <= row ? sc[nt][e] * (ch.dt[col] * expf(d)) : 0.f;
        split3(x, v[0][e], v[1][e], v[2][e]);
      }
#pragma unroll
      for (int k = 0; k < 3; ++k) {
        w[k][2 * half] = pack2(v[k][0], v[k][1]);
        w[k][2 * half + 1] = pack2(v[k][2], v[k][3]);
      }
    }
#pragma unroll
    for (int q = 0; q < PT / 16; ++q) {
      uint32_t b[4];
      ldm_x4_trans(b, Xs + (ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * LDP + q * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int k = 2; k >= 0; --k) {
        mma_bf16(o[2 * q], w[k], b[0], b[1]);
        mma_bf16(o[2 * q + 1], w[k], b[2], b[3]);
      }
    }
  }
  const float D = p.D[h];
#pragma unroll
  for (int i = 0; i < PT / 8; ++i) {
    const int c = i * 8 + (lane & 3) * 2;
    if (p0 + c >= p.P) continue;
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const int row = k ? tb : ta;
      if (row >= rows) continue;
      const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(Xs + row * LDP + c));
      *reinterpret_cast<float2*>(p.out + (int64_t)(t0 + row) * p.H * p.P + (int64_t)h * p.P + p0 + c) =
          make_float2(fmaf(D, x.x, o[i][2 * k]), fmaf(D, x.y, o[i][2 * k + 1]));
    }
  }
}

static size_t sum_smem(int np) { return sizeof(__nv_bfloat16) * ((size_t)L * (np + 8) + 3 * (size_t)L * LDP); }
static size_t out_smem(int np) {
  return sizeof(__nv_bfloat16) * (2 * (size_t)L * (np + 8) + (size_t)L * LDP + 3 * (size_t)np * LDP);
}

}  // namespace ssmtc
}  // namespace atom

ATOM_EXPORT int atom_ssm_tc_supports(int N, int P) { return N > 0 && N % 8 == 0 && N <= 256 && P > 0 && P % 8 == 0 ? 1 : 0; }
ATOM_EXPORT int atom_ssm_tc_chunk(void) { return atom::ssmtc::L; }

// The first (stage 0) and the last (stage 1) of the three launches; sB [ceil(T / 64) + num_seqs, H, N, P] and sA [.., H]
// hold the chunks' sums and, after the prefix over the chunks, the states they begin with.
ATOM_EXPORT int atom_ssm_tc(int stage, float* out, const void* u, const float* dt, const float* la, const float* D,
                            float* sB, float* sA, const int* cu_q, int num_seqs, int T, int H, int G, int N, int P,
                            cudaStream_t stream) {
  using namespace atom::ssmtc;
  if (T <= 0 || num_seqs <= 0) return ATOM_OK;
  if (!atom_ssm_tc_supports(N, P) || H <= 0 || H > 65535 || G <= 0 || H % G || !sB || !sA || ((uintptr_t)u % 16) != 0 ||
      ((uintptr_t)sB % 16) != 0)
    return ATOM_ERR_ARG;
  const int np = (N + 15) & ~15;
  const size_t s0 = sum_smem(np), s1 = out_smem(np);
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(ssm_chunk_sum_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sum_smem(256)) !=
            cudaSuccess ||
        cudaFuncSetAttribute(ssm_chunk_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)out_smem(256)) !=
            cudaSuccess)
      return ATOM_ERR_LAUNCH;
    attr_set = true;
  }
  const Params p{(const __nv_bfloat16*)u, dt, la, D, out, sB, sA, cu_q, num_seqs, H, G, N, P};
  const dim3 grid((T + L - 1) / L + num_seqs, H, (P + PT - 1) / PT);
  if (stage == 0)
    atom::launch_pdl(ssm_chunk_sum_kernel, grid, dim3(THREADS), s0, stream, p);
  else
    atom::launch_pdl(ssm_chunk_out_kernel, grid, dim3(THREADS), s1, stream, p);
  return atom::check_launch();
}
