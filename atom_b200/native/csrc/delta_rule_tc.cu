// The gated delta rule of delta_rule.cu over long portions, in chunks of 64 rows on the tensor cores (bfloat16 q, k, v).
//
// With G_i the sum of the decays' logarithms over a chunk's rows up to i (per key channel), S the state the chunk begins
// with, and  A_ij = sum_c k_i k_j 2^(G_i - G_j),  B_ij = sum_c q_i k_j 2^(G_i - G_j)  (j <= i), the recurrence
//   S <- diag(g_i) S;  u_i = beta_i (v_i - S^T k_i);  S <- S + k_i u_i^T;  o_i = S^T q_i
// over the chunk is, with k~_i = 2^(G_i) k_i, q~_i = 2^(G_i) q_i and k^_j = 2^(G_last - G_j) k_j,
//   (I + diag(beta) A_strictly_lower) [U_v | W] = diag(beta) [V | K~]
//   U = U_v - W S;    O = Q~ S + B_lower U;    S <- diag(2^(G_last)) S + K^T U
//   delta_chunk_prepare_kernel  a CTA per (chunk, head), all chunks side by side: everything that does not need the state.
//       Rows of 16-row block I of A and B take the row before the block as reference: the rows' factor is 2^(sum from the
//       block's first row on), the columns' 2^(sum from the column's next row to the block before) in earlier blocks, and its
//       inverse counterpart 2^-(sum up to the column) within the block, where that stays below 2^60; a block whose decays
//       reach further forms 2^(G_i - G_j) for every pair instead.  Sums run within a block of 16 rows and over whole blocks,
//       so that no difference is one of two large sums (a decay's logarithm counts as -32 at least: 2^-32 of a state is below
//       its last bit).  T = (I + diag(beta) A_strictly_lower)^-1 is formed in 32-bit, block by block, [W | U_v] is T times
//       diag(beta) [K~ | V].
//   delta_chunk_scan_kernel     a CTA per (request, head, 16 value columns) walks the chunks in order.  The transposed state
//       (16 columns x key channels) lies in the accumulators of four warps, a quarter of the channels each, and is the left
//       operand of the products with W and Q~ as it stands (the order of a product's inner index is free, so a lane's
//       accumulators are its operand); partial sums over the quarters meet in shared memory.  The next operands arrive by
//       cp.async meanwhile.
// Products run on mma.sync m16n8k8 in tf32 with every 32-bit operand as two numbers (hi + lo, three products), 32-bit
// sums; state, decays, sums of decays and the system are 32-bit.
#include "common.cuh"

namespace atom {
namespace drtc {

constexpr int C = 64;                    // rows of a chunk
constexpr int PT = 256;                  // threads of the prepare kernel
constexpr int ST = 128;                  // threads of the scan kernel
constexpr int COLS = 16;                 // value columns of a scan CTA
constexpr int LB = C + 8;                // floats per row of B and K^ (transposed)

template <int DKP>
struct Blob {                            // what a (chunk, head) leaves for the scan, in floats
  static constexpr int LW = DKP + 8;
  static constexpr int W = 0;
  static constexpr int Q = W + C * LW;
  static constexpr int KT = Q + C * LW;
  static constexpr int B = KT + DKP * LB;
  static constexpr int GL = B + C * LB;
  static constexpr int UV = GL + DKP;    // [dv][C]
};
template <int DKP>
__host__ __device__ constexpr int64_t blob_floats(int dv) { return Blob<DKP>::UV + (int64_t)dv * C; }

struct Params {
  float* out;                // [T, H dv]
  const __nv_bfloat16* u;    // [T, 2 G dk + H dv]
  const float* rn;           // [T, 2 G]
  const float* la;           // [T, H dk]
  const float* beta;         // [T, H]
  float* state;              // [slots, H, dk, dv]
  float* blobs;              // [chunk slots, H, blob]
  const int* cu_q;
  const int* state_slots;
  int num_seqs, G, H, dk, dv, write_state;
};

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// x = hi + lo with hi and lo of ten mantissa bits (what the tf32 product reads).
__device__ __forceinline__ void split(float x, uint32_t& hi, uint32_t& lo) {
  hi = __float_as_uint(x) & 0xffffe000u;
  lo = __float_as_uint(x - __uint_as_float(hi)) & 0xffffe000u;
}
__device__ __forceinline__ void mma_tf32(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm(
      "mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// d[i] += a b[i] with a and the b[i] as two numbers each (the product of the two small parts is left out); the products of
// one accumulator stand apart.
template <int N>
__device__ __forceinline__ void mma_split(float (*const (&d)[N])[4], const uint32_t (&ah)[4], const uint32_t (&al)[4],
                                          const float2 (&b)[N]) {
  uint32_t h0[N], l0[N], h1[N], l1[N];
#pragma unroll
  for (int i = 0; i < N; ++i) {
    split(b[i].x, h0[i], l0[i]);
    split(b[i].y, h1[i], l1[i]);
  }
#pragma unroll
  for (int i = 0; i < N; ++i) mma_tf32(*d[i], ah, l0[i], l1[i]);
#pragma unroll
  for (int i = 0; i < N; ++i) mma_tf32(*d[i], al, h0[i], h1[i]);
#pragma unroll
  for (int i = 0; i < N; ++i) mma_tf32(*d[i], ah, h0[i], h1[i]);
}
__device__ __forceinline__ void cp_async16(void* smem, const void* gmem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(s), "l"(gmem));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N)); }

// ------------------------------------------------------------------ what does not need the state

template <int DKP>
struct PrepSmem {
  static constexpr int LG = DKP + 4, LK = DKP + 8, LT = C + 4;
  float g[C * LG];                       // sums of the decays' logarithms from the row's block of 16 rows on
  float off[14 * DKP];                   // rows (I, J), J < I <= 4: the sum over blocks J .. I-1; then over the blocks before I
  float a[C * LB];                       // [j][i] = beta_i A_ij for i > j, zero for the other i of j's 16-row block
  float t[C * LT];                       // T
  __nv_bfloat16 k[C * LK], q[C * LK];
  float rk[C], rq[C], rb[C], beta[C];    // rb: rk * beta
  int strong[4];                         // a channel of the block decays beyond 2^-60
};

__device__ __forceinline__ constexpr int off_row(int I, int J) { return I * (I - 1) / 2 + J; }

template <int DKP>
__global__ void __launch_bounds__(PT, 2) delta_chunk_prepare_kernel(const Params p) {
  atom::pdl_trigger();
  atom::pdl_wait();
  extern __shared__ __align__(16) unsigned char dc_smem[];
  PrepSmem<DKP>& sm = *reinterpret_cast<PrepSmem<DKP>*>(dc_smem);
  constexpr int LG = PrepSmem<DKP>::LG, LK = PrepSmem<DKP>::LK;
  using BL = Blob<DKP>;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int hd = blockIdx.y, H = p.H, G = p.G, dk = p.dk, dv = p.dv, g = hd / (H / G);
  int s, r = 0, acc = 0;
  for (s = 0; s < p.num_seqs; ++s) {
    const int n_chunks = (p.cu_q[s + 1] - p.cu_q[s] + C - 1) / C;
    if ((int)blockIdx.x < acc + n_chunks) {
      r = blockIdx.x - acc;
      break;
    }
    acc += n_chunks;
  }
  if (s >= p.num_seqs) return;
  const int64_t t0 = p.cu_q[s] + r * C;
  const int n = min(C, p.cu_q[s + 1] - (int)t0);
  const int nb = (n + 15) / 16;                             // 16-row blocks with rows
  const int64_t CU = 2 * (int64_t)G * dk + (int64_t)H * dv;
  float* blob = p.blobs + ((int64_t)blockIdx.x * H + hd) * blob_floats<DKP>(dv);

  // rows into shared memory; rows behind the last and channels behind dk are zero (no decay, no write)
  if (tid < 4) sm.strong[tid] = 0;
  if (dk % 8 == 0 && CU % 8 == 0 && ((uintptr_t)p.u % 16) == 0 && ((uintptr_t)p.la % 16) == 0) {
#pragma unroll 4
    for (int e = tid; e < C * DKP / 8; e += PT) {
      const int i = e / (DKP / 8), c = (e - i * (DKP / 8)) * 8;
      const bool in = i < n && c < dk;
      const int64_t t = t0 + (in ? i : 0);
      uint4 qv = make_uint4(0u, 0u, 0u, 0u), kv = qv;
      float4 l0 = make_float4(0.f, 0.f, 0.f, 0.f), l1 = l0;
      if (in) {
        qv = *reinterpret_cast<const uint4*>(p.u + t * CU + (int64_t)g * dk + c);
        kv = *reinterpret_cast<const uint4*>(p.u + t * CU + (int64_t)(G + g) * dk + c);
        l0 = *reinterpret_cast<const float4*>(p.la + (t * H + hd) * dk + c);
        l1 = *reinterpret_cast<const float4*>(p.la + (t * H + hd) * dk + c + 4);
      }
      *reinterpret_cast<uint4*>(sm.q + i * LK + c) = qv;
      *reinterpret_cast<uint4*>(sm.k + i * LK + c) = kv;
      *reinterpret_cast<float4*>(sm.g + i * LG + c) =
          make_float4(fmaxf(l0.x, -32.f), fmaxf(l0.y, -32.f), fmaxf(l0.z, -32.f), fmaxf(l0.w, -32.f));
      *reinterpret_cast<float4*>(sm.g + i * LG + c + 4) =
          make_float4(fmaxf(l1.x, -32.f), fmaxf(l1.y, -32.f), fmaxf(l1.z, -32.f), fmaxf(l1.w, -32.f));
    }
  } else {
    for (int e = tid; e < C * DKP; e += PT) {
      const int i = e / DKP, c = e - i * DKP;
      const bool in = i < n && c < dk;
      const int64_t t = t0 + (in ? i : 0);
      sm.g[i * LG + c] = in ? fmaxf(p.la[(t * H + hd) * dk + c], -32.f) : 0.f;
      sm.q[i * LK + c] = in ? p.u[t * CU + (int64_t)g * dk + c] : __float2bfloat16_rn(0.f);
      sm.k[i * LK + c] = in ? p.u[t * CU + (int64_t)(G + g) * dk + c] : __float2bfloat16_rn(0.f);
    }
  }
  for (int i = tid; i < C; i += PT) {
    const int64_t t = t0 + i;
    sm.rq[i] = i < n ? p.rn[t * 2 * G + g] : 0.f;
    sm.rk[i] = i < n ? p.rn[t * 2 * G + G + g] : 0.f;
    sm.beta[i] = i < n ? p.beta[t * H + hd] : 0.f;
    sm.rb[i] = sm.rk[i] * sm.beta[i];
  }
  __syncthreads();
  for (int e = tid; e < 4 * DKP; e += PT) {
    const int b = e / DKP, c = e - b * DKP;
    float v[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) v[i] = sm.g[(b * 16 + i) * LG + c];
#pragma unroll
    for (int i = 1; i < 16; ++i) v[i] += v[i - 1];
#pragma unroll
    for (int i = 1; i < 16; ++i) sm.g[(b * 16 + i) * LG + c] = v[i];
    if (v[15] < -60.f) sm.strong[b] = 1;
  }
  __syncthreads();
  for (int c = tid; c < DKP; c += PT) {
    float tot[4], before = 0.f;
#pragma unroll
    for (int b = 0; b < 4; ++b) tot[b] = sm.g[(16 * b + 15) * LG + c];
#pragma unroll
    for (int b = 0; b < 4; ++b) {
      sm.off[(10 + b) * DKP + c] = before;
      before += tot[b];
      float sum = 0.f;
#pragma unroll
      for (int I = b + 1; I <= 4; ++I) {
        sum += tot[I - 1];
        sm.off[off_row(I, b) * DKP + c] = sum;
      }
    }
  }
  __syncthreads();
  const float* pre = sm.off + 10 * DKP;                     // (row 10 is zero)

  // A and B: a warp takes up to three tiles of 8 columns of one row block (block 3: 8 tiles, 2: 6, 1: 4, 0: 2)
  const int gq = lane >> 2, tq = lane & 3;
  {
    const int I = warp < 3 ? 3 : (warp < 5 ? 2 : (warp < 7 ? 1 : 0));
    const int jt0 = warp < 3 ? 3 * warp : (warp < 5 ? 3 * (warp - 3) : (warp < 7 ? 2 * (warp - 5) : 0));
    const int tiles = warp == 2 || warp >= 5 ? 2 : 3;
    const bool strong = sm.strong[I] != 0;
    const int ia = 16 * I + gq, ib = ia + 8;
    float da[3][4], db[3][4];
#pragma unroll
    for (int x = 0; x < 3; ++x)
#pragma unroll
      for (int e = 0; e < 4; ++e) da[x][e] = db[x][e] = 0.f;
    if (I < nb) {
      const float *orow[3], *grow[3];
      const __nv_bfloat16* krow[3];
      float live[3];
#pragma unroll
      for (int x = 0; x < 3; ++x) {
        const int jt = min(jt0 + x, 2 * I + 1), J = jt >> 1, jc = jt * 8 + gq;
        orow[x] = J < I ? sm.off + off_row(I, J) * DKP + tq : pre + tq;
        grow[x] = sm.g + jc * LG + tq;
        krow[x] = sm.k + jc * LK + tq;
        live[x] = J == I && strong ? 0.f : 1.f;             // (then formed pair by pair below)
      }
      const float *ga = sm.g + ia * LG + tq, *gb = sm.g + ib * LG + tq;
      const __nv_bfloat16 *ka = sm.k + ia * LK + tq, *kb = sm.k + ib * LK + tq;
      const __nv_bfloat16 *qa = sm.q + ia * LK + tq, *qb = sm.q + ib * LK + tq;
#pragma unroll 2
      for (int kk = 0; kk < DKP; kk += 8) {
        uint32_t kh[4], kl[4], qh[4], ql[4];
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const float fa = ex2(ga[kk + 4 * h]), fb = ex2(gb[kk + 4 * h]);
          split(__bfloat162float(ka[kk + 4 * h]) * fa, kh[2 * h], kl[2 * h]);
          split(__bfloat162float(kb[kk + 4 * h]) * fb, kh[2 * h + 1], kl[2 * h + 1]);
          split(__bfloat162float(qa[kk + 4 * h]) * fa, qh[2 * h], ql[2 * h]);
          split(__bfloat162float(qb[kk + 4 * h]) * fb, qh[2 * h + 1], ql[2 * h + 1]);
        }
        float2 bv[3];
#pragma unroll
        for (int x = 0; x < 3; ++x)
          bv[x] = make_float2(__bfloat162float(krow[x][kk]) * ex2((orow[x][kk] - grow[x][kk]) * live[x]),
                              __bfloat162float(krow[x][kk + 4]) * ex2((orow[x][kk + 4] - grow[x][kk + 4]) * live[x]));
        mma_split<3>({&da[0], &da[1], &da[2]}, kh, kl, bv);
        mma_split<3>({&db[0], &db[1], &db[2]}, qh, ql, bv);
      }
    }
#pragma unroll
    for (int x = 0; x < 3; ++x) {
      if (x < tiles && !(strong && (jt0 + x) >> 1 == I)) {
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int i = h ? ib : ia, j = (jt0 + x) * 8 + 2 * tq;
          float2 bo;
          sm.a[j * LB + i] = i > j ? da[x][2 * h] * sm.rk[i] * sm.rk[j] * sm.beta[i] : 0.f;
          sm.a[(j + 1) * LB + i] = i > j + 1 ? da[x][2 * h + 1] * sm.rk[i] * sm.rk[j + 1] * sm.beta[i] : 0.f;
          bo.x = i >= j ? db[x][2 * h] * sm.rq[i] * sm.rk[j] : 0.f;
          bo.y = i >= j + 1 ? db[x][2 * h + 1] * sm.rq[i] * sm.rk[j + 1] : 0.f;
          *reinterpret_cast<float2*>(blob + BL::B + i * LB + j) = bo;
        }
      }
    }
  }
  for (int blk = 0; blk < 4; ++blk) {
    if (!sm.strong[blk]) continue;                          // (the same for all threads)
    const int i = blk * 16 + (tid >> 4), j = blk * 16 + (tid & 15);
    float sa = 0.f, sb = 0.f;
    if (j <= i) {
      for (int c = 0; c < DKP; ++c) {
        const float w = __bfloat162float(sm.k[j * LK + c]) * ex2(sm.g[i * LG + c] - sm.g[j * LG + c]);
        sa = fmaf(__bfloat162float(sm.k[i * LK + c]), w, sa);
        sb = fmaf(__bfloat162float(sm.q[i * LK + c]), w, sb);
      }
    }
    sm.a[j * LB + i] = i > j ? sa * sm.rk[i] * sm.rk[j] * sm.beta[i] : 0.f;
    blob[BL::B + i * LB + j] = sb * sm.rq[i] * sm.rk[j];
  }
  __syncthreads();

  if (warp < 2) {
    // T: the blocks on the diagonal, a thread per column (once x_j stands, every later row loses beta_i A_ij x_j), then
    // block diagonal by block diagonal  T_IJ = -T_II sum_K L_IK T_KJ  (the sum waits in T's unused block (J, I))
    constexpr int LT = PrepSmem<DKP>::LT;
    {
      const int b = tid >> 4, c = tid & 15;
      float x[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) x[i] = i == c ? 1.f : 0.f;
#pragma unroll
      for (int j = 0; j < 15; ++j) {
#pragma unroll
        for (int i4 = (j + 1) / 4; i4 < 4; ++i4) {
          const float4 l = *reinterpret_cast<const float4*>(sm.a + (16 * b + j) * LB + 16 * b + i4 * 4);   // (zero where i <= j)
          x[4 * i4] = fmaf(-l.x, x[j], x[4 * i4]);
          x[4 * i4 + 1] = fmaf(-l.y, x[j], x[4 * i4 + 1]);
          x[4 * i4 + 2] = fmaf(-l.z, x[j], x[4 * i4 + 2]);
          x[4 * i4 + 3] = fmaf(-l.w, x[j], x[4 * i4 + 3]);
        }
      }
#pragma unroll
      for (int i = 0; i < 16; ++i) sm.t[(16 * b + i) * LT + 16 * b + c] = x[i];
    }
    const int c = tid & 15, r = (tid >> 4) * 4;              // a column, four rows of a block
#pragma unroll 1
    for (int d = 1; d < 4; ++d) {
      asm volatile("bar.sync 2, 64;\n" ::: "memory");
#pragma unroll 1
      for (int J = 0; J + d < 4; ++J) {
        const int I = J + d;
        float m[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 8
        for (int j = 16 * J; j < 16 * I; ++j) {
          const float4 l = *reinterpret_cast<const float4*>(sm.a + j * LB + 16 * I + r);
          const float y = sm.t[j * LT + 16 * J + c];
          m[0] = fmaf(l.x, y, m[0]);
          m[1] = fmaf(l.y, y, m[1]);
          m[2] = fmaf(l.z, y, m[2]);
          m[3] = fmaf(l.w, y, m[3]);
        }
#pragma unroll
        for (int q = 0; q < 4; ++q) sm.t[(16 * J + r + q) * LT + 16 * I + c] = m[q];
      }
      asm volatile("bar.sync 2, 64;\n" ::: "memory");
#pragma unroll 1
      for (int J = 0; J + d < 4; ++J) {
        const int I = J + d;
        float o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 8
        for (int k = 0; k < 16; ++k) {
          const float y = sm.t[(16 * J + k) * LT + 16 * I + c];
#pragma unroll
          for (int q = 0; q < 4; ++q) o[q] = fmaf(-sm.t[(16 * I + r + q) * LT + 16 * I + k], y, o[q]);
        }
#pragma unroll
        for (int q = 0; q < 4; ++q) sm.t[(16 * I + r + q) * LT + 16 * J + c] = o[q];
      }
    }
  } else {
    // meanwhile: Q~, K^ transposed, the whole chunk's decays
    const int w = tid - 64;
    constexpr int NW = PT - 64;
#pragma unroll 2
    for (int e = w; e < C * DKP / 4; e += NW) {
      const int i = e / (DKP / 4), c = (e - i * (DKP / 4)) * 4;
      const float4 gl = *reinterpret_cast<const float4*>(sm.g + i * LG + c);
      const float4 pr = *reinterpret_cast<const float4*>(pre + (i / 16) * DKP + c);
      const uint2 qv = *reinterpret_cast<const uint2*>(sm.q + i * LK + c);
      const float2 q0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&qv.x));
      const float2 q1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&qv.y));
      const float f = sm.rq[i];
      *reinterpret_cast<float4*>(blob + BL::Q + i * BL::LW + c) =
          make_float4(q0.x * f * ex2(pr.x + gl.x), q0.y * f * ex2(pr.y + gl.y), q1.x * f * ex2(pr.z + gl.z),
                      q1.y * f * ex2(pr.w + gl.w));
    }
#pragma unroll 1
    for (int e = w; e < DKP * (C / 8); e += NW) {
      const int j8 = e / DKP, c = e - j8 * DKP;             // (eight rows of one block)
      const float d = sm.off[off_row(4, j8 / 2) * DKP + c];
      float o[8];
#pragma unroll
      for (int x = 0; x < 8; ++x) {
        const int j = j8 * 8 + x;
        o[x] = __bfloat162float(sm.k[j * LK + c]) * sm.rk[j] * ex2(d - sm.g[j * LG + c]);
      }
      float* dst = blob + BL::KT + c * LB + j8 * 8;
      *reinterpret_cast<float4*>(dst) = make_float4(o[0], o[1], o[2], o[3]);
      *reinterpret_cast<float4*>(dst + 4) = make_float4(o[4], o[5], o[6], o[7]);
    }
    // the values into the place of the queries
    asm volatile("bar.sync 1, %0;\n" ::"n"(PT - 64) : "memory");
    const __nv_bfloat16* v = p.u + t0 * CU + 2 * (int64_t)G * dk + (int64_t)hd * dv;
    const int dvs = min(dv, DKP);
    if (dk % 4 == 0 && dv % 8 == 0 && ((uintptr_t)p.u % 16) == 0) {
#pragma unroll 4
      for (int e = w; e < C * DKP / 8; e += NW) {
        const int i = e / (DKP / 8), c = (e - i * (DKP / 8)) * 8;
        if (c < dvs)
          *reinterpret_cast<uint4*>(sm.q + i * LK + c) =
              i < n ? *reinterpret_cast<const uint4*>(v + (int64_t)i * CU + c) : make_uint4(0u, 0u, 0u, 0u);
      }
    } else {
      for (int e = w; e < C * DKP; e += NW) {
        const int i = e / DKP, c = e - i * DKP;
        if (c < dvs) sm.q[i * LK + c] = i < n ? v[(int64_t)i * CU + c] : __float2bfloat16_rn(0.f);
      }
    }
    for (int c = w; c < DKP; c += NW) blob[BL::GL + c] = ex2(sm.off[off_row(4, 0) * DKP + c]);
  }
  __syncthreads();

  // [W | U_v] = T diag(beta) [K~ | V]: a warp four tiles of 8 columns at a time, all rows
  for (int base = warp * 32; base < DKP + dv; base += PT) {
    const bool keys = base < DKP;
    float acc[4][4][4];
#pragma unroll
    for (int I = 0; I < 4; ++I)
#pragma unroll
      for (int x = 0; x < 4; ++x)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[I][x][e] = 0.f;
    const __nv_bfloat16* v = p.u + t0 * CU + 2 * (int64_t)G * dk + (int64_t)hd * dv - DKP;
#pragma unroll 1
    for (int ks = 0; ks < C / 8; ++ks) {
      float2 bv[4];
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int col = base + 8 * x + gq;
        float w[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int j = 8 * ks + tq + 4 * e;
          if (keys)
            w[e] = __bfloat162float(sm.k[j * LK + col]) * sm.rb[j] * ex2(pre[(j / 16) * DKP + col] + sm.g[j * LG + col]);
          else if (base < 2 * DKP)                           // (values beyond dv: whatever lies there, not stored)
            w[e] = __bfloat162float(sm.q[j * LK + col - DKP]) * sm.beta[j];
          else
            w[e] = j < n && col < DKP + dv ? __bfloat162float(v[(int64_t)j * CU + col]) * sm.beta[j] : 0.f;
        }
        bv[x] = make_float2(w[0], w[1]);
      }
#pragma unroll
      for (int I = 0; I < 4; ++I) {
        if (I < ks / 2) continue;                            // (zero above the diagonal's blocks)
        uint32_t th[4], tl[4];
#pragma unroll
        for (int e = 0; e < 4; ++e)
          split(sm.t[(16 * I + gq + (e & 1) * 8) * PrepSmem<DKP>::LT + 8 * ks + tq + (e >> 1) * 4], th[e], tl[e]);
        mma_split<4>({&acc[I][0], &acc[I][1], &acc[I][2], &acc[I][3]}, th, tl, bv);
      }
    }
#pragma unroll
    for (int I = 0; I < 4; ++I) {
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int col = base + 8 * x + 2 * tq, i = 16 * I + gq;
        if (keys) {
          *reinterpret_cast<float2*>(blob + BL::W + i * BL::LW + col) = make_float2(acc[I][x][0], acc[I][x][1]);
          *reinterpret_cast<float2*>(blob + BL::W + (i + 8) * BL::LW + col) = make_float2(acc[I][x][2], acc[I][x][3]);
        } else {
          float* dst = blob + BL::UV + (int64_t)(col - DKP) * C + i;
          if (col < DKP + dv) {
            dst[0] = acc[I][x][0];
            dst[8] = acc[I][x][2];
          }
          if (col + 1 < DKP + dv) {
            dst[C] = acc[I][x][1];
            dst[C + 8] = acc[I][x][3];
          }
        }
      }
    }
  }
}

// ------------------------------------------------------------------ the walk over the chunks

template <int DKP>
struct ScanSmem {
  float wq[2][2 * C * (DKP + 8)];        // W and Q~ of two chunks
  float kb[DKP * LB + C * LB + DKP];     // K^ transposed, B, decays of one
  float part[4 * COLS * LB];             // partial sums of -U, a warp each
  float opart[4 * COLS * LB];            // partial outputs
};

template <int DKP>
__global__ void __launch_bounds__(ST, 1) delta_chunk_scan_kernel(const Params p) {
  atom::pdl_trigger();
  atom::pdl_wait();
  extern __shared__ __align__(16) unsigned char dc_smem[];
  ScanSmem<DKP>& sm = *reinterpret_cast<ScanSmem<DKP>*>(dc_smem);
  using BL = Blob<DKP>;
  constexpr int LW = BL::LW, KS = DKP / 32;                 // 8-channel steps of a warp's quarter
  const int s = blockIdx.x, hd = blockIdx.y, col0 = blockIdx.z * COLS;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
  const int first = p.cu_q[s], len = p.cu_q[s + 1] - first;
  if (len <= 0) return;
  const int H = p.H, dk = p.dk, dv = p.dv;
  int x0 = 0;
  for (int q = 0; q < s; ++q) x0 += (p.cu_q[q + 1] - p.cu_q[q] + C - 1) / C;
  const int n_chunks = (len + C - 1) / C;
  const int64_t bf = blob_floats<DKP>(dv);
  const float* blob0 = p.blobs + ((int64_t)x0 * H + hd) * bf;
  auto blob_of = [&](int c) { return blob0 + (int64_t)c * H * bf; };

  auto load = [&](float* dst, const float* src, int floats) {
    for (int e = tid * 4; e < floats; e += ST * 4) cp_async16(dst + e, src + e);
  };
  load(sm.wq[0], blob_of(0) + BL::W, 2 * C * LW);
  cp_async_commit();

  // the transposed state: rows (value columns) gq and gq + 8, channels c0 + 8 nt + 2 tq and the next
  const int c0 = warp * (DKP / 4);
  const int ja = col0 + gq, jb = ja + 8;
  float* S_g = p.state + ((int64_t)p.state_slots[s] * H + hd) * dk * dv;
  float S[KS][4];
#pragma unroll
  for (int nt = 0; nt < KS; ++nt) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = c0 + 8 * nt + 2 * tq + (e & 1), j = e < 2 ? ja : jb;
      S[nt][e] = c < dk && j < dv ? S_g[(int64_t)c * dv + j] : 0.f;
    }
  }
  // U_v of a warp's quarter of the rows, one chunk ahead
  float uv[2][4];
  auto load_uv = [&](int c) {
    const float* src = blob_of(c) + BL::UV + 16 * warp + 2 * tq;
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      float2 a = make_float2(0.f, 0.f), b = a;
      if (ja < dv) a = *reinterpret_cast<const float2*>(src + (int64_t)ja * C + 8 * x);
      if (jb < dv) b = *reinterpret_cast<const float2*>(src + (int64_t)jb * C + 8 * x);
      uv[x][0] = a.x;
      uv[x][1] = a.y;
      uv[x][2] = b.x;
      uv[x][3] = b.y;
    }
  };
  load_uv(0);
  cp_async_wait<0>();
  __syncthreads();

  for (int ch = 0; ch < n_chunks; ++ch) {
    const float* blob = blob_of(ch);
    load(sm.kb, blob + BL::KT, DKP * LB + C * LB + DKP);
    cp_async_commit();
    if (ch + 1 < n_chunks) load(sm.wq[(ch + 1) & 1], blob_of(ch + 1) + BL::W, 2 * C * LW);
    cp_async_commit();
    const float* Ws = sm.wq[ch & 1];
    const float* Qs = Ws + C * LW;

    // -U and O over the warp's quarter of the channels; a warp also takes -U_v of a quarter of the rows
    float u[C / 8][4], o[C / 8][4];
#pragma unroll
    for (int nt = 0; nt < C / 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        u[nt][e] = nt / 2 == warp ? -uv[nt & 1][e] : 0.f;
        o[nt][e] = 0.f;
      }
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      uint32_t ah[4], al[4];
      split(S[ks][0], ah[0], al[0]);
      split(S[ks][2], ah[1], al[1]);
      split(S[ks][1], ah[2], al[2]);
      split(S[ks][3], ah[3], al[3]);
      const int at = c0 + 8 * ks + 2 * tq;
#pragma unroll
      for (int nt = 0; nt < C / 8; nt += 4) {
        float2 w[4], q[4];
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          w[x] = *reinterpret_cast<const float2*>(Ws + (8 * (nt + x) + gq) * LW + at);
          q[x] = *reinterpret_cast<const float2*>(Qs + (8 * (nt + x) + gq) * LW + at);
        }
        mma_split<4>({&u[nt], &u[nt + 1], &u[nt + 2], &u[nt + 3]}, ah, al, w);
        mma_split<4>({&o[nt], &o[nt + 1], &o[nt + 2], &o[nt + 3]}, ah, al, q);
      }
    }
    float* mine = sm.part + warp * COLS * LB;
#pragma unroll
    for (int nt = 0; nt < C / 8; ++nt) {
      *reinterpret_cast<float2*>(mine + gq * LB + 8 * nt + 2 * tq) = make_float2(u[nt][0], u[nt][1]);
      *reinterpret_cast<float2*>(mine + (gq + 8) * LB + 8 * nt + 2 * tq) = make_float2(u[nt][2], u[nt][3]);
    }
    cp_async_wait<1>();
    __syncthreads();                                        // partial sums stand, K^ and B are here

    if (ch + 1 < n_chunks) load_uv(ch + 1);
    const float* KTs = sm.kb;
    const float* Bs = KTs + DKP * LB;
    const float* GLs = Bs + C * LB;
#pragma unroll
    for (int nt = 0; nt < KS; ++nt) {
      const float2 gl = *reinterpret_cast<const float2*>(GLs + c0 + 8 * nt + 2 * tq);
      S[nt][0] *= gl.x;
      S[nt][1] *= gl.y;
      S[nt][2] *= gl.x;
      S[nt][3] *= gl.y;
    }
#pragma unroll
    for (int js = 0; js < C / 8; ++js) {
      float2 a = make_float2(0.f, 0.f), b = a;
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        const float2 x = *reinterpret_cast<const float2*>(sm.part + (w * COLS + gq) * LB + 8 * js + 2 * tq);
        const float2 y = *reinterpret_cast<const float2*>(sm.part + (w * COLS + gq + 8) * LB + 8 * js + 2 * tq);
        a.x -= x.x;
        a.y -= x.y;
        b.x -= y.x;
        b.y -= y.y;
      }
      uint32_t ah[4], al[4];
      split(a.x, ah[0], al[0]);
      split(b.x, ah[1], al[1]);
      split(a.y, ah[2], al[2]);
      split(b.y, ah[3], al[3]);
      const int at = 8 * js + 2 * tq;
      // the state, and O += B_lower U for the warp's row blocks: warp and 7 - warp
      float2 k[KS];
      float(*d[KS])[4];
#pragma unroll
      for (int nt = 0; nt < KS; ++nt) {
        k[nt] = *reinterpret_cast<const float2*>(KTs + (c0 + 8 * nt + gq) * LB + at);
        d[nt] = &S[nt];
      }
      mma_split<KS>(d, ah, al, k);
#pragma unroll
      for (int nt = 0; nt < C / 8; ++nt) {
        if ((nt == warp || nt == 7 - warp) && js <= nt) {
          const float2 x[1] = {*reinterpret_cast<const float2*>(Bs + (8 * nt + gq) * LB + at)};
          mma_split<1>({&o[nt]}, ah, al, x);
        }
      }
    }
    float* omine = sm.opart + warp * COLS * LB;
#pragma unroll
    for (int nt = 0; nt < C / 8; ++nt) {
      *reinterpret_cast<float2*>(omine + gq * LB + 8 * nt + 2 * tq) = make_float2(o[nt][0], o[nt][1]);
      *reinterpret_cast<float2*>(omine + (gq + 8) * LB + 8 * nt + 2 * tq) = make_float2(o[nt][2], o[nt][3]);
    }
    cp_async_wait<0>();
    __syncthreads();                                        // outputs stand, K^ and B are free, the next W and Q~ are here
    {
      const int i = tid & (C - 1), half = tid / C;          // a row, 8 of the 16 columns
      const int row = ch * C + i;
      if (row < len) {
        float r[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          r[e] = 0.f;
#pragma unroll
          for (int w = 0; w < 4; ++w) r[e] += sm.opart[(w * COLS + half * 8 + e) * LB + i];
        }
        float* dst = p.out + ((int64_t)(first + row) * H + hd) * dv + col0 + half * 8;
        if (col0 + half * 8 + 8 <= dv && dv % 4 == 0) {
          *reinterpret_cast<float4*>(dst) = make_float4(r[0], r[1], r[2], r[3]);
          *reinterpret_cast<float4*>(dst + 4) = make_float4(r[4], r[5], r[6], r[7]);
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e)
            if (col0 + half * 8 + e < dv) dst[e] = r[e];
        }
      }
    }
  }
  if (!p.write_state) return;
#pragma unroll
  for (int nt = 0; nt < KS; ++nt) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = c0 + 8 * nt + 2 * tq + (e & 1), j = e < 2 ? ja : jb;
      if (c < dk && j < dv) S_g[(int64_t)c * dv + j] = S[nt][e];
    }
  }
}

template <int DKP>
static int launch(const Params& p, int T, cudaStream_t stream) {
  const int slots = (T + C - 1) / C + p.num_seqs;           // an upper bound of the chunks
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(delta_chunk_prepare_kernel<DKP>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                             (int)sizeof(PrepSmem<DKP>)) != cudaSuccess ||
        cudaFuncSetAttribute(delta_chunk_scan_kernel<DKP>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                             (int)sizeof(ScanSmem<DKP>)) != cudaSuccess)
      return ATOM_ERR_LAUNCH;
    attr_set = true;
  }
  atom::launch_pdl(delta_chunk_prepare_kernel<DKP>, dim3(slots, p.H), dim3(PT), sizeof(PrepSmem<DKP>), stream, p);
  atom::launch_pdl(delta_chunk_scan_kernel<DKP>, dim3(p.num_seqs, p.H, (p.dv + COLS - 1) / COLS), dim3(ST),
                   sizeof(ScanSmem<DKP>), stream, p);
  return atom::check_launch();
}

static int pad_of(int dk) { return dk <= 32 ? 32 : (dk <= 64 ? 64 : (dk <= 96 ? 96 : 128)); }

}  // namespace drtc
}  // namespace atom

ATOM_EXPORT int atom_delta_chunk_supports(int dk, int dv) { return dk > 0 && dk <= 128 && dv > 0 ? 1 : 0; }

// Floats that a (chunk, head) leaves in the scratch.
ATOM_EXPORT int atom_delta_chunk_floats(int dk, int dv) {
  using namespace atom::drtc;
  switch (pad_of(dk)) {
    case 32: return (int)blob_floats<32>(dv);
    case 64: return (int)blob_floats<64>(dv);
    case 96: return (int)blob_floats<96>(dv);
    default: return (int)blob_floats<128>(dv);
  }
}

// blobs: (ceil(T / 64) + num_seqs) * H * atom_delta_chunk_floats(dk, dv) floats, 16-byte aligned; u: bfloat16.
ATOM_EXPORT int atom_delta_chunks(float* out, const void* u, const float* rn, const float* la, const float* beta, float* state,
                                  float* blobs, const int* cu_q, const int* state_slots, int num_seqs, int T, int G, int H,
                                  int dk, int dv, int write_state, cudaStream_t stream) {
  using namespace atom::drtc;
  if (T <= 0 || num_seqs <= 0) return ATOM_OK;
  if (!atom_delta_chunk_supports(dk, dv) || G <= 0 || H <= 0 || H % G || H > 65535 || !blobs || ((uintptr_t)blobs % 16) ||
      ((uintptr_t)out % 16))
    return ATOM_ERR_ARG;
  const Params p{out, (const __nv_bfloat16*)u, rn, la, beta, state, blobs, cu_q, state_slots, num_seqs, G, H, dk, dv, write_state};
  switch (pad_of(dk)) {
    case 32: return launch<32>(p, T, stream);
    case 64: return launch<64>(p, T, stream);
    case 96: return launch<96>(p, T, stream);
    default: return launch<128>(p, T, stream);
  }
}
