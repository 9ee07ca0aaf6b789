// Grouped-query attention behind a short causal convolution, with capped scores and a sliding window that
// always keeps a request's first tokens.  Key size and value size may differ.
//
//   conv_rope_write_kernel    per token: the convolution over time on every channel of [q | k | v]
//                               y_t[c] = sum_j w[c, j] * u_(t - taps + 1 + j)[c]        (zeros before the request's start)
//                             with rows before the step's first token of a request taken from the request's
//                             convolution state (its last taps - 1 projected rows); rotation of the first rot_dims
//                             numbers of every query and key head by position * frequency (pairs (i, i + rot_dims/2),
//                             or neighbours (2i, 2i + 1)), cos and sin times a constant; optionally a bias on every
//                             channel (without a convolution), and values blended with another layer's values of
//                             the same token, v <- (1 - mix) v + mix v_first; optionally every query and key head
//                             divided by its root mean square and times a weight before the rotation; q to a dense
//                             array, k and v to their pages (conv_rope_write_vec_kernel: the same for bfloat16 sizes
//                             in steps of 8, 16 bytes at a time).  Keys and values may have head counts of their own.
//   conv_state_update_kernel  per request: the last taps - 1 projected rows after this step
//   window_attention_kernel   one CTA per (token, query head): keys j <= p with p - j < window or j < keep_first,
//                             s = scale * q.k, s <- cap * tanh(s / cap), online softmax in 32-bit; any sizes, both
//                             precisions; optionally a sink per head (exp(sink_h) is added to the denominator), a
//                             gate number per head (the output times sigmoid(gate)) and a constant on the output.
//                             A window may also be a chunk: keys j <= p with j / window = p / window.
//                             With two maps (differential attention) every head has two queries and every key head two
//                             keys, [map 1, map 2], over the same values: o = a1 - lambda a2 with a1, a2 the two maps'
//                             outputs, divided by its root mean square over the value size
// Convolution sums, angles, scores, weights and sums are 32-bit in both precisions.
#include "common.cuh"

namespace atom {

// Row t' (an index into the step's rows, possibly before the request's first row of this step) of channel c.
template <typename T>
__device__ __forceinline__ float conv_input(const T* __restrict__ qkv, int64_t ld, const T* __restrict__ state_row,
                                            int C, int taps, int first, int tp, int c) {
  if (tp >= first) return to_float(qkv[(int64_t)tp * ld + c]);
  const int d = first - tp;                       // 1 .. taps - 1 rows before the step
  return state_row ? to_float(state_row[(int64_t)(taps - 1 - d) * C + c]) : 0.f;
}

template <typename T>
__device__ __forceinline__ float conv_at(const T* __restrict__ qkv, int64_t ld, const T* __restrict__ state_row, int C,
                                         int taps, const void* __restrict__ w, int w_dtype, int first, int t, int c) {
  if (taps <= 0) return to_float(qkv[(int64_t)t * ld + c]);
  float y = 0.f;
  for (int j = 0; j < taps; ++j)
    y += load_as_float(w, w_dtype, (int64_t)c * taps + j) * conv_input(qkv, ld, state_row, C, taps, first, t - taps + 1 + j, c);
  return y;
}

// What the kernels below take beside the convolution and the plain rotation.
struct RopeExtras {
  const void* bias;      // [C] added to every projected channel (null: none; not together with a convolution)
  int bias_dtype;
  int neighbours;        // 1: rotated pairs are (2i, 2i + 1); 0: (i, i + rot_dims / 2)
  float mag;             // factor on cos and sin
  const void* v_first;   // [T, G dv] dense, activation type: values to blend in (null: none)
  float v_mix;
  void* v_keep;          // [T, GV dv] dense: takes a copy of this layer's values (null: none)
  int GV;                // value heads
  const void* wq;        // [dk] weights of the norm of every query and key head (null: none)
  const void* wk;
  int norm_dtype;
  float norm_eps;
};

template <typename T>
__global__ void __launch_bounds__(256)
conv_rope_write_kernel(T* __restrict__ q_out, const T* __restrict__ qkv, int64_t ld, int H, int G, int dk, int dv,
                       const void* __restrict__ conv_w, int w_dtype, int taps, const T* __restrict__ conv_state,
                       const float* __restrict__ freq, int rot_dims, const int* __restrict__ positions,
                       const int* __restrict__ seq_of_token, const int* __restrict__ cu_q,
                       const int* __restrict__ state_slots, const int* __restrict__ block_table, int max_pages,
                       int page_size, T* __restrict__ k_pages, T* __restrict__ v_pages, int64_t num_pages,
                       int* __restrict__ status, const RopeExtras x) {
  atom::pdl_trigger();
  atom::pdl_wait();
  const int t = blockIdx.x;
  const int s = seq_of_token[t];
  if (s < 0) return;
  const int p = positions[t];
  const int first = cu_q[s];
  const int C = H * dk + G * dk + x.GV * dv;
  const T* state_row = (conv_state && taps > 1) ? conv_state + (int64_t)state_slots[s] * (taps - 1) * C : nullptr;
  const int lp = p / page_size;
  const int page = lp < max_pages ? block_table[(int64_t)s * max_pages + lp] : -1;
  const bool writes = k_pages != nullptr;
  if (writes && (page < 0 || page >= num_pages)) {
    if (threadIdx.x == 0) atomicExch(status, 1);
    return;
  }
  const int slot = p % page_size;
  const int half = rot_dims / 2;
  const float pos = (float)p;
  auto value_at = [&](int c) {
    float y = conv_at(qkv, ld, state_row, C, taps, conv_w, w_dtype, first, t, c);
    if (x.bias) y += load_as_float(x.bias, x.bias_dtype, c);
    return y;
  };
  extern __shared__ __align__(16) float cr_factor[];      // [H + G] with a norm: 1 / root mean square
  if (x.wq) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int n = warp; n < H + G; n += blockDim.x >> 5) {
      float ss = 0.f;
      for (int i = lane; i < dk; i += 32) {
        const float y = value_at(n * dk + i);
        ss = fmaf(y, y, ss);
      }
      ss = warp_sum(ss);
      if (lane == 0) cr_factor[n] = rsqrtf(ss / (float)dk + x.norm_eps);
    }
    __syncthreads();
  }
  auto normed_at = [&](int n, int i) {
    float y = value_at(n * dk + i);
    if (x.wq) y *= cr_factor[n] * load_as_float(n < H ? x.wq : x.wk, x.norm_dtype, i);
    return y;
  };
  // queries and keys: H + G vectors of dk numbers
  for (int idx = threadIdx.x; idx < (H + G) * dk; idx += blockDim.x) {
    const int n = idx / dk, i = idx - n * dk;
    if (x.neighbours ? (i < rot_dims && (i & 1)) : (i >= half && i < rot_dims)) continue;   // written by the pair's first
    T* dst;                                        // (keys follow the queries in the row)
    if (n < H) {
      dst = q_out + ((int64_t)t * H + n) * dk;
    } else {
      if (!writes) continue;
      dst = k_pages + (((int64_t)page * G + (n - H)) * page_size + slot) * dk;
    }
    const float a = normed_at(n, i);
    if (i < rot_dims) {
      const int other = x.neighbours ? 1 : half;
      const float b = normed_at(n, i + other);
      float sn, cs;
      sincosf(pos * freq[x.neighbours ? i >> 1 : i], &sn, &cs);
      sn *= x.mag;
      cs *= x.mag;
      dst[i] = from_float<T>(a * cs - b * sn);
      dst[i + other] = from_float<T>(b * cs + a * sn);
    } else {
      dst[i] = from_float<T>(a);
    }
  }
  const int v0 = (H + G) * dk;
  for (int idx = threadIdx.x; idx < x.GV * dv; idx += blockDim.x) {
    const int g = idx / dv, i = idx - g * dv;
    float v = value_at(v0 + idx);
    if (x.v_first) v = (1.f - x.v_mix) * v + x.v_mix * to_float(((const T*)x.v_first)[(int64_t)t * x.GV * dv + idx]);
    if (x.v_keep) ((T*)x.v_keep)[(int64_t)t * x.GV * dv + idx] = from_float<T>(v);
    if (writes) v_pages[(((int64_t)page * x.GV + g) * page_size + slot) * dv + i] = from_float<T>(v);
  }
}

// The same in bfloat16 for sizes in steps of 8 (key and value sizes, and half of rot_dims): a thread owns 8 channels
// in a row, so every row of inputs, the channels' taps and the outputs move 16 bytes at a time; the token's
// convolved channels pass through shared memory in 32-bit, where a rotated pair finds its other half.  The sums run
// over the taps in the same order as in the kernel above.
template <int TAPS>
__global__ void __launch_bounds__(256)
conv_rope_write_vec_kernel(__nv_bfloat16* __restrict__ q_out, const __nv_bfloat16* __restrict__ qkv, int64_t ld, int H,
                           int G, int dk, int dv, const __nv_bfloat16* __restrict__ conv_w,
                           const __nv_bfloat16* __restrict__ conv_state, const float* __restrict__ freq, int rot_dims,
                           const int* __restrict__ positions, const int* __restrict__ seq_of_token,
                           const int* __restrict__ cu_q, const int* __restrict__ state_slots,
                           const int* __restrict__ block_table, int max_pages, int page_size,
                           __nv_bfloat16* __restrict__ k_pages, __nv_bfloat16* __restrict__ v_pages, int64_t num_pages,
                           int* __restrict__ status, const RopeExtras x) {
  atom::pdl_trigger();
  atom::pdl_wait();
  extern __shared__ __align__(16) float cv_y[];      // [C], cos and sin of the rotated pairs, [(H + G) dk / 8] sums of squares
  const int t = blockIdx.x;
  const int s = seq_of_token[t];
  if (s < 0) return;
  const int p = positions[t];
  const int first = cu_q[s];
  const int C = H * dk + G * dk + x.GV * dv;
  const __nv_bfloat16* state_row =
      (conv_state && TAPS > 1) ? conv_state + (int64_t)state_slots[s] * (TAPS - 1) * C : nullptr;
  const int lp = p / page_size;
  const int page = lp < max_pages ? block_table[(int64_t)s * max_pages + lp] : -1;
  const bool writes = k_pages != nullptr;
  if (writes && (page < 0 || page >= num_pages)) {
    if (threadIdx.x == 0) atomicExch(status, 1);
    return;
  }
  const int slot = p % page_size;
  const int groups = C / 8;
  const int half = rot_dims / 2;
  float* ang_c = cv_y + C;
  float* ang_s = ang_c + half;
  float* squares = ang_s + half;
  for (int i = threadIdx.x; i < half; i += blockDim.x) {      // (all heads of the token share the angles)
    float sn, cs;
    sincosf((float)p * freq[i], &sn, &cs);
    ang_c[i] = cs * x.mag;
    ang_s[i] = sn * x.mag;
  }
  for (int g = threadIdx.x; g < groups; g += blockDim.x) {
    const int c = g * 8;
    float y[8];
    if (TAPS == 0) {
      const uint4 raw = *reinterpret_cast<const uint4*>(qkv + (int64_t)t * ld + c);
      const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 f = __bfloat1622float2(h2[e]);
        y[2 * e] = f.x;
        y[2 * e + 1] = f.y;
      }
      if (x.bias) {
        if (x.bias_dtype == ATOM_F32) {
#pragma unroll
          for (int e = 0; e < 8; ++e) y[e] += ((const float*)x.bias)[c + e];
        } else {
          const uint4 braw = *reinterpret_cast<const uint4*>((const __nv_bfloat16*)x.bias + c);
          const __nv_bfloat162* b2 = reinterpret_cast<const __nv_bfloat162*>(&braw);
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float2 f = __bfloat1622float2(b2[e]);
            y[2 * e] += f.x;
            y[2 * e + 1] += f.y;
          }
        }
      }
    } else {
      constexpr int NW = TAPS > 0 ? TAPS : 1;
      uint4 wraw[NW];                                  // the 8 channels' taps: 8 * TAPS numbers in a row
#pragma unroll
      for (int j = 0; j < NW; ++j) wraw[j] = *reinterpret_cast<const uint4*>(conv_w + (int64_t)c * TAPS + j * 8);
      const __nv_bfloat16* wv = reinterpret_cast<const __nv_bfloat16*>(wraw);
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] = 0.f;
#pragma unroll
      for (int j = 0; j < NW; ++j) {
        const int tp = t - TAPS + 1 + j;
        uint4 raw = make_uint4(0u, 0u, 0u, 0u);
        if (tp >= first)
          raw = *reinterpret_cast<const uint4*>(qkv + (int64_t)tp * ld + c);
        else if (state_row)
          raw = *reinterpret_cast<const uint4*>(state_row + (int64_t)(TAPS - 1 - (first - tp)) * C + c);
        const __nv_bfloat16* xv = reinterpret_cast<const __nv_bfloat16*>(&raw);
#pragma unroll
        for (int e = 0; e < 8; ++e) y[e] += __bfloat162float(wv[e * TAPS + j]) * __bfloat162float(xv[e]);
      }
    }
    *reinterpret_cast<float4*>(cv_y + c) = make_float4(y[0], y[1], y[2], y[3]);
    *reinterpret_cast<float4*>(cv_y + c + 4) = make_float4(y[4], y[5], y[6], y[7]);
    if (x.wq && c < (H + G) * dk) {
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) ss = fmaf(y[e], y[e], ss);
      squares[g] = ss;
    }
  }
  __syncthreads();
  const int qk_end = (H + G) * dk;
  for (int g = threadIdx.x; g < groups; g += blockDim.x) {
    const int c = g * 8;
    __nv_bfloat16* dst;
    int i0 = 0;
    bool rotated = false;
    int64_t keep_at = -1;
    float o[8], own[8];
    float nf = 1.f;                                      // with a norm: the head's factor, and its weights
    const void* wn = nullptr;
    if (c < qk_end) {
      const int n = c / dk;
      i0 = c - n * dk;
      rotated = i0 < rot_dims;
      if (x.wq) {
        wn = n < H ? x.wq : x.wk;
        float ss = 0.f;
        for (int q = 0; q < dk / 8; ++q) ss += squares[n * (dk / 8) + q];
        nf = rsqrtf(ss / (float)dk + x.norm_eps);
      }
      if (n < H) {
        dst = q_out + ((int64_t)t * H + n) * dk + i0;
      } else {
        if (!writes) continue;
        dst = k_pages + (((int64_t)page * G + (n - H)) * page_size + slot) * dk + i0;
      }
    } else {
      if (!writes && !x.v_keep) continue;
      const int idx = c - qk_end;
      const int gg = idx / dv;
      keep_at = (int64_t)t * x.GV * dv + idx;
      dst = writes ? v_pages + (((int64_t)page * x.GV + gg) * page_size + slot) * dv + (idx - gg * dv) : nullptr;
    }
    // eight numbers of the token's row (of the head's, from number i on), normed where there is a norm
    auto load8 = [&](float (&v)[8], int at, int i) {
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] = cv_y[at + e];
      if (!wn) return;
      if (x.norm_dtype == ATOM_BF16) {
        const uint4 raw = *reinterpret_cast<const uint4*>((const __nv_bfloat16*)wn + i);
        const __nv_bfloat16* wv = reinterpret_cast<const __nv_bfloat16*>(&raw);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] *= nf * __bfloat162float(wv[e]);
      } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] *= nf * ((const float*)wn)[i + e];
      }
    };
    load8(own, c, i0);
    if (rotated && x.neighbours) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float a = own[2 * e], b = own[2 * e + 1];
        const float cs = ang_c[(i0 >> 1) + e], sn = ang_s[(i0 >> 1) + e];
        o[2 * e] = a * cs - b * sn;
        o[2 * e + 1] = b * cs + a * sn;
      }
    } else if (rotated) {
      const bool low = i0 < half;                      // the first of the pair: (a, b) = (own, + half); else (- half, own)
      float other[8];
      load8(other, low ? c + half : c - half, low ? i0 + half : i0 - half);
      const int f0 = low ? i0 : i0 - half;
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const float cs = ang_c[f0 + e], sn = ang_s[f0 + e];
        const float a = low ? own[e] : other[e], b = low ? other[e] : own[e];
        o[e] = low ? a * cs - b * sn : b * cs + a * sn;
      }
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) o[e] = own[e];
      if (keep_at >= 0 && x.v_first) {
        const uint4 raw = *reinterpret_cast<const uint4*>((const __nv_bfloat16*)x.v_first + keep_at);
        const __nv_bfloat16* fv = reinterpret_cast<const __nv_bfloat16*>(&raw);
#pragma unroll
        for (int e = 0; e < 8; ++e) o[e] = (1.f - x.v_mix) * o[e] + x.v_mix * __bfloat162float(fv[e]);
      }
    }
    uint4 packed;
    __nv_bfloat162* h2 = reinterpret_cast<__nv_bfloat162*>(&packed);
#pragma unroll
    for (int e = 0; e < 4; ++e) h2[e] = __floats2bfloat162_rn(o[2 * e], o[2 * e + 1]);
    if (keep_at >= 0 && x.v_keep) *reinterpret_cast<uint4*>((__nv_bfloat16*)x.v_keep + keep_at) = packed;
    if (dst) *reinterpret_cast<uint4*>(dst) = packed;
  }
}

// state [slots, taps - 1, C]: row taps - 2 is the request's latest projected row.  A thread owns a channel and walks
// the rows upwards, so a row it still has to read (further up) has not been written.
template <typename T>
__global__ void conv_state_update_kernel(T* __restrict__ conv_state, const T* __restrict__ qkv, int64_t ld, int C,
                                         int taps, const int* __restrict__ cu_q, const int* __restrict__ state_slots) {
  atom::pdl_trigger();
  atom::pdl_wait();
  const int s = blockIdx.y;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= C) return;
  const int first = cu_q[s], len = cu_q[s + 1] - first;
  if (len <= 0) return;
  T* st = conv_state + (int64_t)state_slots[s] * (taps - 1) * C;
  for (int r = 0; r < taps - 1; ++r) {
    const int src = r + len - (taps - 1);          // row of the step (>= 0) or of the old state (< 0)
    st[(int64_t)r * C + c] = src >= 0 ? qkv[(int64_t)(first + src) * ld + c] : st[(int64_t)(r + len) * C + c];
  }
}

// Beside the softmax over keys: a sink per head, a gate number per (token, head), a constant on the output, and the
// output's row stride (a row may be part of a wider one).
struct AttnExtras {
  const float* sink;     // [nh] or null
  const void* gate;      // [T, nh] rows at stride gate_ld, activation type, or null
  int64_t gate_ld;
  float out_mul;
  int64_t out_ld;
  int chunked;           // 1: the window is a chunk, keys j <= p with j / window = p / window
  float lambda, maps_eps;     // with two maps: the second map's weight, and what is added to the mean square
};

// First key that position p sees (kept first tokens apart).
__device__ __forceinline__ int attn_first_key(int p, int window, int chunked) {
  if (window <= 0) return 0;
  return chunked ? p / window * window : max(0, p - window + 1);
}

template <typename T>
__device__ __forceinline__ float attn_out_factor(const AttnExtras& x, int t, int h) {
  float f = x.out_mul;
  if (x.gate) f /= 1.f + expf(-to_float(((const T*)x.gate)[(int64_t)t * x.gate_ld + h]));
  return f;
}

constexpr int kWinThreads = 128;
constexpr int kWinChunk = 256;

// nh heads; with MAPS maps a head has MAPS queries in a row and a key head MAPS keys: q [T, nh MAPS dk], k_pages
// [pages, nkv MAPS, page, dk], v_pages [pages, nkv, page, dv].
template <typename T, int MAPS>
__global__ void __launch_bounds__(kWinThreads)
window_attention_kernel(T* __restrict__ out, const T* __restrict__ q, const T* __restrict__ k_pages,
                        const T* __restrict__ v_pages, const int* __restrict__ block_table, int max_pages,
                        int page_size, const int* __restrict__ positions, const int* __restrict__ seq_of_token, int nh,
                        int nkv, int dk, int dv, float scale, float softcap, int window, int keep_first,
                        const AttnExtras x) {
  atom::pdl_trigger();
  atom::pdl_wait();
  extern __shared__ __align__(16) unsigned char smem_raw[];
  int64_t* row_of = (int64_t*)smem_raw;            // [kWinChunk] (page * nkv + g) * page_size + slot of a key's value
  float* prob = (float*)(row_of + kWinChunk);      // [kWinChunk]
  float* qs = prob + kWinChunk;                    // [dk]
  __shared__ float scratch[32];

  const int t = blockIdx.x, h = blockIdx.y;
  if (seq_of_token[t] < 0) return;
  const int g = h / (nh / nkv);
  const int p = positions[t];
  const int* bt = block_table + (int64_t)seq_of_token[t] * max_pages;
  const int lo = attn_first_key(p, window, x.chunked);
  const int n_first = min(keep_first, lo);         // kept first tokens that the window itself does not reach
  const int n_keys = n_first + (p - lo + 1);
  const float inv_cap = softcap > 0.f ? 1.f / softcap : 0.f;

  float res[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int map = 0; map < MAPS; ++map) {
    const T* qrow = q + (((int64_t)t * nh + h) * MAPS + map) * dk;
    __syncthreads();
    for (int i = threadIdx.x; i < dk; i += blockDim.x) qs[i] = to_float(qrow[i]);
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    float m = -INFINITY, l = 0.f;
    __syncthreads();
    for (int c0 = 0; c0 < n_keys; c0 += kWinChunk) {
      const int n = min(kWinChunk, n_keys - c0);
      float cmax = -INFINITY;
      for (int jj = threadIdx.x; jj < n; jj += blockDim.x) {
        const int e = c0 + jj;
        const int j = e < n_first ? e : lo + (e - n_first);
        const int page = bt[j / page_size];
        row_of[jj] = ((int64_t)page * nkv + g) * page_size + (j % page_size);
        const T* kr = k_pages + (((int64_t)page * nkv + g) * MAPS + map) * page_size * dk + (int64_t)(j % page_size) * dk;
        float sc = 0.f;
        for (int i = 0; i < dk; ++i) sc += qs[i] * to_float(kr[i]);
        sc *= scale;
        if (softcap > 0.f) sc = softcap * tanhf(sc * inv_cap);
        prob[jj] = sc;
        cmax = fmaxf(cmax, sc);
      }
      cmax = block_max(cmax, scratch);
      const float m_new = fmaxf(m, cmax);
      const float corr = expf(m - m_new);
      float lsum = 0.f;
      for (int jj = threadIdx.x; jj < n; jj += blockDim.x) {
        const float e = expf(prob[jj] - m_new);
        prob[jj] = e;
        lsum += e;
      }
      lsum = block_sum(lsum, scratch);
      l = l * corr + lsum;
      m = m_new;
#pragma unroll
      for (int a = 0; a < 4; ++a) {
        const int d = threadIdx.x + a * kWinThreads;
        if (d < dv) {
          float sum = acc[a] * corr;
          for (int jj = 0; jj < n; ++jj) sum += prob[jj] * to_float(v_pages[row_of[jj] * dv + d]);
          acc[a] = sum;
        }
      }
      __syncthreads();
    }
    if (x.sink) l += expf(x.sink[h] - m);
    const float f = (map == 0 ? 1.f : -x.lambda) / l;
#pragma unroll
    for (int a = 0; a < 4; ++a) res[a] = fmaf(acc[a], f, res[a]);
  }
  float mul = attn_out_factor<T>(x, t, h);
  if (MAPS > 1) {
    float ss = 0.f;
#pragma unroll
    for (int a = 0; a < 4; ++a)
      if (threadIdx.x + a * kWinThreads < dv) ss = fmaf(res[a], res[a], ss);
    mul *= rsqrtf(block_sum(ss, scratch) / (float)dv + x.maps_eps);
  }
  T* orow = out + (int64_t)t * x.out_ld + (int64_t)h * dv;
#pragma unroll
  for (int a = 0; a < 4; ++a) {
    const int d = threadIdx.x + a * kWinThreads;
    if (d < dv) orow[d] = from_float<T>(res[a] * mul);
  }
}

// Puts together the shares that window_attention_tc.cu left in `part`: per token and share [m (n) | l (n) | o (n dv)] for
// n = nh MAPS head maps, a share's running maximum (natural logarithm), sum and unnormalised output.  One CTA per (token,
// head), a thread up to four columns.
template <typename T, int MAPS>
__global__ void window_attention_merge_kernel(T* __restrict__ out, const float* __restrict__ part,
                                              const int* __restrict__ seq_of_token, int nh, int dv, int nsplit,
                                              const AttnExtras x) {
  atom::pdl_trigger();
  atom::pdl_wait();
  __shared__ float scratch[32];
  const int t = blockIdx.x, h = blockIdx.y, n = nh * MAPS;
  if (seq_of_token[t] < 0) return;
  const int64_t stride = (int64_t)n * dv + 2 * n;
  const float* pt = part + (int64_t)t * nsplit * stride;
  float res[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int map = 0; map < MAPS; ++map) {
    const int hm = h * MAPS + map;
    float M = -INFINITY;
    for (int s = 0; s < nsplit; ++s) M = fmaxf(M, pt[s * stride + hm]);
    float L = x.sink ? expf(x.sink[h] - M) : 0.f;
    float o[4] = {0.f, 0.f, 0.f, 0.f};
    for (int s = 0; s < nsplit; ++s) {
      const float m = pt[s * stride + hm];
      const float w = (m == -INFINITY) ? 0.f : expf(m - M);      // a share without keys weighs nothing
      L = fmaf(pt[s * stride + n + hm], w, L);
#pragma unroll
      for (int a = 0; a < 4; ++a) {
        const int d = threadIdx.x + a * blockDim.x;
        if (d < dv) o[a] = fmaf(pt[s * stride + 2 * n + (int64_t)hm * dv + d], w, o[a]);
      }
    }
    const float f = (map == 0 ? 1.f : -x.lambda) / L;
#pragma unroll
    for (int a = 0; a < 4; ++a) res[a] = fmaf(o[a], f, res[a]);
  }
  float mul = attn_out_factor<T>(x, t, h);
  if (MAPS > 1) {
    const float ss = res[0] * res[0] + res[1] * res[1] + res[2] * res[2] + res[3] * res[3];
    mul *= rsqrtf(block_sum(ss, scratch) / (float)dv + x.maps_eps);
  }
#pragma unroll
  for (int a = 0; a < 4; ++a) {
    const int d = threadIdx.x + a * blockDim.x;
    if (d < dv) out[(int64_t)t * x.out_ld + (int64_t)h * dv + d] = from_float<T>(res[a] * mul);
  }
}

}  // namespace atom

// qkv: [T, >= C] rows of [q (H dk) | k (G dk) | v (GV dv)], row stride ld; q_out [T, H dk] dense.  conv_w [C, taps]
// (taps 0: no convolution), conv_state [slots, taps - 1, C] (read only here).  k_pages null: nothing is written (G and
// GV may then be 0).  wq, wk [dk]: norm weights of every query and key head (null: no norm; not with a convolution).
ATOM_EXPORT int atom_conv_rope_write(void* q_out, const void* qkv, int dtype, int64_t ld, int T, int H, int G, int dk,
                                     int dv, const void* conv_w, int w_dtype, int taps, const void* conv_state,
                                     const float* freq, int rot_dims, const int* positions, const int* seq_of_token,
                                     const int* cu_q, const int* state_slots, const int* block_table, int max_pages,
                                     int page_size, void* k_pages, void* v_pages, int64_t num_pages, int* status,
                                     const void* bias, int bias_dtype, int neighbours, float mag, const void* v_first,
                                     float v_mix, void* v_keep, int GV, const void* wq, const void* wk, int norm_dtype,
                                     float norm_eps, cudaStream_t stream) {
  if (T <= 0) return ATOM_OK;
  if ((bias || wq) && taps > 0) return ATOM_ERR_ARG;
  const atom::RopeExtras x{bias, bias_dtype, neighbours, mag, v_first, v_mix, v_keep, GV, wq, wk, norm_dtype, norm_eps};
  if (GV < 0 || (k_pages && (G == 0 || GV == 0)) || (wq && G > 0 && !wk)) return ATOM_ERR_ARG;
  if (H <= 0 || G < 0 || dk <= 0 || dv <= 0 || rot_dims < 0 || rot_dims % 2 || rot_dims > dk || taps < 0 ||
      page_size <= 0 || (rot_dims > 0 && !freq) || (taps > 0 && !conv_w))
    return ATOM_ERR_ARG;
  if (dtype == ATOM_F32)
    atom::launch_pdl(atom::conv_rope_write_kernel<float>, dim3(T), dim3(256), (H + G) * sizeof(float), stream, (float*)q_out,
                     (const float*)qkv, ld, H, G, dk, dv, conv_w, w_dtype, taps, (const float*)conv_state, freq,
                     rot_dims, positions, seq_of_token, cu_q, state_slots, block_table, max_pages, page_size,
                     (float*)k_pages, (float*)v_pages, num_pages, status, x);
  else if (dtype == ATOM_BF16 && dk % 8 == 0 && dv % 8 == 0 && rot_dims % (neighbours ? 8 : 16) == 0 && ld % 8 == 0 && taps <= 8 &&
           (taps == 0 || w_dtype == ATOM_BF16) && ((H + G) * dk + GV * dv + rot_dims + (H + G) * dk / 8) * sizeof(float) <= 48 * 1024 &&
           ((uintptr_t)qkv % 16) == 0 && ((uintptr_t)conv_w % 16) == 0 && ((uintptr_t)conv_state % 16) == 0 &&
           ((uintptr_t)bias % 16) == 0 && ((uintptr_t)v_first % 16) == 0 && ((uintptr_t)v_keep % 16) == 0 &&
           ((uintptr_t)q_out % 16) == 0 && ((uintptr_t)wq % 16) == 0 && ((uintptr_t)wk % 16) == 0 && ((uintptr_t)k_pages % 16) == 0 && ((uintptr_t)v_pages % 16) == 0) {
    const int C = (H + G) * dk + GV * dv;
    const int threads = C / 8 >= 256 ? 256 : ((C / 8 + 31) / 32) * 32;
#define ATOM_CV(TAPS)                                                                                               \
  atom::launch_pdl(atom::conv_rope_write_vec_kernel<TAPS>, dim3(T), dim3(threads), (C + rot_dims + (H + G) * dk / 8) * sizeof(float), stream, \
                   (__nv_bfloat16*)q_out, (const __nv_bfloat16*)qkv, ld, H, G, dk, dv, (const __nv_bfloat16*)conv_w, \
                   (const __nv_bfloat16*)conv_state, freq, rot_dims, positions, seq_of_token, cu_q, state_slots,    \
                   block_table, max_pages, page_size, (__nv_bfloat16*)k_pages, (__nv_bfloat16*)v_pages, num_pages,  \
                   status, x)
    switch (taps) {
      case 0: ATOM_CV(0); break;
      case 1: ATOM_CV(1); break;
      case 2: ATOM_CV(2); break;
      case 3: ATOM_CV(3); break;
      case 4: ATOM_CV(4); break;
      case 5: ATOM_CV(5); break;
      case 6: ATOM_CV(6); break;
      case 7: ATOM_CV(7); break;
      default: ATOM_CV(8); break;
    }
#undef ATOM_CV
  } else if (dtype == ATOM_BF16)
    atom::launch_pdl(atom::conv_rope_write_kernel<__nv_bfloat16>, dim3(T), dim3(256), (H + G) * sizeof(float), stream,
                     (__nv_bfloat16*)q_out, (const __nv_bfloat16*)qkv, ld, H, G, dk, dv, conv_w, w_dtype, taps,
                     (const __nv_bfloat16*)conv_state, freq, rot_dims, positions, seq_of_token, cu_q, state_slots,
                     block_table, max_pages, page_size, (__nv_bfloat16*)k_pages, (__nv_bfloat16*)v_pages, num_pages,
                     status, x);
  else
    return ATOM_ERR_ARG;
  return atom::check_launch();
}

ATOM_EXPORT int atom_conv_state_update(void* conv_state, const void* qkv, int dtype, int64_t ld, int C, int taps,
                                       const int* cu_q, const int* state_slots, int num_seqs, cudaStream_t stream) {
  if (num_seqs <= 0 || taps <= 1) return ATOM_OK;
  if (C <= 0 || num_seqs > 65535) return ATOM_ERR_ARG;
  dim3 grid((C + 127) / 128, num_seqs);
  if (dtype == ATOM_F32)
    atom::launch_pdl(atom::conv_state_update_kernel<float>, grid, dim3(128), 0, stream, (float*)conv_state,
                     (const float*)qkv, ld, C, taps, cu_q, state_slots);
  else if (dtype == ATOM_BF16)
    atom::launch_pdl(atom::conv_state_update_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream,
                     (__nv_bfloat16*)conv_state, (const __nv_bfloat16*)qkv, ld, C, taps, cu_q, state_slots);
  else
    return ATOM_ERR_ARG;
  return atom::check_launch();
}

// out: row t at out + t * out_ld, heads packed [nh, dv]; q [T, nh maps dk] dense.  window <= 0: every earlier key;
// softcap <= 0: none; sink, gate null: none; maps: 1 or 2.
ATOM_EXPORT int atom_window_attention(void* out, const void* q, int dtype, const void* k_pages, const void* v_pages,
                                      const int* block_table, int max_pages, int page_size, const int* positions,
                                      const int* seq_of_token, int T, int nh, int nkv, int dk, int dv, float scale,
                                      float softcap, int window, int keep_first, const float* sink, const void* gate,
                                      int64_t gate_ld, float out_mul, int64_t out_ld, int chunked, int maps, float lambda,
                                      float maps_eps, cudaStream_t stream) {
  if (T <= 0) return ATOM_OK;
  const atom::AttnExtras x{sink, gate, gate_ld, out_mul, out_ld, chunked, lambda, maps_eps};
  if (nh <= 0 || nkv <= 0 || nh % nkv != 0 || dk <= 0 || dv <= 0 || dv > 4 * atom::kWinThreads || dk > 4096 ||
      page_size <= 0 || nh > 65535 || keep_first < 0 || maps < 1 || maps > 2 || (dtype != ATOM_F32 && dtype != ATOM_BF16))
    return ATOM_ERR_ARG;
  const size_t smem = sizeof(float) * (dk + atom::kWinChunk) + sizeof(int64_t) * atom::kWinChunk;
#define ATOM_WIN(TT, MAPS)                                                                                            \
  atom::launch_pdl(atom::window_attention_kernel<TT, MAPS>, dim3(T, nh), dim3(atom::kWinThreads), smem, stream, (TT*)out, \
                   (const TT*)q, (const TT*)k_pages, (const TT*)v_pages, block_table, max_pages, page_size, positions, \
                   seq_of_token, nh, nkv, dk, dv, scale, softcap, window, keep_first, x)
  if (dtype == ATOM_F32) {
    if (maps == 1) ATOM_WIN(float, 1);
    else ATOM_WIN(float, 2);
  } else {
    if (maps == 1) ATOM_WIN(__nv_bfloat16, 1);
    else ATOM_WIN(__nv_bfloat16, 2);
  }
#undef ATOM_WIN
  return atom::check_launch();
}

ATOM_EXPORT int atom_window_attention_merge(void* out, int dtype, const float* part, const int* seq_of_token, int T, int nh,
                                            int dv, int nsplit, const float* sink, const void* gate, int64_t gate_ld,
                                            float out_mul, int64_t out_ld, int maps, float lambda, float maps_eps,
                                            cudaStream_t stream) {
  if (T <= 0) return ATOM_OK;
  const atom::AttnExtras x{sink, gate, gate_ld, out_mul, out_ld, 0, lambda, maps_eps};
  if (nsplit < 1 || part == nullptr || nh <= 0 || nh > 65535 || dv <= 0 || dv > 512 || maps < 1 || maps > 2 ||
      (dtype != ATOM_F32 && dtype != ATOM_BF16))
    return ATOM_ERR_ARG;
  const int threads = dv >= 128 ? 128 : (dv >= 64 ? 64 : 32);
#define ATOM_WIN(TT, MAPS)                                                                                            \
  atom::launch_pdl(atom::window_attention_merge_kernel<TT, MAPS>, dim3(T, nh), dim3(threads), 0, stream, (TT*)out, part, \
                   seq_of_token, nh, dv, nsplit, x)
  if (dtype == ATOM_F32) {
    if (maps == 1) ATOM_WIN(float, 1);
    else ATOM_WIN(float, 2);
  } else {
    if (maps == 1) ATOM_WIN(__nv_bfloat16, 1);
    else ATOM_WIN(__nv_bfloat16, 2);
  }
#undef ATOM_WIN
  return atom::check_launch();
}
