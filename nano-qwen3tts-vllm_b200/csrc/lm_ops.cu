// lm_ops.cu - element-wise and per-row kernels of token-id decoder models with a 32-bit residual stream:
//   embedding + learned positions, RMS norm with one gain ("gain norm"), the residual update of a parallel layer fused
//   with the next norm, the short causal convolution over time with its carried state fused with per-head q/k RMS norm
//   and the paged K/V write, the squared-ReLU activation, and the top-k routers with their expert grouping.
//
// Activations are `T` = bf16 (serving) or float (the all-32-bit mode); the residual stream, every norm, the router and
// all per-head constants are float in both.  Nothing allocates or synchronises; every launch is graph-capturable.
#include <math.h>

#include <type_traits>

#include "common.cuh"

namespace b2 {

template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

constexpr int ROW_THREADS = 256;

// sum over the block; every thread gets the result.  `red` holds 33 floats.
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  __syncthreads();                       // red may still be read from a previous call
  if (lane == 0) red[warp] = v;
  __syncthreads();
  if (warp == 0) {
    float t = lane < nw ? red[lane] : 0.f;
    t = warp_sum(t);
    if (lane == 0) red[32] = t;
  }
  __syncthreads();
  return red[32];
}

// h[row] = T(x[row] / sqrt(mean(x[row]^2) + eps) * gain) for the row this block owns (x just written by this block).
template <typename T>
__device__ __forceinline__ void gain_norm_tail(const float* xr, T* hr, int cols, float ssq, const float* gain, float eps,
                                               float* red) {
  const float tot = block_sum(ssq, red);
  const float inv = 1.0f / sqrtf(tot / static_cast<float>(cols) + eps);
  const float g = gain[0];
  for (int c = threadIdx.x; c < cols; c += blockDim.x) hr[c] = from_f<T>(xr[c] * inv * g);
}

// ------------------------------------------------------------------ embedding + learned position (+ first norm)
template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
embed_pos_norm_kernel(const int32_t* __restrict__ tokens, const int32_t* __restrict__ positions, const T* __restrict__ embed,
                      const T* __restrict__ pos_table, float* __restrict__ x, T* __restrict__ h, const float* __restrict__ gain,
                      int cols, int vocab, int max_pos, float eps) {
  __shared__ float red[33];
  const int row = blockIdx.x;
  int tok = tokens[row], p = positions[row];
  tok = min(max(tok, 0), vocab - 1);
  p = min(max(p, 0), max_pos - 1);
  const T* er = embed + static_cast<size_t>(tok) * cols;
  const T* pr = pos_table + static_cast<size_t>(p) * cols;
  float* xr = x + static_cast<size_t>(row) * cols;
  float ssq = 0.f;
  for (int c = threadIdx.x; c < cols; c += blockDim.x) {
    const float v = to_f(er[c]) + to_f(pr[c]);
    xr[c] = v;
    ssq += v * v;
  }
  if (h != nullptr) gain_norm_tail<T>(xr, h + static_cast<size_t>(row) * cols, cols, ssq, gain, eps, red);
}

// ------------------------------------------------------------------ residual update (+ next norm)
// x[row] += mult * (a[row] + b[row] + sum_k w[row, k] * z[row * top + k]) with every term optional; then, if h is
// given, h[row] = gain norm of the NEW x[row].  The expert terms are added in the order k = 0 .. top-1.
template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
residual_norm_kernel(float* __restrict__ x, const T* __restrict__ a, const T* __restrict__ b, const T* __restrict__ z,
                     const float* __restrict__ zw, int top, float mult, T* __restrict__ h, const float* __restrict__ gain,
                     int cols, float eps) {
  __shared__ float red[33];
  const size_t row = blockIdx.x;
  float* xr = x + row * cols;
  float ssq = 0.f;
  for (int c = threadIdx.x; c < cols; c += blockDim.x) {
    float s = 0.f;
    if (a != nullptr) s += to_f(a[row * cols + c]);
    if (b != nullptr) s += to_f(b[row * cols + c]);
    if (z != nullptr) {
      float e = 0.f;
      for (int k = 0; k < top; ++k) e += zw[row * top + k] * to_f(z[(row * top + k) * cols + c]);
      s += e;
    }
    const float v = xr[c] + mult * s;
    xr[c] = v;
    ssq += v * v;
  }
  if (h != nullptr) gain_norm_tail<T>(xr, h + row * cols, cols, ssq, gain, eps, red);
}

// out[i] = gain norm of x[rows[i]] (the rows whose logits are wanted)
template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
gather_gain_norm_kernel(const float* __restrict__ x, const int32_t* __restrict__ rows, T* __restrict__ out,
                        const float* __restrict__ gain, int cols, float eps) {
  __shared__ float red[33];
  const size_t src = rows != nullptr ? rows[blockIdx.x] : blockIdx.x;
  const float* xr = x + src * cols;
  float ssq = 0.f;
  for (int c = threadIdx.x; c < cols; c += blockDim.x) ssq += xr[c] * xr[c];
  gain_norm_tail<T>(xr, out + static_cast<size_t>(blockIdx.x) * cols, cols, ssq, gain, eps, red);
}

// ------------------------------------------------------------------ squared ReLU, in place
template <typename T>
__global__ void relu_sq_kernel(T* __restrict__ y, size_t n) {
  for (size_t i = blockIdx.x * static_cast<size_t>(blockDim.x) + threadIdx.x; i < n; i += static_cast<size_t>(gridDim.x) * blockDim.x) {
    const float v = fmaxf(to_f(y[i]), 0.f);
    y[i] = from_f<T>(v * v);
  }
}

// ------------------------------------------------------------------ cosines and sines of a step's positions
// table[n, i] = cos(position[n] * freq[i]), table[n, half + i] = sin(.), i < half; the angle is formed in float.  One table
// per step serves every layer with the same frequencies.
__global__ void rotary_table_kernel(const int32_t* __restrict__ positions, const float* __restrict__ freq, float* __restrict__ table,
                                    int n, int half) {
  const size_t idx = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (idx >= static_cast<size_t>(n) * half) return;
  const size_t t = idx / half;
  const int i = static_cast<int>(idx % half);
  float sn, cs;
  sincosf(static_cast<float>(positions[t]) * freq[i], &sn, &cs);
  table[t * 2 * half + i] = cs;
  table[t * 2 * half + half + i] = sn;
}

// ------------------------------------------------------------------ short convolution + head norm + paged K/V write
// One warp per (token, head slot); head slots are the H query heads, then the G key heads, then the G value heads of the
// merged projection row u[n] = [q | k | v].  Tap j of the token at position p reads the projection of position
// p - taps + 1 + j: from this step's rows when that position is in the step's portion, from the sequence's carried
// state (its last taps - 1 projections, oldest first) when it came earlier, zero before the sequence's start.
constexpr int CONV_WARPS = 8;
constexpr int CONV_MAX_PER_LANE = 8;       // head sizes up to 256
constexpr int CONV_MAX_TAPS = 16;

// What happens to a head between the convolution and the store.  Default (CONV_ROUND): q and k are rounded to T, divided
// by the root mean square of the head and multiplied by their weight; v is stored as it is.
//   rot, rot_dims   coordinate i < rot_dims / 2 of a q / k head is paired with i + rot_dims / 2 and the pair turned by the
//                   token's angle, before the norm: rot [n, rot_dims] holds the cosines, then the sines (b2tts_rotary_table)
//   CONV_UNIT_V     v is divided by the root mean square of its head too, without a weight
//   without CONV_ROUND the convolution's float results feed rotation and norm unrounded
struct ConvHeadOps {
  const float* rot;
  int rot_dims;
  int flags;
};
constexpr int CONV_ROUND = 1, CONV_UNIT_V = 2;

template <typename T>
__global__ void __launch_bounds__(CONV_WARPS * 32)
conv_headnorm_kvwrite_kernel(const T* __restrict__ u, int64_t u_stride, const float* __restrict__ conv_w /* [C, taps] */,
                             const T* __restrict__ state /* [slots, taps-1, C] */, const int32_t* __restrict__ tok_seq,
                             const int32_t* __restrict__ positions, const int32_t* __restrict__ seq_start,
                             const int32_t* __restrict__ seq_pos0, const int32_t* __restrict__ seq_slot,
                             const int32_t* __restrict__ slot_mapping, const float* __restrict__ q_norm_w,
                             const float* __restrict__ k_norm_w, T* __restrict__ q_out /* [n, H*d] */,
                             T* __restrict__ k_cache /* [slots, G*d] */, T* __restrict__ v_cache /* [slots, G*dv] */,
                             int n_tokens, int H, int G, int d, int dv, int taps, float eps, const ConvHeadOps ops) {
  __shared__ float rbuf[CONV_WARPS][32 * CONV_MAX_PER_LANE];
  const int lane = threadIdx.x & 31;
  const int item = blockIdx.x * CONV_WARPS + (threadIdx.x >> 5);
  const int heads = H + 2 * G;
  if (item >= n_tokens * heads) return;
  const int n = item / heads, hs = item % heads;
  const int slot = slot_mapping[n];
  if (slot < 0) return;                                  // padding row
  const int C = H * d + G * d + G * dv;
  int kind, head, width, c0;
  if (hs < H) { kind = 0; head = hs; width = d; c0 = head * d; }
  else if (hs < H + G) { kind = 1; head = hs - H; width = d; c0 = H * d + head * d; }
  else { kind = 2; head = hs - H - G; width = dv; c0 = H * d + G * d + head * dv; }
  const int b = tok_seq[n], p = positions[n];
  const int pos0 = seq_pos0[b], start = seq_start[b], sslot = seq_slot[b];
  const int R = taps - 1;
  // where tap j comes from: a row of u (>= 0), a state entry (encoded as -2 - r) or nothing (-1)
  int src[CONV_MAX_TAPS];
#pragma unroll
  for (int j = 0; j < CONV_MAX_TAPS; ++j) {
    src[j] = -1;
    if (j < taps) {
      const int pj = p - R + j;
      if (pj >= pos0) src[j] = start + (pj - pos0);
      else if (pj >= 0) src[j] = -2 - (pj - (pos0 - R));  // state entry r holds position pos0 - R + r
    }
  }
  float y[CONV_MAX_PER_LANE];
  float ssq = 0.f;
#pragma unroll
  for (int i = 0; i < CONV_MAX_PER_LANE; ++i) {
    const int cc = lane + 32 * i;
    y[i] = 0.f;
    if (cc < width) {
      const int c = c0 + cc;
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < CONV_MAX_TAPS; ++j) {
        if (j < taps && src[j] != -1) {
          const float uv = src[j] >= 0 ? to_f(u[static_cast<int64_t>(src[j]) * u_stride + c])
                                       : to_f(state[(static_cast<size_t>(sslot) * R + (-2 - src[j])) * C + c]);
          acc += conv_w[c * taps + j] * uv;
        }
      }
      y[i] = acc;
    }
  }
  if (kind != 2 && (ops.flags & CONV_ROUND)) {
    // the projection and convolution outputs are activations: the norm reads them as stored in T
#pragma unroll
    for (int i = 0; i < CONV_MAX_PER_LANE; ++i) y[i] = to_f(from_f<T>(y[i]));
  }
  if (kind != 2 && ops.rot_dims > 0) {
    float* buf = rbuf[threadIdx.x >> 5];
    const int half = ops.rot_dims / 2;
    const float* rt = ops.rot + static_cast<size_t>(n) * ops.rot_dims;
#pragma unroll
    for (int i = 0; i < CONV_MAX_PER_LANE; ++i) buf[lane + 32 * i] = y[i];
    __syncwarp();
#pragma unroll
    for (int i = 0; i < CONV_MAX_PER_LANE; ++i) {
      const int cc = lane + 32 * i;
      if (cc < half) y[i] = y[i] * rt[cc] - buf[cc + half] * rt[half + cc];
      else if (cc < ops.rot_dims) y[i] = y[i] * rt[cc - half] + buf[cc - half] * rt[cc];
    }
  }
  if (kind != 2 || (ops.flags & CONV_UNIT_V)) {
    ssq = 0.f;
#pragma unroll
    for (int i = 0; i < CONV_MAX_PER_LANE; ++i) ssq += y[i] * y[i];
    ssq = warp_sum(ssq);
    const float inv = 1.0f / sqrtf(ssq / static_cast<float>(width) + eps);
    const float* w = kind == 0 ? q_norm_w : kind == 1 ? k_norm_w : nullptr;
#pragma unroll
    for (int i = 0; i < CONV_MAX_PER_LANE; ++i) {
      const int cc = lane + 32 * i;
      if (cc < width) y[i] = y[i] * inv * (w != nullptr ? w[cc] : 1.f);
    }
  }
  T* dst = kind == 0 ? q_out + static_cast<size_t>(n) * H * d + head * d
         : kind == 1 ? k_cache + static_cast<size_t>(slot) * G * d + head * d
                     : v_cache + static_cast<size_t>(slot) * G * dv + head * dv;
#pragma unroll
  for (int i = 0; i < CONV_MAX_PER_LANE; ++i) {
    const int cc = lane + 32 * i;
    if (cc < width) dst[cc] = from_f<T>(y[i]);
  }
}

// The same with four adjacent channels per lane (8- or 16-byte loads and stores) for head sizes that are multiples of 4.
template <typename T> struct Vec4;
template <> struct Vec4<float> {
  __device__ static void load(const float* p, float* f) { const float4 r = *reinterpret_cast<const float4*>(p); f[0] = r.x; f[1] = r.y; f[2] = r.z; f[3] = r.w; }
  __device__ static void store(float* p, const float* f) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
};
template <> struct Vec4<__nv_bfloat16> {
  __device__ static void load(const __nv_bfloat16* p, float* f) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    f[0] = bf16lo(r.x); f[1] = bf16hi(r.x); f[2] = bf16lo(r.y); f[3] = bf16hi(r.y);
  }
  __device__ static void store(__nv_bfloat16* p, const float* f) { *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3])); }
};
constexpr int CONV4_CHUNKS = 2;            // head sizes up to 256
constexpr int CONV4_TOKENS = 8;            // consecutive rows of a prompt step per warp: the taps' weights are loaded once for all

// One warp per (block of TOK rows, head slice): TOK = CONV4_TOKENS, or 1 for steps of few rows, which then spread over more
// warps.  The lane keeps the taps of its four channels in registers.
template <typename T, int TAPS, int NCH, bool ROT, int TOK>
__global__ void __launch_bounds__(CONV_WARPS * 32)
conv_headnorm_kvwrite_vec4_kernel(const T* __restrict__ u, int64_t u_stride, const float* __restrict__ conv_w,
                                  const T* __restrict__ state, const int32_t* __restrict__ tok_seq,
                                  const int32_t* __restrict__ positions, const int32_t* __restrict__ seq_start,
                                  const int32_t* __restrict__ seq_pos0, const int32_t* __restrict__ seq_slot,
                                  const int32_t* __restrict__ slot_mapping, const float* __restrict__ q_norm_w,
                                  const float* __restrict__ k_norm_w, T* __restrict__ q_out, T* __restrict__ k_cache,
                                  T* __restrict__ v_cache, int n_tokens, int H, int G, int d, int dv, float eps,
                                  const ConvHeadOps ops) {
  const int lane = threadIdx.x & 31;
  const int item = blockIdx.x * CONV_WARPS + (threadIdx.x >> 5);
  const int heads = H + 2 * G;
  const int n_blocks = (n_tokens + TOK - 1) / TOK;
  if (item >= n_blocks * heads) return;
  const int n0 = (item / heads) * TOK, hs = item % heads;
  const int C = H * d + G * d + G * dv;
  int kind, head, width, c0;
  if (hs < H) { kind = 0; head = hs; width = d; c0 = head * d; }
  else if (hs < H + G) { kind = 1; head = hs - H; width = d; c0 = H * d + head * d; }
  else { kind = 2; head = hs - H - G; width = dv; c0 = H * d + G * d + head * dv; }
  constexpr int R = TAPS - 1;
  float w[NCH][4][TAPS];
  float g4[NCH][4];
#pragma unroll
  for (int i = 0; i < NCH; ++i) {
    const int cc = (lane + 32 * i) * 4;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      g4[i][e] = 1.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) w[i][e][j] = 0.f;
    }
    if (cc < width) {
      // the lane's 4 channels x TAPS taps are 16 * TAPS contiguous, 16-byte aligned bytes: TAPS vector loads
      float flat[4 * TAPS];
#pragma unroll
      for (int v = 0; v < TAPS; ++v) {
        const float4 r = *reinterpret_cast<const float4*>(conv_w + static_cast<size_t>(c0 + cc) * TAPS + 4 * v);
        flat[4 * v] = r.x; flat[4 * v + 1] = r.y; flat[4 * v + 2] = r.z; flat[4 * v + 3] = r.w;
      }
#pragma unroll
      for (int e = 0; e < 4; ++e)
#pragma unroll
        for (int j = 0; j < TAPS; ++j) w[i][e][j] = flat[e * TAPS + j];
      if (kind != 2 && q_norm_w != nullptr) {
        const float4 r = *reinterpret_cast<const float4*>((kind == 0 ? q_norm_w : k_norm_w) + cc);
        g4[i][0] = r.x; g4[i][1] = r.y; g4[i][2] = r.z; g4[i][3] = r.w;
      }
    }
  }
  // the rows' bookkeeping (three dependent loads each) is fetched by one lane per row, all rows at once
  int m_slot = -1, m_p = 0, m_pos0 = 0, m_start = 0, m_sslot = 0;
  if (lane < TOK && n0 + lane < n_tokens) {
    m_slot = slot_mapping[n0 + lane];
    if (m_slot >= 0) {
      const int b = tok_seq[n0 + lane];
      m_p = positions[n0 + lane];
      m_pos0 = seq_pos0[b]; m_start = seq_start[b]; m_sslot = seq_slot[b];
    }
  }
  // the lane's cosines and sines for row n (ROT; rot_dims / 2 is a multiple of four: partners are whole quads)
  struct Turn { float cs[ROT ? NCH : 1][4], sn[ROT ? NCH : 1][4]; };
  auto turn_of = [&](int n) {
    Turn t;
    if constexpr (ROT) {
      const int half = ops.rot_dims / 2;
      const float* rt = ops.rot + static_cast<size_t>(n) * ops.rot_dims;
#pragma unroll
      for (int i = 0; i < NCH; ++i) {
        const int cc = (lane + 32 * i) * 4, c1 = cc < half ? cc : cc - half;
#pragma unroll
        for (int e = 0; e < 4; ++e) { t.cs[i][e] = 1.f; t.sn[i][e] = 0.f; }
        if (kind != 2 && cc < ops.rot_dims && n < n_tokens) {
          Vec4<float>::load(rt + c1, t.cs[i]);
          Vec4<float>::load(rt + half + c1, t.sn[i]);
        }
      }
    }
    return t;
  };
  // rotation and norm of a head (see ConvHeadOps), then the row's destination
  auto finish = [&](float (&y)[NCH][4], int n, int slot, const Turn& turn) {
    if (kind != 2 && (ops.flags & CONV_ROUND)) {
#pragma unroll
      for (int i = 0; i < NCH; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) y[i][e] = to_f(from_f<T>(y[i][e]));
    }
    if constexpr (ROT) {
      if (kind != 2) {
        const int half = ops.rot_dims / 2;
        float r[NCH][4];
#pragma unroll
        for (int i = 0; i < NCH; ++i) {
          const int cc = (lane + 32 * i) * 4;
          const bool first = cc < half;
          const int c2 = cc >= ops.rot_dims ? cc : first ? cc + half : cc - half;      // the partner's channel
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            float pr = __shfl_sync(0xffffffffu, y[0][e], (c2 >> 2) & 31);
            if constexpr (NCH == 2) {
              const float other = __shfl_sync(0xffffffffu, y[1][e], (c2 >> 2) & 31);
              if (c2 >= 128) pr = other;
            }
            r[i][e] = y[i][e] * turn.cs[i][e] + (first ? -pr : pr) * turn.sn[i][e];
          }
        }
#pragma unroll
        for (int i = 0; i < NCH; ++i)
#pragma unroll
          for (int e = 0; e < 4; ++e) y[i][e] = r[i][e];
      }
    }
    if (kind != 2 || (ops.flags & CONV_UNIT_V)) {
      float ssq = 0.f;
#pragma unroll
      for (int i = 0; i < NCH; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) ssq += y[i][e] * y[i][e];
      ssq = warp_sum(ssq);
      const float inv = 1.0f / sqrtf(ssq / static_cast<float>(width) + eps);
#pragma unroll
      for (int i = 0; i < NCH; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) y[i][e] *= inv * g4[i][e];
    }
    T* dst = kind == 0 ? q_out + static_cast<size_t>(n) * H * d + head * d
           : kind == 1 ? k_cache + static_cast<size_t>(slot) * G * d + head * d
                       : v_cache + static_cast<size_t>(slot) * G * dv + head * dv;
#pragma unroll
    for (int i = 0; i < NCH; ++i) {
      const int cc = (lane + 32 * i) * 4;
      if (cc < width) Vec4<T>::store(dst + cc, y[i]);
    }
  };
  // The usual block of a prompt portion: TOK consecutive tokens of one sequence.  Their projections and the
  // taps - 1 before the first are loaded once, all loads issued before the first use; row t then reads entries t .. t + R.
  const int p0 = __shfl_sync(0xffffffffu, m_p, 0), start0 = __shfl_sync(0xffffffffu, m_start, 0);
  const bool mine = lane >= TOK || (m_slot >= 0 && m_start == start0 && m_p == p0 + lane);
  if (__all_sync(0xffffffffu, mine)) {
    const int pos0 = __shfl_sync(0xffffffffu, m_pos0, 0), sslot = __shfl_sync(0xffffffffu, m_sslot, 0);
    float uv[TOK + R][NCH][4];
#pragma unroll
    for (int k = 0; k < TOK + R; ++k) {
      const int pk = p0 - R + k;
#pragma unroll
      for (int i = 0; i < NCH; ++i) {
        const int cc = (lane + 32 * i) * 4;
#pragma unroll
        for (int e = 0; e < 4; ++e) uv[k][i][e] = 0.f;             // before the sequence's start
        if (cc < width) {
          if (pk >= pos0) Vec4<T>::load(u + static_cast<int64_t>(start0 + pk - pos0) * u_stride + c0 + cc, uv[k][i]);
          else if (pk >= 0) Vec4<T>::load(state + (static_cast<size_t>(sslot) * R + (pk - (pos0 - R))) * C + c0 + cc, uv[k][i]);
        }
      }
    }
    Turn ahead = turn_of(n0);                // a row ahead of its use
#pragma unroll
    for (int t = 0; t < TOK; ++t) {
      const Turn turn = ahead;
      if (t + 1 < TOK) ahead = turn_of(n0 + t + 1);
      float y[NCH][4];
#pragma unroll
      for (int i = 0; i < NCH; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          y[i][e] = 0.f;
#pragma unroll
          for (int j = 0; j < TAPS; ++j) y[i][e] = fmaf(w[i][e][j], uv[t + j][i][e], y[i][e]);
        }
      finish(y, n0 + t, __shfl_sync(0xffffffffu, m_slot, t), turn);
    }
    return;
  }
  // anything else (decoded tokens, the seam of two sequences, padding): row by row
#pragma unroll
  for (int t = 0; t < TOK; ++t) {
    const int n = n0 + t;
    const int slot = __shfl_sync(0xffffffffu, m_slot, t);
    if (slot < 0) continue;                  // padding row, or past the step's last row
    const int p = __shfl_sync(0xffffffffu, m_p, t), pos0 = __shfl_sync(0xffffffffu, m_pos0, t);
    const int start = __shfl_sync(0xffffffffu, m_start, t), sslot = __shfl_sync(0xffffffffu, m_sslot, t);
    const T* src[TAPS];                      // row of tap j (nullptr: before the sequence's start)
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const int pj = p - R + j;
      src[j] = nullptr;
      if (pj >= pos0) src[j] = u + static_cast<int64_t>(start + pj - pos0) * u_stride;
      else if (pj >= 0) src[j] = state + (static_cast<size_t>(sslot) * R + (pj - (pos0 - R))) * C;
    }
    float y[NCH][4];
#pragma unroll
    for (int i = 0; i < NCH; ++i) {
      const int cc = (lane + 32 * i) * 4;
#pragma unroll
      for (int e = 0; e < 4; ++e) y[i][e] = 0.f;
      if (cc < width) {
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
          if (src[j] != nullptr) {
            float uv[4];
            Vec4<T>::load(src[j] + c0 + cc, uv);
#pragma unroll
            for (int e = 0; e < 4; ++e) y[i][e] = fmaf(w[i][e][j], uv[e], y[i][e]);
          }
        }
      }
    }
    finish(y, n, slot, turn_of(n));
  }
}

// The carried state after the step: entry r holds the projection of position end - R + r (end = pos0 + new tokens).
// One thread per (sequence, channel) reads its old entries before it writes any, so the shift is safe in place.
template <typename T>
__global__ void conv_state_update_kernel(const T* __restrict__ u, int64_t u_stride, T* __restrict__ state,
                                         const int32_t* __restrict__ seq_start, const int32_t* __restrict__ seq_pos0,
                                         const int32_t* __restrict__ seq_len, const int32_t* __restrict__ seq_slot,
                                         int n_seqs, int C, int taps) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  const int b = blockIdx.y;
  if (c >= C || b >= n_seqs) return;
  const int len = seq_len[b];
  if (len <= 0) return;                                  // padding row
  const int R = taps - 1, pos0 = seq_pos0[b], start = seq_start[b];
  T* st = state + static_cast<size_t>(seq_slot[b]) * R * C + c;
  T old[CONV_MAX_TAPS];
#pragma unroll
  for (int r = 0; r < CONV_MAX_TAPS; ++r) if (r < R) old[r] = st[static_cast<size_t>(r) * C];
  const int end = pos0 + len;
#pragma unroll
  for (int r = 0; r < CONV_MAX_TAPS; ++r) {
    if (r < R) {
      const int pj = end - R + r;
      T v = from_f<T>(0.f);
      if (pj >= pos0) v = u[static_cast<int64_t>(start + pj - pos0) * u_stride + c];
      else if (pj >= 0) v = old[pj - (pos0 - R)];
      st[static_cast<size_t>(r) * C] = v;
    }
  }
}

// ------------------------------------------------------------------ top-k router
// A CTA scores and chooses for ROUTE_TOKENS (or one) tokens: their rows are staged in shared memory, the warps split the experts,
// and a router row is read once (in 32-bit products and sums) for all of the CTA's tokens; then a warp per token makes the
// choice: the `top` largest scores (ties: the lower index).  The order of a score's additions does not depend on how many
// tokens share the CTA.
// mode 0: scores = sigmoid, weights = score / (sum of the chosen scores + 1e-20) * scale.
// mode 1: scores = logits + bias, weights = softmax over the chosen scores * scale.
// mode 2: scores = softmax over ALL logits; the choice is made on score + bias, the weights are the chosen scores
//         themselves * scale, not renormalised.
// groups > 1: the experts form that many equal groups of neighbours, a group counts as much as its largest choice score, and
// only experts of the groups_keep best groups (ties: the lower group) can be chosen.
constexpr int ROUTE_WARPS = 8, ROUTE_TOKENS = 8;
constexpr int ROUTE_MAX_EXPERTS = 256;

struct RouteArgs {
  const float* router;                       // [E, cols]
  int32_t* top_idx; float* top_w;
  int n_tokens, cols, E, top;
  float scale;
  const float* bias;                         // [E] or null
  int mode, groups, groups_keep;
};

// One warp's choice for token n; score, weight, gscore: the token's [E] rows in shared memory (score: the raw logits on entry).
__device__ __forceinline__ void route_choose(const RouteArgs& p, int n, int lane, float* score, float* weight, float* gscore) {
  const int E = p.E, top = p.top, mode = p.mode, groups = p.groups, groups_keep = p.groups_keep;
  const float* bias = p.bias;
  const float scale = p.scale;
  const int softmax_chosen = mode == 1;
  for (int e = lane; e < E; e += 32) {
    const float acc = score[e];
    if (mode == 2) {
      score[e] = acc >= -3.0e38f ? acc : -3.0e38f;
    } else if (softmax_chosen) {
      const float sc = acc + (bias != nullptr ? bias[e] : 0.f);
      score[e] = sc >= -3.0e38f ? sc : -3.0e38f;          // a NaN input still yields valid expert ids
    } else {
      const float sc = 1.0f / (1.0f + expf(-acc));
      score[e] = sc >= 0.f ? sc : 0.f;
    }
  }
  __syncwarp();
  if (mode == 2) {                                       // softmax over all experts, then the choice scores
    float mx = -INFINITY;
    for (int e = lane; e < E; e += 32) mx = fmaxf(mx, score[e]);
    mx = warp_max(mx);
    float den = 0.f;
    for (int e = lane; e < E; e += 32) den += expf(score[e] - mx);
    den = warp_sum(den);
    for (int e = lane; e < E; e += 32) {
      const float prob = expf(score[e] - mx) / den;
      weight[e] = prob;
      score[e] = prob + (bias != nullptr ? bias[e] : 0.f);
    }
    __syncwarp();
  }
  if (groups > 1) {
    const int per = E / groups;
    for (int g = lane; g < groups; g += 32) {
      float best = -INFINITY;
      for (int e = g * per; e < (g + 1) * per; ++e) best = fmaxf(best, score[e]);
      gscore[g] = best;
    }
    __syncwarp();
    // a group is kept when fewer than groups_keep others come before it
    unsigned long long kept = 0ull;                       // bit i: the lane's group lane + 32 i
    for (int g = lane, i = 0; g < groups; g += 32, ++i) {
      const float mine = gscore[g];
      int before = 0;
      for (int o = 0; o < groups; ++o) before += gscore[o] > mine || (gscore[o] == mine && o < g);
      if (before < groups_keep) kept |= 1ull << i;
    }
    for (int g = lane, i = 0; g < groups; g += 32, ++i)
      if (!(kept >> i & 1ull))
        for (int e = g * per; e < (g + 1) * per; ++e) score[e] = -INFINITY;
    __syncwarp();
  }
  float sum = 0.f, first = 0.f;
  float chosen_s = 0.f;          // lane k keeps the k-th choice
  int chosen_e = 0;
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int be = 0x7fffffff;
    for (int e = lane; e < E; e += 32) {
      const float s = score[e];
      if (s > best) { best = s; be = e; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      if (ob > best || (ob == best && oe < be)) { best = ob; be = oe; }
    }
    if (be >= E) be = 0;                                  // no finite score left (NaN inputs): still a valid expert id
    if (k == 0) first = best;
    if (softmax_chosen) best = expf(best - first);       // weights: the softmax over the chosen logits only
    if (mode == 2) best = weight[be];
    if (lane == (k & 31)) { chosen_s = best; chosen_e = be; }
    sum += best;
    if (lane == 0) score[be] = -INFINITY;
    __syncwarp();
  }
  if (lane < top) {
    p.top_idx[static_cast<size_t>(n) * top + lane] = chosen_e;
    p.top_w[static_cast<size_t>(n) * top + lane] = mode == 2 ? chosen_s * scale
                                                 : softmax_chosen ? chosen_s / sum * scale : chosen_s / (sum + 1e-20f) * scale;
  }
}

template <typename T> __device__ __forceinline__ void route_load4(const T* p, float* f);
template <> __device__ __forceinline__ void route_load4<float>(const float* p, float* f) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
}
template <> __device__ __forceinline__ void route_load4<__nv_bfloat16>(const __nv_bfloat16* p, float* f) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  f[0] = bf16lo(v.x); f[1] = bf16hi(v.x); f[2] = bf16lo(v.y); f[3] = bf16hi(v.y);
}

// V = 4: rows of whole 4-column vectors; V = 1: any row length.
template <typename T, int TOK, int V>
__global__ void __launch_bounds__(ROUTE_WARPS * 32)
moe_route_kernel(const T* __restrict__ h, const RouteArgs p) {
  extern __shared__ __align__(16) unsigned char route_smem[];
  const int cols = p.cols, E = p.E, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float* score = reinterpret_cast<float*>(route_smem);                 // [3][TOK][E]: scores, weights, groups
  T* hs = reinterpret_cast<T*>(score + (3 * TOK * E + 3) / 4 * 4);     // [TOK][cols]
  const int n0 = blockIdx.x * TOK, cnt = min(TOK, p.n_tokens - n0);
  const T* src = h + static_cast<size_t>(n0) * cols;
  if constexpr (V == 4) {
    using W = typename std::conditional<sizeof(T) == 4, float4, uint2>::type;
    const int per = cols / 4;
    for (int i = threadIdx.x; i < TOK * per; i += blockDim.x) {
      W v{};
      if (i < cnt * per) v = reinterpret_cast<const W*>(src)[i];
      reinterpret_cast<W*>(hs)[i] = v;
    }
  } else {
    for (int i = threadIdx.x; i < TOK * cols; i += blockDim.x) hs[i] = i < cnt * cols ? src[i] : from_f<T>(0.f);
  }
  __syncthreads();
  for (int e = warp; e < E; e += ROUTE_WARPS) {
    const float* wr = p.router + static_cast<size_t>(e) * cols;
    float acc[TOK];
#pragma unroll
    for (int t = 0; t < TOK; ++t) acc[t] = 0.f;
    if constexpr (V == 4) {
#pragma unroll 4
      for (int c = lane * 4; c < cols; c += 128) {
        const float4 w = *reinterpret_cast<const float4*>(wr + c);
#pragma unroll
        for (int t = 0; t < TOK; ++t) {
          float f[4];
          route_load4<T>(hs + t * cols + c, f);
          acc[t] = fmaf(f[3], w.w, fmaf(f[2], w.z, fmaf(f[1], w.y, fmaf(f[0], w.x, acc[t]))));
        }
      }
    } else {
      for (int c = lane; c < cols; c += 32) {
        const float w = wr[c];
#pragma unroll
        for (int t = 0; t < TOK; ++t) acc[t] = fmaf(to_f(hs[t * cols + c]), w, acc[t]);
      }
    }
#pragma unroll
    for (int t = 0; t < TOK; ++t) {
      const float s = warp_sum(acc[t]);
      if (lane == 0) score[t * E + e] = s;
    }
  }
  __syncthreads();
  for (int t = warp; t < cnt; t += ROUTE_WARPS)
    route_choose(p, n0 + t, lane, score + t * E, score + (TOK + t) * E, score + (2 * TOK + t) * E);
}

// Group the (token, choice) pairs by expert: offsets[e] .. offsets[e+1] index `sorted_pair`, which holds pair ids
// (token * top + choice) in ascending order.  One block; every warp owns a run of consecutive pairs and counts it into a row
// of its own, lanes with the same expert in one addition, so no two warps touch the same counter.
constexpr int GROUP_WARPS = 32;

__global__ void __launch_bounds__(GROUP_WARPS * 32)
moe_group_kernel(const int32_t* __restrict__ top_idx, int32_t* __restrict__ offsets, int32_t* __restrict__ sorted_pair,
                 int n_pairs, int E) {
  extern __shared__ int cursor[];                         // [GROUP_WARPS][E], then [E] totals
  int* total = cursor + GROUP_WARPS * E;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  for (int i = threadIdx.x; i < GROUP_WARPS * E; i += blockDim.x) cursor[i] = 0;
  __syncthreads();
  const int run = (n_pairs + GROUP_WARPS * 32 - 1) / (GROUP_WARPS * 32) * 32;       // whole warps' worth of pairs
  const int i0 = warp * run, i1 = min(n_pairs, i0 + run);
  int* mine = cursor + warp * E;
  for (int i = i0; i < i1; i += 32) {
    const int e = i + lane < i1 ? top_idx[i + lane] : -1;
    const unsigned same = __match_any_sync(0xffffffffu, e);
    if (e >= 0 && (same & ((1u << lane) - 1u)) == 0) mine[e] += __popc(same);
    __syncwarp();
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) {     // per expert: each warp's start inside the group
    int sum = 0;
    for (int w = 0; w < GROUP_WARPS; ++w) { const int c = cursor[w * E + e]; cursor[w * E + e] = sum; sum += c; }
    total[e] = sum;
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    int sum = 0;
    for (int e = 0; e < E; ++e) { const int c = total[e]; total[e] = sum; offsets[e] = sum; sum += c; }
    offsets[E] = sum;
  }
  __syncthreads();
  for (int i = i0; i < i1; i += 32) {
    const int e = i + lane < i1 ? top_idx[i + lane] : -1;
    const unsigned same = __match_any_sync(0xffffffffu, e);
    const int before = __popc(same & ((1u << lane) - 1u));
    if (e >= 0) sorted_pair[total[e] + mine[e] + before] = i + lane;
    __syncwarp();
    if (e >= 0 && before == 0) mine[e] += __popc(same);
    __syncwarp();
  }
}

template <typename T>
static cudaError_t launch_route(const void* h, const RouteArgs& p, cudaStream_t st) {
  // tokens per CTA: one while that leaves the machine short of CTAs, or where the rows do not fit
  const auto smem = [&](int tok) { return ((3 * tok * p.E + 3) / 4 * 4) * sizeof(float) + static_cast<size_t>(tok) * p.cols * sizeof(T); };
  const bool many = p.n_tokens >= 4 * sm_count() && smem(ROUTE_TOKENS) <= 100 * 1024;
  const int tok = many ? ROUTE_TOKENS : 1;
  const bool vec = p.cols % 4 == 0 && aligned16(h) && aligned16(p.router);
  const int grid = (p.n_tokens + tok - 1) / tok;
#define ROUTE_GO(TOK, V) do { \
    auto kern = moe_route_kernel<T, TOK, V>; \
    if (smem(TOK) > 48 * 1024) { \
      const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024); \
      if (e != cudaSuccess) return e; \
    } \
    kern<<<grid, ROUTE_WARPS * 32, smem(TOK), st>>>(static_cast<const T*>(h), p); } while (0)
  if (many) { if (vec) ROUTE_GO(ROUTE_TOKENS, 4); else ROUTE_GO(ROUTE_TOKENS, 1); }
  else { if (vec) ROUTE_GO(1, 4); else ROUTE_GO(1, 1); }
#undef ROUTE_GO
  return cudaSuccess;
}

template <typename T>
static void launch_conv(bool vec4, int grid, cudaStream_t st, const void* u, int64_t u_stride, const float* conv_w, void* state,
                        const int32_t* tok_seq, const int32_t* positions, const int32_t* seq_start, const int32_t* seq_pos0,
                        const int32_t* seq_len, const int32_t* seq_slot, const int32_t* slot_mapping, const float* q_norm_w,
                        const float* k_norm_w, void* q_out, void* k_cache, void* v_cache, int n_tokens, int n_seqs, int H, int G, int d,
                        int dv, int taps, float eps, int C, const ConvHeadOps& ops) {
#define CONV4_GO_T(TP, NCH, ROT, TOK) conv_headnorm_kvwrite_vec4_kernel<T, TP, NCH, ROT, TOK><<<grid, CONV_WARPS * 32, 0, st>>>(static_cast<const T*>(u), u_stride, conv_w, \
      static_cast<const T*>(state), tok_seq, positions, seq_start, seq_pos0, seq_slot, slot_mapping, q_norm_w, k_norm_w, \
      static_cast<T*>(q_out), static_cast<T*>(k_cache), static_cast<T*>(v_cache), n_tokens, H, G, d, dv, eps, ops)
#define CONV4_GO_R(TP, NCH, ROT) do { if (tok == 1) CONV4_GO_T(TP, NCH, ROT, 1); else CONV4_GO_T(TP, NCH, ROT, CONV4_TOKENS); } while (0)
#define CONV4_GO_N(TP, NCH) do { if (ops.rot_dims > 0) CONV4_GO_R(TP, NCH, true); else CONV4_GO_R(TP, NCH, false); } while (0)
#define CONV4_GO(TP) do { if (d <= 128 && dv <= 128) CONV4_GO_N(TP, 1); else CONV4_GO_N(TP, 2); } while (0)
  // rows per warp: one while that leaves the machine short of warps
  const int tok = static_cast<int64_t>(n_tokens) * (H + 2 * G) <= static_cast<int64_t>(sm_count()) * 64 ? 1 : CONV4_TOKENS;
  if (vec4) grid = ((n_tokens + tok - 1) / tok * (H + 2 * G) + CONV_WARPS - 1) / CONV_WARPS;
  if (vec4 && taps == 4) CONV4_GO(4);
  else if (vec4 && taps == 3) CONV4_GO(3);
  else if (vec4 && taps == 2) CONV4_GO(2);
  else if (vec4 && taps == 1) CONV4_GO(1);
  else
    conv_headnorm_kvwrite_kernel<T><<<grid, CONV_WARPS * 32, 0, st>>>(static_cast<const T*>(u), u_stride, conv_w, static_cast<const T*>(state),
        tok_seq, positions, seq_start, seq_pos0, seq_slot, slot_mapping, q_norm_w, k_norm_w, static_cast<T*>(q_out),
        static_cast<T*>(k_cache), static_cast<T*>(v_cache), n_tokens, H, G, d, dv, taps, eps, ops);
#undef CONV4_GO
#undef CONV4_GO_N
#undef CONV4_GO_R
#undef CONV4_GO_T
  if (taps > 1)
    conv_state_update_kernel<T><<<dim3((C + 127) / 128, n_seqs), 128, 0, st>>>(static_cast<const T*>(u), u_stride, static_cast<T*>(state),
        seq_start, seq_pos0, seq_len, seq_slot, n_seqs, C, taps);
}

template <typename T>
static int launch_residual(float* x, const void* a, const void* b, const void* z, const float* zw, int top, float mult,
                           void* h, const float* gain, int rows, int cols, float eps, cudaStream_t st) {
  residual_norm_kernel<T><<<rows, ROW_THREADS, 0, st>>>(x, static_cast<const T*>(a), static_cast<const T*>(b),
                                                         static_cast<const T*>(z), zw, top, mult, static_cast<T*>(h), gain,
                                                         cols, eps);
  return 0;
}

}  // namespace b2

#define LM_DTYPE_OK(dt) ((dt) == B2TTS_DTYPE_BF16 || (dt) == B2TTS_DTYPE_F32)

extern "C" int b2tts_embed_pos_norm(const int32_t* tokens, const int32_t* positions, const void* embed, const void* pos_table,
                                    float* x, void* h, const float* gain, int rows, int cols, int vocab, int max_pos,
                                    float eps, int dtype, void* stream) {
  using namespace b2;
  B2_REQUIRE(rows >= 0 && cols > 0 && vocab > 0 && max_pos > 0, B2TTS_EINVAL, "embed_pos_norm: rows=%d cols=%d", rows, cols);
  B2_REQUIRE(LM_DTYPE_OK(dtype), B2TTS_EINVAL, "embed_pos_norm: dtype %d", dtype);
  if (rows == 0) return B2TTS_OK;
  B2_REQUIRE(tokens && positions && embed && pos_table && x && (!h || gain), B2TTS_EINVAL, "embed_pos_norm: null pointer");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype == B2TTS_DTYPE_BF16)
    embed_pos_norm_kernel<__nv_bfloat16><<<rows, ROW_THREADS, 0, st>>>(tokens, positions, static_cast<const __nv_bfloat16*>(embed),
        static_cast<const __nv_bfloat16*>(pos_table), x, static_cast<__nv_bfloat16*>(h), gain, cols, vocab, max_pos, eps);
  else
    embed_pos_norm_kernel<float><<<rows, ROW_THREADS, 0, st>>>(tokens, positions, static_cast<const float*>(embed),
        static_cast<const float*>(pos_table), x, static_cast<float*>(h), gain, cols, vocab, max_pos, eps);
  B2_CHECK_LAUNCH("embed_pos_norm");
  return B2TTS_OK;
}

extern "C" int b2tts_residual_norm(float* x, const void* a, const void* b, const void* z, const float* zw, int top, float mult,
                                   void* h, const float* gain, int rows, int cols, float eps, int dtype, void* stream) {
  using namespace b2;
  B2_REQUIRE(rows >= 0 && cols > 0 && top >= 0, B2TTS_EINVAL, "residual_norm: rows=%d cols=%d top=%d", rows, cols, top);
  B2_REQUIRE(LM_DTYPE_OK(dtype), B2TTS_EINVAL, "residual_norm: dtype %d", dtype);
  if (rows == 0) return B2TTS_OK;
  B2_REQUIRE(x && (!h || gain) && (!z || (zw && top > 0)), B2TTS_EINVAL, "residual_norm: null pointer");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype == B2TTS_DTYPE_BF16) launch_residual<__nv_bfloat16>(x, a, b, z, zw, top, mult, h, gain, rows, cols, eps, st);
  else launch_residual<float>(x, a, b, z, zw, top, mult, h, gain, rows, cols, eps, st);
  B2_CHECK_LAUNCH("residual_norm");
  return B2TTS_OK;
}

extern "C" int b2tts_gather_gain_norm(const float* x, const int32_t* rows_idx, void* out, const float* gain, int rows, int cols,
                                      float eps, int dtype, void* stream) {
  using namespace b2;
  B2_REQUIRE(rows >= 0 && cols > 0, B2TTS_EINVAL, "gather_gain_norm: rows=%d cols=%d", rows, cols);
  B2_REQUIRE(LM_DTYPE_OK(dtype), B2TTS_EINVAL, "gather_gain_norm: dtype %d", dtype);
  if (rows == 0) return B2TTS_OK;
  B2_REQUIRE(x && out && gain, B2TTS_EINVAL, "gather_gain_norm: null pointer");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype == B2TTS_DTYPE_BF16)
    gather_gain_norm_kernel<__nv_bfloat16><<<rows, ROW_THREADS, 0, st>>>(x, rows_idx, static_cast<__nv_bfloat16*>(out), gain, cols, eps);
  else
    gather_gain_norm_kernel<float><<<rows, ROW_THREADS, 0, st>>>(x, rows_idx, static_cast<float*>(out), gain, cols, eps);
  B2_CHECK_LAUNCH("gather_gain_norm");
  return B2TTS_OK;
}

extern "C" int b2tts_relu_sq(void* y, int64_t n, int dtype, void* stream) {
  using namespace b2;
  B2_REQUIRE(n >= 0 && LM_DTYPE_OK(dtype), B2TTS_EINVAL, "relu_sq: n=%lld dtype=%d", static_cast<long long>(n), dtype);
  if (n == 0) return B2TTS_OK;
  B2_REQUIRE(y, B2TTS_EINVAL, "relu_sq: null pointer");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int grid = static_cast<int>(std::min<int64_t>((n + 255) / 256, 148 * 16));
  if (dtype == B2TTS_DTYPE_BF16) relu_sq_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>(static_cast<__nv_bfloat16*>(y), static_cast<size_t>(n));
  else relu_sq_kernel<float><<<grid, 256, 0, st>>>(static_cast<float*>(y), static_cast<size_t>(n));
  B2_CHECK_LAUNCH("relu_sq");
  return B2TTS_OK;
}

extern "C" int b2tts_rotary_table(const int32_t* positions, const float* freq, float* table, int n, int half, void* stream) {
  using namespace b2;
  B2_REQUIRE(n >= 0 && half >= 0, B2TTS_EINVAL, "rotary_table: n=%d half=%d", n, half);
  if (n == 0 || half == 0) return B2TTS_OK;
  B2_REQUIRE(positions && freq && table, B2TTS_EINVAL, "rotary_table: null pointer");
  const size_t total = static_cast<size_t>(n) * half;
  rotary_table_kernel<<<static_cast<unsigned>((total + 255) / 256), 256, 0, static_cast<cudaStream_t>(stream)>>>(positions, freq, table, n, half);
  B2_CHECK_LAUNCH("rotary_table");
  return B2TTS_OK;
}

extern "C" int b2tts_conv_headnorm_kvwrite(const void* u, int64_t u_stride, const float* conv_w, void* state,
                                           const int32_t* tok_seq, const int32_t* positions, const int32_t* seq_start,
                                           const int32_t* seq_pos0, const int32_t* seq_len, const int32_t* seq_slot,
                                           const int32_t* slot_mapping, const float* q_norm_w, const float* k_norm_w,
                                           void* q_out, void* k_cache, void* v_cache, int n_tokens, int n_seqs, int heads,
                                           int kv_heads, int dim, int vdim, int taps, float eps, const float* rot, int rot_dims,
                                           int flags, int dtype, void* stream) {
  using namespace b2;
  B2_REQUIRE(n_tokens >= 0 && n_seqs >= 0 && heads > 0 && kv_heads > 0 && dim > 0 && vdim > 0, B2TTS_EINVAL,
             "conv_headnorm_kvwrite: bad sizes");
  B2_REQUIRE(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= dim && (rot_dims == 0 || rot), B2TTS_EINVAL,
             "conv_headnorm_kvwrite: %d rotated of %d coordinates", rot_dims, dim);
  B2_REQUIRE((flags & ~(CONV_ROUND | CONV_UNIT_V)) == 0 && (q_norm_w == nullptr) == (k_norm_w == nullptr), B2TTS_EINVAL,
             "conv_headnorm_kvwrite: flags %d, or a norm weight for only one of q and k", flags);
  B2_REQUIRE(taps >= 1 && taps <= CONV_MAX_TAPS, B2TTS_EUNSUPPORTED, "conv_headnorm_kvwrite: taps %d not in 1..%d", taps, CONV_MAX_TAPS);
  B2_REQUIRE(dim <= 32 * CONV_MAX_PER_LANE && vdim <= 32 * CONV_MAX_PER_LANE, B2TTS_EUNSUPPORTED,
             "conv_headnorm_kvwrite: head size above %d", 32 * CONV_MAX_PER_LANE);
  B2_REQUIRE(LM_DTYPE_OK(dtype), B2TTS_EINVAL, "conv_headnorm_kvwrite: dtype %d", dtype);
  if (n_tokens == 0 || n_seqs == 0) return B2TTS_OK;
  B2_REQUIRE(u && conv_w && (state || taps == 1) && tok_seq && positions && seq_start && seq_pos0 && seq_len && seq_slot &&
             slot_mapping && q_out && k_cache && v_cache, B2TTS_EINVAL, "conv_headnorm_kvwrite: null pointer");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int items = n_tokens * (heads + 2 * kv_heads);
  const int grid = (items + CONV_WARPS - 1) / CONV_WARPS;
  const int C = heads * dim + kv_heads * dim + kv_heads * vdim;
  // four channels per lane when every head slice and row starts on a 16-byte (float) / 8-byte (bf16) boundary
  const bool vec4 = dim % 4 == 0 && vdim % 4 == 0 && u_stride % 4 == 0 && dim <= 128 * CONV4_CHUNKS && vdim <= 128 * CONV4_CHUNKS &&
                    (taps == 1 || taps == 2 || taps == 3 || taps == 4) && aligned16(u) && aligned16(q_out) && aligned16(k_cache) &&
                    aligned16(v_cache) && aligned16(conv_w) && (!q_norm_w || (aligned16(q_norm_w) && aligned16(k_norm_w))) && (taps == 1 || aligned16(state)) &&
                    (rot_dims == 0 || (rot_dims % 8 == 0 && aligned16(rot)));
  const ConvHeadOps ops{rot, rot_dims, flags};
  if (dtype == B2TTS_DTYPE_BF16)
    launch_conv<__nv_bfloat16>(vec4, grid, st, u, u_stride, conv_w, state, tok_seq, positions, seq_start, seq_pos0, seq_len, seq_slot,
                               slot_mapping, q_norm_w, k_norm_w, q_out, k_cache, v_cache, n_tokens, n_seqs, heads, kv_heads, dim, vdim, taps, eps, C, ops);
  else
    launch_conv<float>(vec4, grid, st, u, u_stride, conv_w, state, tok_seq, positions, seq_start, seq_pos0, seq_len, seq_slot,
                       slot_mapping, q_norm_w, k_norm_w, q_out, k_cache, v_cache, n_tokens, n_seqs, heads, kv_heads, dim, vdim, taps, eps, C, ops);
  B2_CHECK_LAUNCH("conv_headnorm_kvwrite");
  return B2TTS_OK;
}

extern "C" int b2tts_moe_route(const void* h, const float* router, int32_t* top_idx, float* top_w, int32_t* offsets,
                               int32_t* sorted_pair, int n_tokens, int cols, int experts, int top, float scale,
                               const float* bias, int mode, int groups, int groups_keep, int dtype, void* stream) {
  using namespace b2;
  B2_REQUIRE(n_tokens >= 0 && cols > 0 && experts > 0 && top > 0 && top <= experts, B2TTS_EINVAL, "moe_route: bad sizes");
  B2_REQUIRE(groups >= 1 && experts % groups == 0 && groups_keep >= 1 && groups_keep <= groups && top <= groups_keep * (experts / groups),
             B2TTS_EINVAL, "moe_route: top %d of %d of %d groups over %d experts", top, groups_keep, groups, experts);
  B2_REQUIRE(mode >= 0 && mode <= 2, B2TTS_EINVAL, "moe_route: mode %d", mode);
  B2_REQUIRE(experts <= ROUTE_MAX_EXPERTS && top <= 32, B2TTS_EUNSUPPORTED, "moe_route: experts %d > %d or top %d > 32", experts,
             ROUTE_MAX_EXPERTS, top);
  B2_REQUIRE(LM_DTYPE_OK(dtype), B2TTS_EINVAL, "moe_route: dtype %d", dtype);
  B2_REQUIRE(offsets && sorted_pair, B2TTS_EINVAL, "moe_route: null pointer");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (n_tokens > 0) {
    B2_REQUIRE(h && router && top_idx && top_w, B2TTS_EINVAL, "moe_route: null pointer");
    B2_REQUIRE(static_cast<size_t>(cols) * sizeof(float) + 3 * experts * sizeof(float) + 64 <= 227 * 1024, B2TTS_EUNSUPPORTED,
               "moe_route: rows of %d numbers", cols);
    const RouteArgs p{router, top_idx, top_w, n_tokens, cols, experts, top, scale, bias, mode, groups, groups_keep};
    const cudaError_t e = dtype == B2TTS_DTYPE_BF16 ? launch_route<__nv_bfloat16>(h, p, st) : launch_route<float>(h, p, st);
    if (e != cudaSuccess) return cuda_fail(e, "moe_route");
    B2_CHECK_LAUNCH("moe_route");
  }
  moe_group_kernel<<<1, GROUP_WARPS * 32, (GROUP_WARPS + 1) * experts * sizeof(int), st>>>(top_idx, offsets, sorted_pair, n_tokens * top, experts);
  B2_CHECK_LAUNCH("moe_group");
  return B2TTS_OK;
}
