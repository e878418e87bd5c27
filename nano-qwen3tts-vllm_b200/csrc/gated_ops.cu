// gated_ops.cu - per-row kernels of decoders whose sublayers pass an element-wise gate before they join a 32-bit residual
// stream:
//
//   x <- x + sigmoid(z + b) * y   [+ table[index[r]]]  [+ add]           h = N(x) * w         N(v) = v / sqrt(mean(v^2) + eps)
//
// One launch does the gated residual update of a finished sublayer, what a looped range of layers adds in front of a pass (the
// token's embedding again, a vector of the pass), and the input norm of the next sublayer.  With `init` the stream starts from
// zero: the same kernel is the embedding.  Plus the gated product of a GELU feed-forward for rows the native GEMM does not take.
//
// Activations are `T` = bf16 (serving) or float (the all-32-bit mode); the stream, gates, sums of squares and norms are float
// in both.  Nothing allocates or synchronises; every launch is graph-capturable.
#include <algorithm>

#include "row_ops.cuh"
#include "umma.cuh"

namespace b2 {
namespace row {

constexpr int GR_THREADS = 256;
constexpr int GR_KEEP = 4;                // column groups a thread keeps in registers: rows of up to 4 * 4 * 256 columns

struct GatedResidualArgs {
  float* x;                               // [rows, cols], in place
  const void* y;                          // [rows, cols] or null
  const void* z; int64_t ldz;             // gate pre-activations, or null (the sublayer's result is added as it is)
  const float* zb;                        // [cols] or null
  const void* table; const int32_t* index; int table_rows;   // row index[r] is added (ids outside read as row 0), or null
  const float* add;                       // [cols] or null
  const float* w;                         // [cols] (with h)
  void* h;                                // [rows, cols] or null
  int cols, init;
  float eps;
};

template <typename T, int V>
__device__ __forceinline__ void cols_in(const T* p, float* f) {
  if constexpr (V == 1) {
    f[0] = to_f(p[0]);
  } else if constexpr (sizeof(T) == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
  } else {
    const uint2 r = ldg_v2(p);
    f[0] = bf16lo(r.x); f[1] = bf16hi(r.x); f[2] = bf16lo(r.y); f[3] = bf16hi(r.y);
  }
}
template <typename T, int V>
__device__ __forceinline__ void cols_out(T* p, const float* f) {
  if constexpr (V == 1) {
    p[0] = from_f<T>(f[0]);
  } else if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  } else {
    stg_v2(p, make_uint2(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3])));
  }
}

// One CTA per row.  V = 4: vector accesses and the new row in registers until its norm is known; V = 1: any row.
template <typename T, int V>
__global__ void __launch_bounds__(GR_THREADS)
gated_residual_kernel(const GatedResidualArgs p) {
  __shared__ float red[33];
  const size_t r = blockIdx.x;
  const int cols = p.cols;
  float* xr = p.x + r * cols;
  const T* yr = p.y != nullptr ? static_cast<const T*>(p.y) + r * cols : nullptr;
  const T* zr = p.z != nullptr ? static_cast<const T*>(p.z) + r * p.ldz : nullptr;
  const T* tr = nullptr;
  if (p.table != nullptr) {
    const int id = p.index[r];
    tr = static_cast<const T*>(p.table) + static_cast<size_t>(id >= 0 && id < p.table_rows ? id : 0) * cols;
  }
  float ssq = 0.f;
  auto update = [&](int c, float* xv) {                   // the new values of columns c .. c + V - 1
    float t[V], g[V];
    if (p.init) {
#pragma unroll
      for (int i = 0; i < V; ++i) xv[i] = 0.f;
    } else {
      cols_in<float, V>(xr + c, xv);
    }
    if (yr != nullptr) {
      cols_in<T, V>(yr + c, t);
      if (zr != nullptr) {
        cols_in<T, V>(zr + c, g);
        float b[V];
#pragma unroll
        for (int i = 0; i < V; ++i) b[i] = 0.f;
        if (p.zb != nullptr) cols_in<float, V>(p.zb + c, b);
#pragma unroll
        for (int i = 0; i < V; ++i) t[i] *= sigmoid_f(g[i] + b[i]);
      }
#pragma unroll
      for (int i = 0; i < V; ++i) xv[i] += t[i];
    }
    if (tr != nullptr) {
      cols_in<T, V>(tr + c, t);
#pragma unroll
      for (int i = 0; i < V; ++i) xv[i] += t[i];
    }
    if (p.add != nullptr) {
      cols_in<float, V>(p.add + c, t);
#pragma unroll
      for (int i = 0; i < V; ++i) xv[i] += t[i];
    }
    cols_out<float, V>(xr + c, xv);
#pragma unroll
    for (int i = 0; i < V; ++i) ssq += xv[i] * xv[i];
  };
  auto emit = [&](int c, const float* xv, float inv) {
    float w[V], o[V];
    cols_in<float, V>(p.w + c, w);
#pragma unroll
    for (int i = 0; i < V; ++i) o[i] = xv[i] * inv * w[i];
    cols_out<T, V>(static_cast<T*>(p.h) + r * cols + c, o);
  };
  if constexpr (V == 4) {
    float keep[GR_KEEP][V];
#pragma unroll
    for (int it = 0; it < GR_KEEP; ++it) {
      const int c = (threadIdx.x + it * GR_THREADS) * V;
      if (c < cols) update(c, keep[it]);
    }
    if (p.h == nullptr) return;
    const float inv = 1.0f / sqrtf(block_sum(ssq, red) / static_cast<float>(cols) + p.eps);
#pragma unroll
    for (int it = 0; it < GR_KEEP; ++it) {
      const int c = (threadIdx.x + it * GR_THREADS) * V;
      if (c < cols) emit(c, keep[it], inv);
    }
  } else {
    float xv[V];
    for (int c = threadIdx.x; c < cols; c += GR_THREADS) update(c, xv);
    if (p.h == nullptr) return;
    const float inv = 1.0f / sqrtf(block_sum(ssq, red) / static_cast<float>(cols) + p.eps);
    for (int c = threadIdx.x; c < cols; c += GR_THREADS) {   // the same thread wrote these columns above
      xv[0] = xr[c];
      emit(c, xv, inv);
    }
  }
}

// y[r, c] = gelu_tanh(gu[r, c]) * gu[r, ff + c]; V = 4 needs ff % 4 == 0
template <typename T, int V>
__global__ void __launch_bounds__(256)
gelu_mul_kernel(const T* __restrict__ gu, T* __restrict__ y, size_t rows, int ff) {
  const size_t n = rows * ff / V;
  for (size_t i = blockIdx.x * static_cast<size_t>(blockDim.x) + threadIdx.x; i < n; i += static_cast<size_t>(gridDim.x) * blockDim.x) {
    const size_t r = i * V / ff;
    const int c = static_cast<int>(i * V - r * ff);
    float g[V], u[V];
    cols_in<T, V>(gu + r * 2 * ff + c, g);
    cols_in<T, V>(gu + r * 2 * ff + ff + c, u);
#pragma unroll
    for (int e = 0; e < V; ++e) g[e] = gelu_tanh_f(g[e]) * u[e];
    cols_out<T, V>(y + r * ff + c, g);
  }
}

}  // namespace row
}  // namespace b2

using namespace b2;
using namespace b2::row;

extern "C" int b2tts_gated_residual(float* x, const void* y, const void* z, int64_t ldz, const float* zb, const void* table,
                                    const int32_t* index, int table_rows, const float* add, const float* w, void* h, int rows,
                                    int cols, int init, float eps, int dtype, void* stream) {
  B2_REQUIRE(rows >= 0 && cols > 0, B2TTS_EINVAL, "gated_residual: rows=%d cols=%d", rows, cols);
  B2_REQUIRE(B2_ROW_DTYPE_OK(dtype), B2TTS_EINVAL, "gated_residual: dtype %d", dtype);
  if (rows == 0) return B2TTS_OK;
  B2_REQUIRE(x && (!h || w) && (!z || y) && (!table || (index && table_rows > 0)), B2TTS_EINVAL, "gated_residual: null pointer");
  const GatedResidualArgs p{x, y, z, ldz, zb, table, index, table_rows, add, w, h, cols, init, eps};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const size_t el = dtype == B2TTS_DTYPE_BF16 ? 2 : 4;
  // vector accesses: rows of whole 4-column groups, every tensor on 16-byte boundaries, gate rows on 4-element ones
  bool vec = cols % 4 == 0 && cols <= 4 * GR_KEEP * GR_THREADS;
  for (const void* q : {static_cast<const void*>(x), y, static_cast<const void*>(zb), table, static_cast<const void*>(add),
                        static_cast<const void*>(w), static_cast<const void*>(h)})
    vec = vec && (q == nullptr || aligned16(q));
  if (z != nullptr) vec = vec && ldz % 4 == 0 && reinterpret_cast<uintptr_t>(z) % (4 * el) == 0;
  if (dtype == B2TTS_DTYPE_BF16) {
    if (vec) gated_residual_kernel<__nv_bfloat16, 4><<<rows, GR_THREADS, 0, st>>>(p);
    else gated_residual_kernel<__nv_bfloat16, 1><<<rows, GR_THREADS, 0, st>>>(p);
  } else {
    if (vec) gated_residual_kernel<float, 4><<<rows, GR_THREADS, 0, st>>>(p);
    else gated_residual_kernel<float, 1><<<rows, GR_THREADS, 0, st>>>(p);
  }
  B2_CHECK_LAUNCH("gated_residual");
  return B2TTS_OK;
}

extern "C" int b2tts_gelu_mul(const void* gu, void* y, int64_t rows, int ff, int dtype, void* stream) {
  B2_REQUIRE(rows >= 0 && ff > 0, B2TTS_EINVAL, "gelu_mul: rows=%lld ff=%d", static_cast<long long>(rows), ff);
  B2_REQUIRE(B2_ROW_DTYPE_OK(dtype), B2TTS_EINVAL, "gelu_mul: dtype %d", dtype);
  if (rows == 0) return B2TTS_OK;
  B2_REQUIRE(gu && y, B2TTS_EINVAL, "gelu_mul: null pointer");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool vec = ff % 4 == 0 && aligned16(gu) && aligned16(y);
  const size_t n = static_cast<size_t>(rows) * ff / (vec ? 4 : 1);
  const unsigned grid = static_cast<unsigned>(std::min<size_t>((n + 255) / 256, static_cast<size_t>(sm_count()) * 32));
  if (dtype == B2TTS_DTYPE_BF16) {
    using B = __nv_bfloat16;
    if (vec) gelu_mul_kernel<B, 4><<<grid, 256, 0, st>>>(static_cast<const B*>(gu), static_cast<B*>(y), rows, ff);
    else gelu_mul_kernel<B, 1><<<grid, 256, 0, st>>>(static_cast<const B*>(gu), static_cast<B*>(y), rows, ff);
  } else {
    if (vec) gelu_mul_kernel<float, 4><<<grid, 256, 0, st>>>(static_cast<const float*>(gu), static_cast<float*>(y), rows, ff);
    else gelu_mul_kernel<float, 1><<<grid, 256, 0, st>>>(static_cast<const float*>(gu), static_cast<float*>(y), rows, ff);
  }
  B2_CHECK_LAUNCH("gelu_mul");
  return B2TTS_OK;
}
