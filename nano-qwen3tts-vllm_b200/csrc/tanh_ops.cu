// tanh_ops.cu - per-row kernels of decoders whose norms are dynamic tanh (no statistics over the row):
//
//   D(v) = tanh(alpha v) * w + b          alpha one number, w and b vectors
//
//   x <- x + mult * D_out(y),   h = D_in(x)          y = a + sum_k zw[r, k] * z[r * top + k]
//
// Every output element depends on its own column only, so one elementwise launch does the residual update of a finished
// sublayer (a dense output, the weighted outputs of a token's experts, or both) and the input norm of the next one.  With
// `init` the stream starts as an embedding row.  In front of a pass of looped layers the launch writes, instead of h, the
// operand of the pass's input projection: the stream and the token's embedding row side by side (`cat`).  In bf16 the stream
// goes in as two bf16 numbers, hi + lo = x to 16 mantissa bits, so that the projection does not round the residual stream to
// 8 bits.  Plus the gated product of clamped experts for rows that no GEMM epilogue takes.
//
// Activations are `T` = bf16 (serving) or float (the all-32-bit mode); the stream, the norms and every sum are float in both.
// Nothing allocates or synchronises; every launch is graph-capturable.
#include <algorithm>

#include "row_ops.cuh"
#include "clamped_gate.cuh"

namespace b2 {
namespace row {

constexpr int TR_THREADS = 128;

struct TanhNorm { const float* w; const float* b; const float* alpha; };

struct TanhResidualArgs {
  float* x;                               // [rows, cols], in place
  const void* table; const int32_t* index; int table_rows;   // row index[r] (ids outside read as row 0): the start of x, and cat's tail
  const void* a;                          // [rows, cols] or null
  const void* z; const float* zw; int top;                   // [rows * top, cols] with weights [rows, top], or null
  TanhNorm out; float mult;
  TanhNorm in; void* h;                   // [rows, cols] or null
  void* cat;                              // [rows, 3 cols] bf16 (hi | lo | embedding) or [rows, 2 cols] float (x | embedding), or null
  int rows, cols, init, rows_per_thread;
};

template <typename T, int V>
__device__ __forceinline__ void tr_in(const T* p, float* f) {
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
__device__ __forceinline__ void tr_out(T* p, const float* f) {
  if constexpr (V == 1) {
    p[0] = from_f<T>(f[0]);
  } else if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  } else {
    stg_v2(p, make_uint2(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3])));
  }
}

// tanh as 1 - 2 / (e^(2v) + 1) where activations are bf16: absolute error of a float rounding, a quarter of the instructions
template <typename T> __device__ __forceinline__ float tanh_of(float v);
template <> __device__ __forceinline__ float tanh_of<float>(float v) { return tanhf(v); }
template <> __device__ __forceinline__ float tanh_of<__nv_bfloat16>(float v) { return 1.0f - __fdividef(2.0f, __expf(2.0f * v) + 1.0f); }

// A thread owns V consecutive columns and walks `rows_per_thread` rows with the norms' vectors in registers.
template <typename T, int V>
__global__ void __launch_bounds__(TR_THREADS)
tanh_residual_kernel(const TanhResidualArgs p) {
  const int c = (blockIdx.y * TR_THREADS + threadIdx.x) * V;
  if (c >= p.cols) return;
  const int cols = p.cols;
  const T* a = static_cast<const T*>(p.a);
  const T* z = static_cast<const T*>(p.z);
  const T* table = static_cast<const T*>(p.table);
  const bool upd = a != nullptr || z != nullptr;
  float ow[V], ob[V], iw[V], ib[V], oa = 0.f, ia = 0.f;
  if (upd) { tr_in<float, V>(p.out.w + c, ow); tr_in<float, V>(p.out.b + c, ob); oa = p.out.alpha[0]; }
  if (p.h != nullptr) { tr_in<float, V>(p.in.w + c, iw); tr_in<float, V>(p.in.b + c, ib); ia = p.in.alpha[0]; }
  const size_t r0 = static_cast<size_t>(blockIdx.x) * p.rows_per_thread;
  const size_t r1 = min(static_cast<size_t>(p.rows), r0 + p.rows_per_thread);
  for (size_t r = r0; r < r1; ++r) {
    float xv[V], tv[V];
    if (table != nullptr) {
      const int id = p.index[r];
      tr_in<T, V>(table + static_cast<size_t>(id >= 0 && id < p.table_rows ? id : 0) * cols + c, tv);
    }
    if (p.init) {
#pragma unroll
      for (int i = 0; i < V; ++i) xv[i] = tv[i];
    } else {
      tr_in<float, V>(p.x + r * cols + c, xv);
    }
    if (upd) {
      float y[V];
      if (a != nullptr) {
        tr_in<T, V>(a + r * cols + c, y);
      } else {
#pragma unroll
        for (int i = 0; i < V; ++i) y[i] = 0.f;
      }
      for (int k = 0; k < p.top; ++k) {                       // choices in ascending order: a fixed order of additions
        const size_t pr = r * p.top + k;
        const float w = p.zw[pr];
        float zv[V];
        tr_in<T, V>(z + pr * cols + c, zv);
#pragma unroll
        for (int i = 0; i < V; ++i) y[i] = fmaf(w, zv[i], y[i]);
      }
#pragma unroll
      for (int i = 0; i < V; ++i) xv[i] = fmaf(p.mult, fmaf(tanh_of<T>(oa * y[i]), ow[i], ob[i]), xv[i]);
    }
    if (upd || p.init) tr_out<float, V>(p.x + r * cols + c, xv);
    if (p.h != nullptr) {
      float o[V];
#pragma unroll
      for (int i = 0; i < V; ++i) o[i] = fmaf(tanh_of<T>(ia * xv[i]), iw[i], ib[i]);
      tr_out<T, V>(static_cast<T*>(p.h) + r * cols + c, o);
    }
    if (p.cat != nullptr) {
      if constexpr (sizeof(T) == 2) {
        T* cr = static_cast<T*>(p.cat) + r * 3 * cols + c;
        float lo[V];
#pragma unroll
        for (int i = 0; i < V; ++i) lo[i] = xv[i] - __bfloat162float(__float2bfloat16_rn(xv[i]));
        tr_out<T, V>(cr, xv);
        tr_out<T, V>(cr + cols, lo);
        tr_out<T, V>(cr + 2 * cols, tv);
      } else {
        T* cr = static_cast<T*>(p.cat) + r * 2 * cols + c;
        tr_out<T, V>(cr, xv);
        tr_out<T, V>(cr + cols, tv);
      }
    }
  }
}

// out[i] = D(x[rows_idx[i]]) (the rows whose logits are wanted; rows_idx null: row i)
template <typename T>
__global__ void tanh_gather_kernel(const float* __restrict__ x, const int32_t* __restrict__ rows_idx, T* __restrict__ out, const TanhNorm n,
                                   int cols) {
  const size_t r = rows_idx != nullptr ? static_cast<size_t>(rows_idx[blockIdx.x]) : blockIdx.x;
  const float alpha = n.alpha[0];
  for (int c = threadIdx.x; c < cols; c += blockDim.x)
    out[static_cast<size_t>(blockIdx.x) * cols + c] = from_f<T>(tanhf(alpha * x[r * cols + c]) * n.w[c] + n.b[c]);
}

// gu [rows, 2 ff] = [gate | up] -> y [rows, ff]
template <typename T, int V>
__global__ void clamped_gate_mul_kernel(const T* __restrict__ gu, T* __restrict__ y, size_t rows, int ff, float limit, float alpha) {
  const int per = ff / V;
  const size_t n = rows * per;
  for (size_t i = blockIdx.x * static_cast<size_t>(blockDim.x) + threadIdx.x; i < n; i += static_cast<size_t>(gridDim.x) * blockDim.x) {
    const size_t r = i / per;
    const int c = static_cast<int>(i % per) * V;
    float g[V], u[V];
    tr_in<T, V>(gu + r * 2 * ff + c, g);
    tr_in<T, V>(gu + r * 2 * ff + ff + c, u);
#pragma unroll
    for (int j = 0; j < V; ++j) g[j] = clamped_gate(g[j], u[j], limit, alpha);
    tr_out<T, V>(y + r * ff + c, g);
  }
}

}  // namespace row
}  // namespace b2

using namespace b2;
using namespace b2::row;

extern "C" int b2tts_tanh_residual(float* x, const void* table, const int32_t* index, int table_rows, const void* a, const void* z,
                                   const float* zw, int top, const float* out_w, const float* out_b, const float* out_alpha, float mult,
                                   const float* in_w, const float* in_b, const float* in_alpha, void* h, void* cat, int rows, int cols,
                                   int init, int dtype, void* stream) {
  B2_REQUIRE(rows >= 0 && cols > 0 && top >= 0, B2TTS_EINVAL, "tanh_residual: rows=%d cols=%d top=%d", rows, cols, top);
  B2_REQUIRE(B2_ROW_DTYPE_OK(dtype), B2TTS_EINVAL, "tanh_residual: dtype %d", dtype);
  if (rows == 0) return B2TTS_OK;
  B2_REQUIRE(x && (!table || (index && table_rows > 0)) && (table || (!init && !cat)), B2TTS_EINVAL, "tanh_residual: null pointer");
  B2_REQUIRE((!z || (zw && top > 0)) && ((!a && !z) || (out_w && out_b && out_alpha)) && (!h || (in_w && in_b && in_alpha)), B2TTS_EINVAL,
             "tanh_residual: null pointer");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  TanhResidualArgs p{x, table, index, table_rows, a, z, zw, z ? top : 0, {out_w, out_b, out_alpha}, mult, {in_w, in_b, in_alpha}, h, cat,
                     rows, cols, init, 1};
  bool vec = cols % 4 == 0;
  for (const void* q : {static_cast<const void*>(x), table, a, z, static_cast<const void*>(out_w), static_cast<const void*>(out_b),
                        static_cast<const void*>(in_w), static_cast<const void*>(in_b), static_cast<const void*>(h), static_cast<const void*>(cat)})
    vec = vec && (q == nullptr || aligned16(q));
  const int V = vec ? 4 : 1;
  // the vectors are re-read per row only while that is what fills the machine
  while (p.rows_per_thread < 8 && static_cast<int64_t>(rows) * cols / V / (2 * p.rows_per_thread) >= static_cast<int64_t>(sm_count()) * 4096)
    p.rows_per_thread *= 2;
  const dim3 grid((rows + p.rows_per_thread - 1) / p.rows_per_thread, (cols / V + TR_THREADS - 1) / TR_THREADS);
  B2_REQUIRE(grid.y <= 65535, B2TTS_EUNSUPPORTED, "tanh_residual: %d columns", cols);
#define TR_GO(T) do { if (vec) tanh_residual_kernel<T, 4><<<grid, TR_THREADS, 0, st>>>(p); else tanh_residual_kernel<T, 1><<<grid, TR_THREADS, 0, st>>>(p); } while (0)
  if (dtype == B2TTS_DTYPE_BF16) TR_GO(__nv_bfloat16);
  else TR_GO(float);
#undef TR_GO
  B2_CHECK_LAUNCH("tanh_residual");
  return B2TTS_OK;
}

extern "C" int b2tts_tanh_gather(const float* x, const int32_t* rows_idx, void* out, const float* w, const float* b, const float* alpha,
                                 int rows, int cols, int dtype, void* stream) {
  B2_REQUIRE(rows >= 0 && cols > 0, B2TTS_EINVAL, "tanh_gather: rows=%d cols=%d", rows, cols);
  B2_REQUIRE(B2_ROW_DTYPE_OK(dtype), B2TTS_EINVAL, "tanh_gather: dtype %d", dtype);
  if (rows == 0) return B2TTS_OK;
  B2_REQUIRE(x && out && w && b && alpha, B2TTS_EINVAL, "tanh_gather: null pointer");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype == B2TTS_DTYPE_BF16)
    tanh_gather_kernel<__nv_bfloat16><<<rows, 256, 0, st>>>(x, rows_idx, static_cast<__nv_bfloat16*>(out), TanhNorm{w, b, alpha}, cols);
  else
    tanh_gather_kernel<float><<<rows, 256, 0, st>>>(x, rows_idx, static_cast<float*>(out), TanhNorm{w, b, alpha}, cols);
  B2_CHECK_LAUNCH("tanh_gather");
  return B2TTS_OK;
}

extern "C" int b2tts_clamped_gate_mul(const void* gu, void* y, int64_t rows, int ff, float limit, float alpha, int dtype, void* stream) {
  B2_REQUIRE(rows >= 0 && ff > 0, B2TTS_EINVAL, "clamped_gate_mul: rows=%lld ff=%d", static_cast<long long>(rows), ff);
  B2_REQUIRE(B2_ROW_DTYPE_OK(dtype), B2TTS_EINVAL, "clamped_gate_mul: dtype %d", dtype);
  if (rows == 0) return B2TTS_OK;
  B2_REQUIRE(gu && y, B2TTS_EINVAL, "clamped_gate_mul: null pointer");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool vec = ff % 4 == 0 && aligned16(gu) && aligned16(y);
  const int64_t n = rows * (ff / (vec ? 4 : 1));
  const int grid = static_cast<int>(std::min<int64_t>((n + 255) / 256, sm_count() * 16));
#define CG_GO(T) do { if (vec) clamped_gate_mul_kernel<T, 4><<<grid, 256, 0, st>>>(static_cast<const T*>(gu), static_cast<T*>(y), rows, ff, limit, alpha); \
                      else clamped_gate_mul_kernel<T, 1><<<grid, 256, 0, st>>>(static_cast<const T*>(gu), static_cast<T*>(y), rows, ff, limit, alpha); } while (0)
  if (dtype == B2TTS_DTYPE_BF16) CG_GO(__nv_bfloat16);
  else CG_GO(float);
#undef CG_GO
  B2_CHECK_LAUNCH("clamped_gate_mul");
  return B2TTS_OK;
}
