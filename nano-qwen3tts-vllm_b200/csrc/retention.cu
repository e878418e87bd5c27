// retention.cu - linear attention with a fixed decay per head, carried from token to token in per-sequence state slots:
//
//   q, k rotated (coordinate i with i + dims/2), k times k_scale        S <- decay_h S + k v^T,   o = S^T q
//   out = o / sqrt(mean(o^2) + eps) * silu(gate)                        (mean over the head's values)
//
// Three forms of the recurrence share a call; each takes the sequences of the step that suit it:
//   one new token      retention_step_kernel: one CTA per (sequence, head) rotates q and k, streams the state through
//                      registers once (read, updated, read out, written back) and, when the whole step is single tokens,
//                      norms and gates the head's output before it leaves the CTA;
//   prompt portions    retention_chunk_kernel (bf16 activations, key sizes 32, 64, 96, 128): chunks of 64 tokens on the
//                      tensor cores, the state in registers from chunk to chunk;
//   anything else      rotated float copies of q, k, v and the token-by-token scan of recurrent.cu.
// The state is float in one slot per live sequence; it counts as zero when the portion starts at position 0, so a slot is
// never cleared between owners.  Rotated q and k, decays, sums, norm and gate are float whatever the activation type.
#include <math.h>

#include <algorithm>

#include "row_ops.cuh"

namespace b2 {
namespace row {

struct RetArgs {
  const void* q; int64_t ldq;             // (row, head h, i) at q[row * ldq + h * d + i]
  const void* k; int64_t ldk;
  const void* v; int64_t ldv;             // (row, head h, c) at v[row * ldv + h * dv + c]
  const float* rot; int rot_dims;         // [rows, rot_dims]: cosines, then sines (rot_dims 0: no rotation)
  const float* decay;                     // [H]
  float k_scale;
  float* state;                           // [slots, H, d, dv]
  float* o;                               // [rows, H * dv] float: raw read-outs
  const void* gate; int64_t ldg;          // [rows, H * dv] column slice
  void* out;                              // [rows, H * dv] normed and gated
  const int32_t* seq_start; const int32_t* seq_pos0; const int32_t* seq_len; const int32_t* seq_slot;
  int H, d, dv;
  float eps;
};

// rotated coordinate i of the head vector p (d coordinates); rt: the token's row of the table
template <typename T>
__device__ __forceinline__ float rotated(const T* p, int i, const float* rt, int rot_dims) {
  const int half = rot_dims >> 1;
  const float x = to_f(p[i]);
  if (i < half) return x * rt[i] - to_f(p[i + half]) * rt[half + i];
  if (i < rot_dims) return x * rt[i - half] + to_f(p[i - half]) * rt[i];
  return x;
}

// ------------------------------------------------------------------ float copies for the token-by-token scan
// row t of qkv = [q rotated: H d | k rotated and scaled: H d | v: H dv]
template <typename T>
__global__ void __launch_bounds__(256)
retention_prep_kernel(const RetArgs a, float* __restrict__ qkv) {
  const size_t t = blockIdx.x;
  const int hd = a.H * a.d, hv = a.H * a.dv;
  const float* rt = a.rot + t * a.rot_dims;
  const T* q = static_cast<const T*>(a.q) + t * a.ldq;
  const T* k = static_cast<const T*>(a.k) + t * a.ldk;
  const T* v = static_cast<const T*>(a.v) + t * a.ldv;
  float* o = qkv + t * (2 * static_cast<size_t>(hd) + hv);
  for (int c = threadIdx.x; c < hd; c += blockDim.x) {
    const int h0 = c / a.d * a.d, i = c - h0;
    o[c] = rotated(q + h0, i, rt, a.rot_dims);
    o[hd + c] = rotated(k + h0, i, rt, a.rot_dims) * a.k_scale;
  }
  for (int c = threadIdx.x; c < hv; c += blockDim.x) o[2 * hd + c] = to_f(v[c]);
}

// ------------------------------------------------------------------ one new token per sequence
// 256 threads; dv / 4 of them share a state row (four columns each), the row groups walk the d rows.  RS_BATCH rows of a
// thread are asked for before the first is used.  dv is a multiple of 4, d and dv at most 256.
constexpr int RS_THREADS = 256, RS_BATCH = 8;

template <typename T, bool FUSED>
__global__ void __launch_bounds__(RS_THREADS)
retention_step_kernel(const RetArgs a) {
  __shared__ float qs[256], ks[256];
  __shared__ __align__(16) float part[RS_THREADS * 4];
  __shared__ float red[33];
  const int b = blockIdx.y, h = blockIdx.x, tid = threadIdx.x;
  const int len = a.seq_len[b], d = a.d, dv = a.dv, H = a.H;
  const size_t t = a.seq_start[b], obase = t * H * dv + static_cast<size_t>(h) * dv;
  if (len != 1) {
    if (FUSED && len <= 0)                                 // padding row
      for (int c = tid; c < dv; c += RS_THREADS) static_cast<T*>(a.out)[obase + c] = from_f<T>(0.f);
    return;
  }
  const bool fresh = a.seq_pos0[b] == 0;
  const int tpr = dv >> 2, groups = RS_THREADS / tpr, grp = tid / tpr, c4 = (tid - grp * tpr) * 4;
  const bool live = grp < groups;
  float* S = a.state + (static_cast<size_t>(a.seq_slot[b]) * H + h) * d * dv + c4;
  float4 s[RS_BATCH];
  auto fetch = [&](int r0) {
#pragma unroll
    for (int u = 0; u < RS_BATCH; ++u) {
      const int r = r0 + u * groups;
      s[u] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (live && !fresh && r < d) s[u] = *reinterpret_cast<const float4*>(S + static_cast<size_t>(r) * dv);
    }
  };
  fetch(grp);                                              // in flight while q and k are rotated
  const float* rt = a.rot + t * a.rot_dims;
  const T* qp = static_cast<const T*>(a.q) + t * a.ldq + static_cast<size_t>(h) * d;
  const T* kp = static_cast<const T*>(a.k) + t * a.ldk + static_cast<size_t>(h) * d;
  const T* vp = static_cast<const T*>(a.v) + t * a.ldv + static_cast<size_t>(h) * dv;
  if (tid < d) {
    qs[tid] = rotated(qp, tid, rt, a.rot_dims);
    ks[tid] = rotated(kp, tid, rt, a.rot_dims) * a.k_scale;
  }
  float4 v = make_float4(0.f, 0.f, 0.f, 0.f), o = v;
  if (live) v = make_float4(to_f(vp[c4]), to_f(vp[c4 + 1]), to_f(vp[c4 + 2]), to_f(vp[c4 + 3]));
  const float dec = a.decay[h];
  __syncthreads();
  for (int r0 = grp; r0 < d && live; r0 += RS_BATCH * groups) {
    if (r0 != grp) fetch(r0);
#pragma unroll
    for (int u = 0; u < RS_BATCH; ++u) {
      const int r = r0 + u * groups;
      if (r < d) {
        const float kr = ks[r], qr = qs[r];
        s[u].x = dec * s[u].x + kr * v.x; o.x += s[u].x * qr;
        s[u].y = dec * s[u].y + kr * v.y; o.y += s[u].y * qr;
        s[u].z = dec * s[u].z + kr * v.z; o.z += s[u].z * qr;
        s[u].w = dec * s[u].w + kr * v.w; o.w += s[u].w * qr;
        *reinterpret_cast<float4*>(S + static_cast<size_t>(r) * dv) = s[u];
      }
    }
  }
  if (live) *reinterpret_cast<float4*>(part + grp * dv + c4) = o;
  __syncthreads();
  float val = 0.f;                                         // dv <= 256: one value per thread
  if (tid < dv)
    for (int g = 0; g < groups; ++g) val += part[g * dv + tid];
  if constexpr (FUSED) {
    const float inv = 1.0f / sqrtf(block_sum(val * val, red) / static_cast<float>(dv) + a.eps);
    if (tid < dv) {
      const float g = to_f((static_cast<const T*>(a.gate) + t * a.ldg + static_cast<size_t>(h) * dv)[tid]);
      static_cast<T*>(a.out)[obase + tid] = from_f<T>(val * inv * silu_f(g));
    }
  } else if (tid < dv) {
    a.o[obase + tid] = val;
  }
}

// ------------------------------------------------------------------ prompt portions on the tensor cores (bf16 activations)
// One CTA of eight warps per (sequence, head, DVT value columns) walks the portion in chunks of 64 tokens.  With L the
// chunk's length, g the decay and S the state in front of the chunk,
//   O_i = g^(i+1) S^T q_i + sum_(j <= i) g^(i-j) (q_i . k_j) v_j,        S <- g^L S + sum_j g^(L-1-j) k_j v_j^T.
// Rotated q and k, the weighted scores and S are floats: each enters its product as a bf16 pair hi + lo (16 mantissa bits;
// the lo * lo term is dropped), v is bf16 as it comes, every sum is float (m16n8k16 MMAs).  Warp (wr, wc) owns rows 16 wr .. + 15
// of O; wc halves the contraction (key columns of the scores, key channels of S^T q) and the two partial sums meet in shared
// memory.  For the state, warp w owns key channels 16 w .. + 15, in registers across the chunks; a copy as hi + lo in shared
// memory serves the next chunk's S^T q.  The next chunk's rows arrive by 16-byte asynchronous copies meanwhile.
constexpr int RC_C = 64, RC_THREADS = 256;

__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(x, y);
  lo = pack_bf16(x - bf16lo(hi), y - bf16hi(hi));
}
// 8 floats -> 16 bytes of bf16 and 16 bytes of remainders
__device__ __forceinline__ void store_split8(__nv_bfloat16* hi, __nv_bfloat16* lo, const float* f) {
  uint4 h, l;
  split2(f[0], f[1], h.x, l.x); split2(f[2], f[3], h.y, l.y);
  split2(f[4], f[5], h.z, l.z); split2(f[6], f[7], h.w, l.w);
  *reinterpret_cast<uint4*>(hi) = h;
  *reinterpret_cast<uint4*>(lo) = l;
}
__device__ __forceinline__ void unpack8(const uint4& r, float* f) {
  f[0] = bf16lo(r.x); f[1] = bf16hi(r.x); f[2] = bf16lo(r.y); f[3] = bf16hi(r.y);
  f[4] = bf16lo(r.z); f[5] = bf16hi(r.z); f[6] = bf16lo(r.w); f[7] = bf16hi(r.w);
}
__device__ __forceinline__ void load8f(const float* p, float* f) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}

template <int D, int DVT> struct ChunkSmem {
  static constexpr int KS = D + 8, VS = DVT + 8, OS = DVT + 4;   // padded rows: 16-byte aligned, ldmatrix rows in distinct banks
  __nv_bfloat16 raw[2][RC_C * D];                                 // q, k of the next chunk as projected
  __nv_bfloat16 qh[RC_C * KS], ql[RC_C * KS], kh[RC_C * KS], kl[RC_C * KS];
  __nv_bfloat16 v[2][RC_C * VS];
  __nv_bfloat16 sh[D * VS], sl[D * VS];
  float ob[RC_C * OS];
  float pw[RC_C + 4];                                             // g^0 .. g^64
};

template <int D, int DVT>
__global__ void __launch_bounds__(RC_THREADS)
retention_chunk_kernel(const RetArgs a) {
  using Sm = ChunkSmem<D, DVT>;
  constexpr int KS = Sm::KS, VS = Sm::VS, OS = Sm::OS, NT = DVT / 8;
  extern __shared__ __align__(16) unsigned char sm_raw[];
  Sm& sm = *reinterpret_cast<Sm*>(sm_raw);
  const int b = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * DVT;
  const int len = a.seq_len[b];
  if (len <= 1) return;                                    // one-token and padding rows belong to the step kernel
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, wr = warp & 3, wc = warp >> 2;
  const int g4 = lane >> 2, c2 = 2 * (lane & 3);
  const int H = a.H, dv = a.dv;
  const size_t start = a.seq_start[b];
  using B = __nv_bfloat16;
  const B* qg = static_cast<const B*>(a.q) + start * a.ldq + static_cast<size_t>(h) * D;
  const B* kg = static_cast<const B*>(a.k) + start * a.ldk + static_cast<size_t>(h) * D;
  const B* vg = static_cast<const B*>(a.v) + start * a.ldv + static_cast<size_t>(h) * dv + v0;
  const float* rg = a.rot + start * a.rot_dims;
  float* Sg = a.state + (static_cast<size_t>(a.seq_slot[b]) * H + h) * D * dv + v0;
  float* og = a.o + start * H * dv + static_cast<size_t>(h) * dv + v0;
  auto load_chunk = [&](int t0, int stage) {
    for (int idx = tid; idx < RC_C * (D / 8); idx += RC_THREADS) {
      const int j = idx / (D / 8), ch = (idx % (D / 8)) * 8;
      const bool ok = t0 + j < len;
      const size_t row = ok ? t0 + j : 0;
      cp_async_16(sm.raw[0] + j * D + ch, qg + row * a.ldq + ch, ok);
      cp_async_16(sm.raw[1] + j * D + ch, kg + row * a.ldk + ch, ok);
    }
    for (int idx = tid; idx < RC_C * (DVT / 8); idx += RC_THREADS) {
      const int j = idx / (DVT / 8), ch = (idx % (DVT / 8)) * 8;
      const bool ok = t0 + j < len;
      cp_async_16(sm.v[stage] + j * VS + ch, vg + (ok ? t0 + j : 0) * a.ldv + ch, ok);
    }
  };
  load_chunk(0, 0);
  cp_async_commit();
  if (tid <= RC_C) sm.pw[tid] = powf(a.decay[h], static_cast<float>(tid));
  // the state's fragments: rows mt * 16 + g4 (+ 8), columns nt * 8 + c2 (+ 1)
  const bool owner = warp < D / 16;
  const int srow = warp * 16 + g4;
  float S[NT][4];
  const bool carried = a.seq_pos0[b] > 0;
#pragma unroll
  for (int nt = 0; nt < NT; ++nt) {
#pragma unroll
    for (int e = 0; e < 4; ++e) S[nt][e] = 0.f;
    if (owner && carried) {
      const float2 x = *reinterpret_cast<const float2*>(Sg + static_cast<size_t>(srow) * dv + nt * 8 + c2);
      const float2 y = *reinterpret_cast<const float2*>(Sg + static_cast<size_t>(srow + 8) * dv + nt * 8 + c2);
      S[nt][0] = x.x; S[nt][1] = x.y; S[nt][2] = y.x; S[nt][3] = y.y;
    }
  }
  const int half = a.rot_dims >> 1, hch = half / 8;        // half is a multiple of eight
  for (int t0 = 0, stage = 0; t0 < len; t0 += RC_C, stage ^= 1) {
    const int L = min(RC_C, len - t0);
    cp_async_wait<0>();
    __syncthreads();                                       // the chunk has landed; the previous one is consumed
    // ---- rotate, scale, split; the state's copy
    for (int idx = tid; idx < RC_C * (D / 16); idx += RC_THREADS) {
      const int j = idx / (D / 16), cc = idx % (D / 16);   // an item: two groups of eight channels, a rotation pair or two that pass
      float x0[8], x1[8], y0[8], y1[8];
      const bool turn = cc < hch;
      const int i0 = turn ? cc * 8 : a.rot_dims + (cc - hch) * 16, i1 = turn ? half + cc * 8 : i0 + 8;
      unpack8(*reinterpret_cast<const uint4*>(sm.raw[0] + j * D + i0), x0);
      unpack8(*reinterpret_cast<const uint4*>(sm.raw[0] + j * D + i1), x1);
      unpack8(*reinterpret_cast<const uint4*>(sm.raw[1] + j * D + i0), y0);
      unpack8(*reinterpret_cast<const uint4*>(sm.raw[1] + j * D + i1), y1);
      if (turn && j < L) {
        float cs[8], sn[8];
        const float* rt = rg + static_cast<size_t>(t0 + j) * a.rot_dims;
        load8f(rt + i0, cs);
        load8f(rt + half + i0, sn);
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const float u = x0[e], w = y0[e];
          x0[e] = u * cs[e] - x1[e] * sn[e]; x1[e] = x1[e] * cs[e] + u * sn[e];
          y0[e] = w * cs[e] - y1[e] * sn[e]; y1[e] = y1[e] * cs[e] + w * sn[e];
        }
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) { y0[e] *= a.k_scale; y1[e] *= a.k_scale; }
      store_split8(sm.qh + j * KS + i0, sm.ql + j * KS + i0, x0);
      store_split8(sm.qh + j * KS + i1, sm.ql + j * KS + i1, x1);
      store_split8(sm.kh + j * KS + i0, sm.kl + j * KS + i0, y0);
      store_split8(sm.kh + j * KS + i1, sm.kl + j * KS + i1, y1);
    }
    if (owner) {
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        uint32_t hi, lo;
        split2(S[nt][0], S[nt][1], hi, lo);
        *reinterpret_cast<uint32_t*>(sm.sh + srow * VS + nt * 8 + c2) = hi;
        *reinterpret_cast<uint32_t*>(sm.sl + srow * VS + nt * 8 + c2) = lo;
        split2(S[nt][2], S[nt][3], hi, lo);
        *reinterpret_cast<uint32_t*>(sm.sh + (srow + 8) * VS + nt * 8 + c2) = hi;
        *reinterpret_cast<uint32_t*>(sm.sl + (srow + 8) * VS + nt * 8 + c2) = lo;
      }
    }
    __syncthreads();
    if (t0 + RC_C < len) load_chunk(t0 + RC_C, stage ^ 1);
    cp_async_commit();
    // ---- S^T q over this warp's half of the key channels, scaled by g^(i+1)
    float o[NT][4];
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[nt][e] = 0.f;
    const int arow = (wr * 16 + (lane & 15)) * KS + (lane >> 4) * 8;         // A fragments of q
    const int trow = ((lane >> 3) & 1) * 8 + (lane & 7), tcol = (lane >> 4) * 8;   // B fragments by transposed loads
    const bool rows_live = wr * 16 < L;
    if (rows_live && (carried || t0 > 0)) {
#pragma unroll
      for (int ks = 0; ks < D / 32; ++ks) {
        const int kk = wc * (D / 2) + ks * 16;
        uint32_t ah[4], al[4];
        ldsm_x4(ah[0], ah[1], ah[2], ah[3], sm.qh + arow + kk);
        ldsm_x4(al[0], al[1], al[2], al[3], sm.ql + arow + kk);
#pragma unroll
        for (int np = 0; np < DVT / 16; ++np) {
          uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
          ldsm_x4_t(h0, h1, h2, h3, sm.sh + (kk + trow) * VS + np * 16 + tcol);
          ldsm_x4_t(l0, l1, l2, l3, sm.sl + (kk + trow) * VS + np * 16 + tcol);
          mma_bf16_16816(o[2 * np], ah, h0, h1);
          mma_bf16_16816(o[2 * np + 1], ah, h2, h3);
          mma_bf16_16816(o[2 * np], ah, l0, l1);
          mma_bf16_16816(o[2 * np + 1], ah, l2, l3);
          mma_bf16_16816(o[2 * np], al, h0, h1);
          mma_bf16_16816(o[2 * np + 1], al, h2, h3);
        }
      }
      const float s0 = sm.pw[wr * 16 + g4 + 1], s1 = sm.pw[wr * 16 + g4 + 9];
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) { o[nt][0] *= s0; o[nt][1] *= s0; o[nt][2] *= s1; o[nt][3] *= s1; }
    }
    // ---- scores against this warp's half of the chunk's keys, weighted, times v
    if (rows_live && wc * 32 <= wr * 16 + 15) {
      float s[4][4];
#pragma unroll
      for (int nt = 0; nt < 4; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[nt][e] = 0.f;
#pragma unroll
      for (int ks = 0; ks < D / 16; ++ks) {
        uint32_t ah[4], al[4];
        ldsm_x4(ah[0], ah[1], ah[2], ah[3], sm.qh + arow + ks * 16);
        ldsm_x4(al[0], al[1], al[2], al[3], sm.ql + arow + ks * 16);
#pragma unroll
        for (int np = 0; np < 2; ++np) {
          const int bo = (wc * 32 + np * 16 + (lane >> 4) * 8 + (lane & 7)) * KS + ks * 16 + ((lane >> 3) & 1) * 8;
          uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
          ldsm_x4(h0, h1, h2, h3, sm.kh + bo);
          ldsm_x4(l0, l1, l2, l3, sm.kl + bo);
          mma_bf16_16816(s[2 * np], ah, h0, h1);
          mma_bf16_16816(s[2 * np + 1], ah, h2, h3);
          mma_bf16_16816(s[2 * np], ah, l0, l1);
          mma_bf16_16816(s[2 * np + 1], ah, l2, l3);
          mma_bf16_16816(s[2 * np], al, h0, h1);
          mma_bf16_16816(s[2 * np + 1], al, h2, h3);
        }
      }
#pragma unroll
      for (int nt = 0; nt < 4; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int back = wr * 16 + g4 + (e >> 1) * 8 - (wc * 32 + nt * 8 + c2 + (e & 1));
          s[nt][e] = back >= 0 ? s[nt][e] * sm.pw[back] : 0.f;
        }
#pragma unroll
      for (int kk = 0; kk < 2; ++kk) {
        uint32_t ah[4], al[4];
        split2(s[2 * kk][0], s[2 * kk][1], ah[0], al[0]);
        split2(s[2 * kk][2], s[2 * kk][3], ah[1], al[1]);
        split2(s[2 * kk + 1][0], s[2 * kk + 1][1], ah[2], al[2]);
        split2(s[2 * kk + 1][2], s[2 * kk + 1][3], ah[3], al[3]);
#pragma unroll
        for (int np = 0; np < DVT / 16; ++np) {
          uint32_t b0, b1, b2, b3;
          ldsm_x4_t(b0, b1, b2, b3, sm.v[stage] + (wc * 32 + kk * 16 + trow) * VS + np * 16 + tcol);
          mma_bf16_16816(o[2 * np], ah, b0, b1);
          mma_bf16_16816(o[2 * np + 1], ah, b2, b3);
          mma_bf16_16816(o[2 * np], al, b0, b1);
          mma_bf16_16816(o[2 * np + 1], al, b2, b3);
        }
      }
    }
    if (wc == 1 && rows_live) {
      float* ob = sm.ob + (wr * 16 + g4) * OS + c2;
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        *reinterpret_cast<float2*>(ob + nt * 8) = make_float2(o[nt][0], o[nt][1]);
        *reinterpret_cast<float2*>(ob + 8 * OS + nt * 8) = make_float2(o[nt][2], o[nt][3]);
      }
    }
    // ---- the state behind the chunk: 16 key channels per warp, contraction over the chunk's tokens
    if (owner) {
      const float gl = sm.pw[L];
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[nt][e] *= gl;
#pragma unroll
      for (int js = 0; js < RC_C / 16; ++js) {
        if (js * 16 >= L) break;
        const int ko = (js * 16 + (lane >> 4) * 8 + (lane & 7)) * KS + warp * 16 + ((lane >> 3) & 1) * 8;
        uint32_t ah[4], al[4];
        ldsm_x4_t(ah[0], ah[1], ah[2], ah[3], sm.kh + ko);
        ldsm_x4_t(al[0], al[1], al[2], al[3], sm.kl + ko);
#pragma unroll
        for (int e = 0; e < 4; ++e) {                      // registers 0, 1: tokens c2, c2 + 1; registers 2, 3: eight further on
          const int j = js * 16 + (e >> 1) * 8 + c2;
          const float w0 = j < L ? sm.pw[L - 1 - j] : 0.f, w1 = j + 1 < L ? sm.pw[L - 2 - j] : 0.f;
          split2((bf16lo(ah[e]) + bf16lo(al[e])) * w0, (bf16hi(ah[e]) + bf16hi(al[e])) * w1, ah[e], al[e]);
        }
#pragma unroll
        for (int np = 0; np < DVT / 16; ++np) {
          uint32_t b0, b1, b2, b3;
          ldsm_x4_t(b0, b1, b2, b3, sm.v[stage] + (js * 16 + trow) * VS + np * 16 + tcol);
          mma_bf16_16816(S[2 * np], ah, b0, b1);
          mma_bf16_16816(S[2 * np + 1], ah, b2, b3);
          mma_bf16_16816(S[2 * np], al, b0, b1);
          mma_bf16_16816(S[2 * np + 1], al, b2, b3);
        }
      }
    }
    __syncthreads();                                       // the second halves of O are in shared memory
    if (wc == 0) {
#pragma unroll
      for (int half8 = 0; half8 < 2; ++half8) {
        const int i = wr * 16 + g4 + 8 * half8;
        if (i >= L) continue;
        const float* ob = sm.ob + i * OS + c2;
        float* orow = og + static_cast<size_t>(t0 + i) * H * dv + c2;
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
          const float2 p = *reinterpret_cast<const float2*>(ob + nt * 8);
          *reinterpret_cast<float2*>(orow + nt * 8) = make_float2(o[nt][2 * half8] + p.x, o[nt][2 * half8 + 1] + p.y);
        }
      }
    }
  }
  cp_async_wait<0>();
  if (owner) {
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      *reinterpret_cast<float2*>(Sg + static_cast<size_t>(srow) * dv + nt * 8 + c2) = make_float2(S[nt][0], S[nt][1]);
      *reinterpret_cast<float2*>(Sg + static_cast<size_t>(srow + 8) * dv + nt * 8 + c2) = make_float2(S[nt][2], S[nt][3]);
    }
  }
}

template <int D, int DVT>
static cudaError_t launch_chunk(const RetArgs& a, int n_seqs, cudaStream_t st) {
  auto kern = retention_chunk_kernel<D, DVT>;
  const size_t smem = sizeof(ChunkSmem<D, DVT>);
  static bool opted = false;
  if (!opted) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return e;
    opted = true;
  }
  kern<<<dim3(a.dv / DVT, a.H, n_seqs), RC_THREADS, smem, st>>>(a);
  return cudaSuccess;
}

template <int D>
static cudaError_t launch_chunk_dv(const RetArgs& a, int n_seqs, cudaStream_t st) {
  return a.dv % 64 == 0 ? launch_chunk<D, 64>(a, n_seqs, st) : launch_chunk<D, 32>(a, n_seqs, st);
}

static bool chunk_shape(int d, int dv) { return (d == 32 || d == 64 || d == 96 || d == 128) && dv % 32 == 0; }

template <typename T>
static void launch_step(const RetArgs& a, int n_seqs, bool fused, cudaStream_t st) {
  const dim3 grid(a.H, n_seqs);
  if (fused) retention_step_kernel<T, true><<<grid, RS_THREADS, 0, st>>>(a);
  else retention_step_kernel<T, false><<<grid, RS_THREADS, 0, st>>>(a);
}

}  // namespace row
}  // namespace b2

using namespace b2;
using namespace b2::row;

extern "C" int b2tts_retention(const void* q, int64_t ldq, const void* k, int64_t ldk, const void* v, int64_t ldv, const float* rot,
                               int rot_dims, const float* decay, float k_scale, float* state, const void* gate, int64_t ldg, float* o,
                               float* qkv, void* out, const int32_t* seq_start, const int32_t* seq_pos0, const int32_t* seq_len,
                               const int32_t* seq_slot, int n_tokens, int n_seqs, int max_new, int heads, int dim, int vdim, float eps,
                               int dtype, int path, void* stream) {
  B2_REQUIRE(n_tokens >= 0 && n_seqs >= 0 && heads > 0 && dim > 0 && vdim > 0, B2TTS_EINVAL, "retention: bad sizes");
  B2_REQUIRE(heads <= 65535 && n_seqs <= 65535, B2TTS_EUNSUPPORTED, "retention: %d heads, %d sequences", heads, n_seqs);
  B2_REQUIRE(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= dim && (rot_dims == 0 || rot), B2TTS_EINVAL,
             "retention: %d rotated of %d coordinates", rot_dims, dim);
  B2_REQUIRE(B2_ROW_DTYPE_OK(dtype), B2TTS_EINVAL, "retention: dtype %d", dtype);
  B2_REQUIRE(path >= 0 && path <= 2, B2TTS_EINVAL, "retention: path %d", path);
  if (n_tokens == 0 || n_seqs == 0) return B2TTS_OK;
  B2_REQUIRE(q && k && v && decay && state && gate && out && seq_start && seq_pos0 && seq_len && seq_slot, B2TTS_EINVAL,
             "retention: null pointer");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool bf16 = dtype == B2TTS_DTYPE_BF16;
  const RetArgs a{q, ldq, k, ldk, v, ldv, rot, rot_dims, decay, k_scale, state, o, gate, ldg, out, seq_start, seq_pos0, seq_len, seq_slot,
                  heads, dim, vdim, eps};
  const bool step_ok = path != 1 && dim <= 256 && vdim <= 256 && vdim % 4 == 0 && aligned16(state);
  if (step_ok && max_new == 1) {                           // a step of single tokens: norm and gate ride in the launch
    if (bf16) launch_step<__nv_bfloat16>(a, n_seqs, true, st);
    else launch_step<float>(a, n_seqs, true, st);
    B2_CHECK_LAUNCH("retention (single tokens)");
    return B2TTS_OK;
  }
  const bool chunk_ok = bf16 && path != 1 && chunk_shape(dim, vdim) && rot_dims % 16 == 0 && ldq % 8 == 0 && ldk % 8 == 0 && ldv % 8 == 0 &&
                        aligned16(q) && aligned16(k) && aligned16(v) && aligned16(state) && aligned16(o) && (rot_dims == 0 || aligned16(rot));
  B2_REQUIRE(path != 2 || chunk_ok, B2TTS_EUNSUPPORTED, "retention: the tensor-core kernel takes bf16, key sizes 32 / 64 / 96 / 128, "
             "value sizes of whole 32s, 16-byte aligned rows and rotations of whole 16s");
  B2_REQUIRE(o && (chunk_ok || qkv), B2TTS_EINVAL, "retention: scratch missing");
  const bool chunk = chunk_ok && max_new > 1;
  if (chunk) {
    cudaError_t e;
    switch (dim) {
      case 32: e = launch_chunk_dv<32>(a, n_seqs, st); break;
      case 64: e = launch_chunk_dv<64>(a, n_seqs, st); break;
      case 96: e = launch_chunk_dv<96>(a, n_seqs, st); break;
      default: e = launch_chunk_dv<128>(a, n_seqs, st); break;
    }
    if (e != cudaSuccess) return cuda_fail(e, "retention (chunks)");
    B2_CHECK_LAUNCH("retention (chunks)");
  }
  if (step_ok) {
    if (bf16) launch_step<__nv_bfloat16>(a, n_seqs, false, st);
    else launch_step<float>(a, n_seqs, false, st);
    B2_CHECK_LAUNCH("retention (single tokens)");
  }
  if (!chunk || !step_ok) {
    B2_REQUIRE(qkv, B2TTS_EINVAL, "retention: scratch missing");
    if (bf16) retention_prep_kernel<__nv_bfloat16><<<n_tokens, 256, 0, st>>>(a, qkv);
    else retention_prep_kernel<float><<<n_tokens, 256, 0, st>>>(a, qkv);
    B2_CHECK_LAUNCH("retention (rotation)");
    const int hd = heads * dim;
    const int64_t ld = 2 * static_cast<int64_t>(hd) + static_cast<int64_t>(heads) * vdim;
    const int rc = b2tts_fixed_decay_scan(qkv, ld, qkv + hd, ld, qkv + 2 * hd, ld, decay, state, o, seq_start, seq_pos0, seq_len, seq_slot,
                                          n_tokens, n_seqs, heads, dim, vdim, chunk ? 2 : step_ok ? 1 : 0, stream);
    if (rc != B2TTS_OK) return rc;
  }
  return b2tts_gated_group_norm(o, gate, ldg, nullptr, 0, heads, 1, 0, eps, out, n_tokens, heads * vdim, dtype, stream);
}

extern "C" int b2tts_retention_scratch(int dim, int vdim, int max_new, int rot_dims, int aligned, int dtype, int path) {
  const bool step_ok = path != 1 && dim <= 256 && vdim <= 256 && vdim % 4 == 0;
  if (step_ok && max_new == 1) return 0;
  const bool chunk = dtype == B2TTS_DTYPE_BF16 && path != 1 && chunk_shape(dim, vdim) && rot_dims % 16 == 0 && aligned && max_new > 1;
  return chunk && step_ok ? 1 : 2;
}
