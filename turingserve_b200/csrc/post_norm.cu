// The norm of layers that norm what a sublayer RETURNS (not what it reads) over a residual stream in 32-bit:
//     n = y / sqrt(mean(y^2) + eps) * w,    stream <- stream + n,    out = T(stream),
// or, where a norm reads the new stream next (the model's last one), out = T(stream / sqrt(mean(stream^2) + eps) * w2).
// All in 32-bit, out rounded once.  The stream starts from the embedding rows (`base`) at a model's first such norm.
// y is one of
//     * a tensor in the engine's type,
//     * a product left unreduced by its kernel: [splits, T, hidden] 32-bit partial sums (+ bias), summed in split order,
//     * what a routed feed-forward leaves before its sum: scale * sum over a token's choices r (ascending) of
//       (pair_w[t, r] *) rows[place[t top + r], :], 32-bit rows, plus one of the two forms above (a shared expert).
// One block a token.
#include "common.cuh"

namespace {

struct PostNorm {
  const float* part;           // partial sums, or null
  size_t split_stride;
  const float* rows;           // the routed feed-forward's rows, or null
  const int* place;
  const float* pair_w;         // or null
  const float* w;              // [hidden]
  const float* w2;             // [hidden] of the norm that reads the stream next, or null
  int splits, top, hidden;
  float scale, eps, eps2;
};

template <typename T, int N>
__device__ __forceinline__ void pn_load(const T* p, float* f) {
#pragma unroll
  for (int k = 0; k < N; ++k) f[k] = to_f(p[k]);
}
template <> __device__ __forceinline__ void pn_load<bf16, 4>(const bf16* p, float* f) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
}
template <> __device__ __forceinline__ void pn_load<float, 4>(const float* p, float* f) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
}
template <typename T> __device__ __forceinline__ void pn_store4(T* p, const float* f);
template <> __device__ __forceinline__ void pn_store4<bf16>(bf16* p, const float* f) {
  uint2 v;
  *reinterpret_cast<__nv_bfloat162*>(&v.x) = __floats2bfloat162_rn(f[0], f[1]);
  *reinterpret_cast<__nv_bfloat162*>(&v.y) = __floats2bfloat162_rn(f[2], f[3]);
  *reinterpret_cast<uint2*>(p) = v;
}
template <> __device__ __forceinline__ void pn_store4<float>(float* p, const float* f) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
}

// y of the N columns from i on
template <typename T, int N>
__device__ __forceinline__ void pn_gather(const PostNorm& a, const T* y, const T* bias, size_t t, int i, float* v) {
#pragma unroll
  for (int k = 0; k < N; ++k) v[k] = 0.f;
  if (a.rows != nullptr) {
    for (int r = 0; r < a.top; ++r) {
      const size_t p = t * a.top + r;
      const float s = a.pair_w != nullptr ? a.pair_w[p] : 1.f;
      float x[N];
      pn_load<float, N>(a.rows + (size_t)a.place[p] * a.hidden + i, x);
#pragma unroll
      for (int k = 0; k < N; ++k) v[k] = fmaf(s, x[k], v[k]);
    }
#pragma unroll
    for (int k = 0; k < N; ++k) v[k] *= a.scale;
  }
  if (a.part != nullptr) {
    float s[N];
#pragma unroll
    for (int k = 0; k < N; ++k) s[k] = 0.f;
    for (int sp = 0; sp < a.splits; ++sp) {
      float x[N];
      pn_load<float, N>(a.part + (size_t)sp * a.split_stride + t * a.hidden + i, x);
#pragma unroll
      for (int k = 0; k < N; ++k) s[k] += x[k];
    }
#pragma unroll
    for (int k = 0; k < N; ++k) v[k] += bias != nullptr ? s[k] + to_f(bias[i + k]) : s[k];
  } else if (y != nullptr) {
    float x[N];
    pn_load<T, N>(y + t * a.hidden + i, x);
#pragma unroll
    for (int k = 0; k < N; ++k) v[k] += x[k];
  }
}

// any row length; the row in shared memory
template <typename T>
__global__ void __launch_bounds__(256)
post_norm_kernel(T* __restrict__ out, float* __restrict__ stream, const T* __restrict__ base, const T* __restrict__ y,
                 const T* __restrict__ bias, PostNorm a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float pn_s[];
  __shared__ float scratch[32];
  const size_t t = blockIdx.x, at = t * a.hidden;
  float ss = 0.f;
  for (int i = threadIdx.x; i < a.hidden; i += blockDim.x) {
    float v;
    pn_gather<T, 1>(a, y, bias, t, i, &v);
    pn_s[i] = v;
    ss = fmaf(v, v, ss);
  }
  ss = block_sum(ss, scratch);
  const float rstd = 1.f / sqrtf(ss / (float)a.hidden + a.eps);
  float s2 = 0.f;
  for (int i = threadIdx.x; i < a.hidden; i += blockDim.x) {           // (a thread reads back what it wrote itself)
    const float v = (base != nullptr ? to_f(base[at + i]) : stream[at + i]) + pn_s[i] * rstd * a.w[i];
    stream[at + i] = v;
    pn_s[i] = v;
    s2 = fmaf(v, v, s2);
  }
  if (out == nullptr) return;
  float r2 = 1.f;
  if (a.w2 != nullptr) r2 = 1.f / sqrtf(block_sum(s2, scratch) / (float)a.hidden + a.eps2);
  for (int i = threadIdx.x; i < a.hidden; i += blockDim.x)
    out[at + i] = from_f<T>(a.w2 != nullptr ? pn_s[i] * r2 * a.w2[i] : pn_s[i]);
}

// Rows a multiple of 4 long and at most 4 CH blockDim on 16-byte boundaries: the row stays in registers, 16 bytes a load
// (8 of bfloat16), the stream's own row is on its way before the sum is known.
template <typename T, int CH>
__global__ void __launch_bounds__(256)
post_norm_vec_kernel(T* __restrict__ out, float* __restrict__ stream, const T* __restrict__ base, const T* __restrict__ y,
                     const T* __restrict__ bias, PostNorm a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float scratch[32];
  const size_t t = blockIdx.x, at = t * a.hidden;
  float v[CH][4], x[CH][4];
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = (c * blockDim.x + threadIdx.x) * 4;
    if (i < a.hidden) {
      if (base != nullptr) pn_load<T, 4>(base + at + i, x[c]);
      else pn_load<float, 4>(stream + at + i, x[c]);
      pn_gather<T, 4>(a, y, bias, t, i, v[c]);
#pragma unroll
      for (int k = 0; k < 4; ++k) ss = fmaf(v[c][k], v[c][k], ss);
    }
  }
  ss = block_sum(ss, scratch);
  const float rstd = 1.f / sqrtf(ss / (float)a.hidden + a.eps);
  float s2 = 0.f;
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = (c * blockDim.x + threadIdx.x) * 4;
    if (i < a.hidden) {
      float w[4];
      pn_load<float, 4>(a.w + i, w);
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        v[c][k] = x[c][k] + v[c][k] * rstd * w[k];
        s2 = fmaf(v[c][k], v[c][k], s2);
      }
      pn_store4<float>(stream + at + i, v[c]);
      if (out != nullptr && a.w2 == nullptr) pn_store4<T>(out + at + i, v[c]);
    }
  }
  if (out == nullptr || a.w2 == nullptr) return;
  const float r2 = 1.f / sqrtf(block_sum(s2, scratch) / (float)a.hidden + a.eps2);
#pragma unroll
  for (int c = 0; c < CH; ++c) {
    const int i = (c * blockDim.x + threadIdx.x) * 4;
    if (i < a.hidden) {
      float w[4];
      pn_load<float, 4>(a.w2 + i, w);
#pragma unroll
      for (int k = 0; k < 4; ++k) w[k] *= v[c][k] * r2;
      pn_store4<T>(out + at + i, w);
    }
  }
}

}  // namespace

// out [T, hidden] (may be null) in `dtype`; stream [T, hidden] 32-bit; base [T, hidden] in `dtype`: the stream starts from
// it (null: the stream is added to).  y [T, hidden], or part [splits, T, hidden] (+ bias [hidden]); rows [., hidden] with
// place [T, top] and pair_w [T, top] or null; w [hidden]; w2 [hidden] or null.
TS_API int ts_post_norm(void* out, float* stream, const void* base, const void* y, const float* part, int splits,
                        const void* bias, const float* rows, const int* place, const float* pair_w, int top, float scale,
                        const float* w, float eps, const float* w2, float eps2, int T, int hidden, int dtype, void* stream_) {
  if (T <= 0) return 0;
  if (y == nullptr && part == nullptr && rows == nullptr) TS_REFUSE(TS_ERR_SHAPE, "ts_post_norm: nothing to norm");
  if (rows != nullptr && (place == nullptr || top < 1)) TS_REFUSE(TS_ERR_SHAPE, "ts_post_norm: rows without their places");
  if (hidden <= 0 || hidden > 48 * 1024) TS_REFUSE(TS_ERR_LIMIT, "ts_post_norm: rows of %d", hidden);
  PostNorm a;
  a.part = part; a.split_stride = (size_t)T * hidden; a.splits = splits; a.rows = rows; a.place = place; a.pair_w = pair_w;
  a.top = top; a.scale = scale; a.w = w; a.w2 = w2; a.eps = eps; a.eps2 = eps2; a.hidden = hidden;
  cudaStream_t s = (cudaStream_t)stream_;
  const uintptr_t ptrs = (uintptr_t)out | (uintptr_t)stream | (uintptr_t)base | (uintptr_t)y | (uintptr_t)part | (uintptr_t)rows |
                         (uintptr_t)w | (uintptr_t)w2;
  const bool vec = hidden % 4 == 0 && hidden <= 4 * 4 * 256 && !(ptrs & 15);
  const int ch = hidden <= 1024 ? 1 : (hidden <= 2048 ? 2 : 4);
  const dim3 vblock((((hidden / 4 + ch - 1) / ch) + 31) / 32 * 32), block(hidden >= 512 ? 256 : 128);
  const size_t smem = sizeof(float) * hidden;
#define TS_PN(TT)                                                                                                      \
  do {                                                                                                                 \
    if (vec && ch == 1) ts_launch(post_norm_vec_kernel<TT, 1>, dim3(T), vblock, 0, s, (TT*)out, stream, (const TT*)base, (const TT*)y, (const TT*)bias, a); \
    else if (vec && ch == 2) ts_launch(post_norm_vec_kernel<TT, 2>, dim3(T), vblock, 0, s, (TT*)out, stream, (const TT*)base, (const TT*)y, (const TT*)bias, a); \
    else if (vec) ts_launch(post_norm_vec_kernel<TT, 4>, dim3(T), vblock, 0, s, (TT*)out, stream, (const TT*)base, (const TT*)y, (const TT*)bias, a); \
    else {                                                                                                             \
      if (smem > 48 * 1024) {                                                                                          \
        cudaError_t e = cudaFuncSetAttribute(post_norm_kernel<TT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        if (e != cudaSuccess) TS_REFUSE((int)e, "ts_post_norm: shared memory %zu: %s", smem, cudaGetErrorString(e));   \
      }                                                                                                                \
      ts_launch(post_norm_kernel<TT>, dim3(T), block, smem, s, (TT*)out, stream, (const TT*)base, (const TT*)y, (const TT*)bias, a); \
    }                                                                                                                  \
  } while (0)
  if (dtype == TS_F32) TS_PN(float);
  else if (dtype == TS_BF16) TS_PN(bf16);
  else TS_REFUSE(TS_ERR_DTYPE, "ts_post_norm: dtype %d", dtype);
#undef TS_PN
  TS_LAUNCH_CHECK();
}
