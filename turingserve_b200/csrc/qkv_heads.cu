// Between a fused q/k/v projection and an attention that norms, rotates and caches what it reads; 32-bit arithmetic, one
// rounding:
//   q and k heads  x <- x / sqrt(mean(x^2) + eps) * w  (one learned weight for all q heads, one for all k heads), then
//                  dimension i turned with dimension i + R/2, i < R/2, by position * freq[i], cosine and sine times a
//                  magnitude; the dimensions from R on pass
//   value heads    divided by their own root mean square (no weight), then all V dimensions turned in pairs (m, m + V/2)
//                  by position * v_freq[m]: an attention over such values returns sums turned by the keys' positions,
//                  which the attention kernels turn back by the query's
// Every one of these is optional.  q goes back where it came from, k and v go to their cache pages.  The projection may be
// the partial sums of a product cut along K (summed here in split order and rounded as the product's own last pass would
// have); columns behind the values (gates) are then finished too.
#include "common.cuh"

namespace {

constexpr int QH_WARPS = 4;

struct QkvHeads {
  int H, G, D, V, page, k_off, v_off;
  const float* q_w;            // [D], null: no norm of q and k
  const float* k_w;
  const float* freq;           // [rot / 2]
  const float* v_freq;         // [V / 2], null: values are not turned
  int rot, v_norm;
  float eps, magnitude;
};

// One warp a (token, head), the head's values in shared memory: any size and type.
template <typename T>
__global__ void __launch_bounds__(QH_WARPS * 32)
qkv_heads_kernel(T* __restrict__ proj, int stride, const int* __restrict__ positions, T* __restrict__ k_cache,
                 T* __restrict__ v_cache, const int* __restrict__ slots, QkvHeads a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float qh_s[];
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int head = blockIdx.y * QH_WARPS + warp;
  if (head >= a.H + 2 * a.G) return;
  const bool is_q = head < a.H, is_v = head >= a.H + a.G;
  const int g = is_v ? head - a.H - a.G : head - a.H;
  const int slot = slots != nullptr ? slots[t] : -1;
  if (!is_q && slot < 0) return;
  const int n = is_v ? a.V : a.D;
  float* x = qh_s + warp * max(a.D, a.V);
  T* src = proj + (size_t)t * stride + (is_q ? (size_t)head * a.D : (is_v ? a.v_off + (size_t)g * a.V : a.k_off + (size_t)g * a.D));
  float ss = 0.f;
  for (int i = lane; i < n; i += 32) {
    const float v = to_f(src[i]);
    x[i] = v;
    ss = fmaf(v, v, ss);
  }
  ss = warp_sum(ss);
  const float* w = is_q ? a.q_w : (is_v ? nullptr : a.k_w);
  const bool norm = is_v ? a.v_norm != 0 : w != nullptr;
  const float r = norm ? 1.f / sqrtf(ss / (float)n + a.eps) : 1.f;
  __syncwarp();
  for (int i = lane; i < n; i += 32) x[i] = w != nullptr ? x[i] * r * w[i] : x[i] * r;
  __syncwarp();
  T* dst = src;
  if (!is_q) {
    const size_t pg = slot / a.page, off = slot % a.page;
    dst = (is_v ? v_cache : k_cache) + ((pg * a.G + g) * a.page + off) * n;
  }
  const float* f = is_v ? a.v_freq : a.freq;
  const int half = is_v ? (f != nullptr ? a.V / 2 : 0) : a.rot / 2;
  const float mag = is_v ? 1.f : a.magnitude, pos = (float)positions[t];
  for (int i = lane; i < half; i += 32) {
    float sn, cs;
    sincosf(pos * f[i], &sn, &cs);
    sn *= mag;
    cs *= mag;
    const float u = x[i], v = x[i + half];
    dst[i] = from_f<T>(u * cs - v * sn);
    dst[i + half] = from_f<T>(v * cs + u * sn);
  }
  for (int i = 2 * half + lane; i < n; i += 32) dst[i] = from_f<T>(x[i]);
}

__device__ __forceinline__ void qh_unpack(const uint4& v, float* f) {
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&v);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 t = __bfloat1622float2(h[j]);
    f[2 * j] = t.x;
    f[2 * j + 1] = t.y;
  }
}

// bfloat16 heads of up to 8 L columns, everything in multiples of 8 on 16-byte boundaries: a lane holds 8 neighbouring
// columns in registers, partner columns come by shuffles, the block works the token's cosines and sines out once.
// L lanes a head (16: a warp takes two heads).
template <int L>
__global__ void __launch_bounds__(QH_WARPS * 32)
qkv_heads_vec_kernel(bf16* __restrict__ proj, int stride, const int* __restrict__ positions, bf16* __restrict__ k_cache,
                     bf16* __restrict__ v_cache, const int* __restrict__ slots, const float* __restrict__ part, int splits,
                     int extra_off, int extra_n, QkvHeads a) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float qh_s[];          // cosines of the keys, their sines, cosines and sines of the values
  constexpr int PER = 32 / L;
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int sub = lane % L, which = lane / L;
  const int head = (blockIdx.y * QH_WARPS + warp) * PER + which;
  const bool is_q = head < a.H, is_v = head >= a.H + a.G;
  const int g = is_v ? head - a.H - a.G : head - a.H;
  const int n = is_v ? a.V : a.D, c = sub * 8;
  const bool holds = head < a.H + 2 * a.G && c < n;
  // (positions and slots come from the host, before the step's first kernel)
  const int slot = slots != nullptr ? slots[t] : -1;
  const float pos = (float)positions[t];
  const int kh = a.rot / 2, vh = a.v_freq != nullptr ? a.V / 2 : 0;
  float* kc = qh_s;
  float* ks = kc + kh;
  float* vc = ks + kh;
  float* vs = vc + vh;
  for (int i = threadIdx.x; i < kh + vh; i += QH_WARPS * 32) {
    float sn, cs;
    if (i < kh) {
      sincosf(pos * a.freq[i], &sn, &cs);
      kc[i] = cs * a.magnitude;
      ks[i] = sn * a.magnitude;
    } else {
      sincosf(pos * a.v_freq[i - kh], &sn, &cs);
      vc[i - kh] = cs;
      vs[i - kh] = sn;
    }
  }
  pdl_wait();
  bf16* row = proj + (size_t)t * stride;
  const size_t split_stride = (size_t)gridDim.x * stride;
  const float* prow = part != nullptr ? part + (size_t)t * stride : nullptr;
  const int col0 = !holds ? 0 : (is_q ? head * a.D : (is_v ? a.v_off + g * a.V : a.k_off + g * a.D));
  bf16* src = row + col0 + (holds ? c : 0);
  float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
  if (holds) {
    if (prow == nullptr) {
      qh_unpack(*reinterpret_cast<const uint4*>(src), f);
    } else {
      for (int sp = 0; sp < splits; ++sp) {
        const float4* p4 = reinterpret_cast<const float4*>(prow + sp * split_stride + col0 + c);
        const float4 x = p4[0], y = p4[1];
        f[0] += x.x; f[1] += x.y; f[2] += x.z; f[3] += x.w;
        f[4] += y.x; f[5] += y.y; f[6] += y.z; f[7] += y.w;
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = round_to<bf16>(f[j]);
    }
  }
  if (prow != nullptr && blockIdx.y == 0)
    for (int i = threadIdx.x; i < extra_n; i += QH_WARPS * 32) {
      float v = 0.f;
      for (int sp = 0; sp < splits; ++sp) v += prow[sp * split_stride + extra_off + i];
      row[extra_off + i] = from_f<bf16>(v);
    }
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < 8; ++j) ss = fmaf(f[j], f[j], ss);
#pragma unroll
  for (int o = L / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);         // (stays within the head's lanes)
  const float* w = is_q ? a.q_w : (is_v ? nullptr : a.k_w);
  const bool norm = is_v ? a.v_norm != 0 : w != nullptr;
  if (norm) {
    const float r = 1.f / sqrtf(ss / (float)n + a.eps);
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] *= r;
    if (w != nullptr && holds) {
      const float4 w0 = *reinterpret_cast<const float4*>(w + c), w1 = *reinterpret_cast<const float4*>(w + c + 4);
      f[0] *= w0.x; f[1] *= w0.y; f[2] *= w0.z; f[3] *= w0.w;
      f[4] *= w1.x; f[5] *= w1.y; f[6] *= w1.z; f[7] *= w1.w;
    }
  }
  __syncthreads();
  const int hl = (is_v ? vh : kh) / 8;                   // lanes that hold the first columns of the pairs
  const int partner = which * L + (sub < hl ? sub + hl : (sub < 2 * hl ? sub - hl : sub));
  float p[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) p[j] = __shfl_sync(0xffffffffu, f[j], partner);
  if (sub < 2 * hl) {
    const bool low = sub < hl;
    const int i0 = (low ? sub : sub - hl) * 8;
    const float* cp = (is_v ? vc : kc) + i0;
    const float* sp = (is_v ? vs : ks) + i0;
    const float4 c0 = *reinterpret_cast<const float4*>(cp), c1 = *reinterpret_cast<const float4*>(cp + 4);
    const float4 s0 = *reinterpret_cast<const float4*>(sp), s1 = *reinterpret_cast<const float4*>(sp + 4);
    const float cv[8] = {c0.x, c0.y, c0.z, c0.w, c1.x, c1.y, c1.z, c1.w};
    const float sv[8] = {s0.x, s0.y, s0.z, s0.w, s1.x, s1.y, s1.z, s1.w};
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] = low ? f[j] * cv[j] - p[j] * sv[j] : f[j] * cv[j] + p[j] * sv[j];
  }
  if (!holds || (!is_q && slot < 0)) return;
  bf16* dst = src;
  if (!is_q) {
    const size_t pg = slot / a.page, off = slot % a.page;
    dst = (is_v ? v_cache : k_cache) + ((pg * a.G + g) * a.page + off) * n + c;
  }
  uint4 o;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
  for (int j = 0; j < 4; ++j) h[j] = __floats2bfloat162_rn(f[2 * j], f[2 * j + 1]);
  *reinterpret_cast<uint4*>(dst) = o;
}

bool vec_takes(int stride, int k_off, int v_off, int D, int V, int rot, int v_turned, int dtype) {
  return dtype == TS_BF16 && D % 8 == 0 && V % 8 == 0 && D <= 256 && V <= 256 && stride % 8 == 0 && k_off % 8 == 0 &&
         v_off % 8 == 0 && rot % 16 == 0 && (!v_turned || V % 16 == 0);
}

}  // namespace

// Whether the projection may come as partial sums (the pointers then on 16-byte boundaries).
TS_API int ts_qkv_heads_supports_parts(int stride, int k_off, int v_off, int D, int V, int rot, int v_turned, int dtype) {
  return vec_takes(stride, k_off, v_off, D, V, rot, v_turned, dtype);
}

// proj [T, stride]: q heads in the columns [0, H D), k heads from k_off (G D), value rows from v_off (G V).  q_w, k_w [D]
// 32-bit or both null; freq [rot_dims / 2]; v_freq [V / 2] or null; k_cache [pages, G, page, D], v_cache [pages, G, page,
// V]; slots null or -1: nothing is cached.  part: [splits, T, stride] 32-bit or null; of `proj` then only q and the columns
// [extra_off, extra_off + extra_n) are written.
TS_API int ts_qkv_heads_write(void* proj, int stride, int k_off, int v_off, const int* positions, const float* q_w,
                              const float* k_w, float eps, const float* freq, float magnitude, int rot_dims, int v_norm,
                              const float* v_freq, void* k_cache, void* v_cache, const int* slots, int T, int H, int G, int D,
                              int V, int page, int dtype, const float* part, int splits, int extra_off, int extra_n,
                              void* stream) {
  if (T <= 0) return 0;
  if (H <= 0 || G <= 0 || D <= 0 || V <= 0 || D > 2048 || V > 2048) TS_REFUSE(TS_ERR_LIMIT, "ts_qkv_heads_write: %d / %d heads of %d / %d", H, G, D, V);
  if (rot_dims < 0 || rot_dims % 2 || rot_dims > D) TS_REFUSE(TS_ERR_SHAPE, "ts_qkv_heads_write: %d rotated dimensions of %d", rot_dims, D);
  if (rot_dims > 0 && freq == nullptr) TS_REFUSE(TS_ERR_SHAPE, "ts_qkv_heads_write: a rotation without frequencies");
  if (v_freq != nullptr && V % 2) TS_REFUSE(TS_ERR_SHAPE, "ts_qkv_heads_write: %d value dimensions do not pair", V);
  if ((q_w == nullptr) != (k_w == nullptr)) TS_REFUSE(TS_ERR_SHAPE, "ts_qkv_heads_write: q and k are normed together");
  const int heads = H + 2 * G;
  if (heads > 65535) TS_REFUSE(TS_ERR_LIMIT, "ts_qkv_heads_write: %d heads", heads);
  QkvHeads a;
  a.H = H; a.G = G; a.D = D; a.V = V; a.page = page; a.k_off = k_off; a.v_off = v_off;
  a.q_w = q_w; a.k_w = k_w; a.freq = freq; a.v_freq = v_freq; a.rot = rot_dims; a.v_norm = v_norm;
  a.eps = eps; a.magnitude = magnitude;
  cudaStream_t s = (cudaStream_t)stream;
  const uintptr_t ptrs = (uintptr_t)proj | (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)q_w | (uintptr_t)k_w | (uintptr_t)part;
  if (vec_takes(stride, k_off, v_off, D, V, rot_dims, v_freq != nullptr, dtype) && !(ptrs & 15)) {
    const int wide = D > V ? D : V, per = wide <= 128 ? 2 : 1;
    const size_t smem = sizeof(float) * (rot_dims + (v_freq != nullptr ? V : 0) + 8);
    auto kernel = per == 2 ? qkv_heads_vec_kernel<16> : qkv_heads_vec_kernel<32>;
    ts_launch(kernel, dim3(T, ceil_div(heads, QH_WARPS * per)), dim3(QH_WARPS * 32), smem, s, (bf16*)proj, stride, positions,
              (bf16*)k_cache, (bf16*)v_cache, slots, part, splits, extra_off, extra_n, a);
    TS_LAUNCH_CHECK();
  }
  if (part != nullptr) TS_REFUSE(TS_ERR_ALIGN, "ts_qkv_heads_write: partial sums need bfloat16 heads of multiples of 8 on 16-byte boundaries");
  const size_t smem = sizeof(float) * QH_WARPS * (D > V ? D : V);      // (at most 32 KB)
  const dim3 grid(T, ceil_div(heads, QH_WARPS));
  if (dtype == TS_F32)
    ts_launch(qkv_heads_kernel<float>, grid, dim3(QH_WARPS * 32), smem, s, (float*)proj, stride, positions, (float*)k_cache,
              (float*)v_cache, slots, a);
  else if (dtype == TS_BF16)
    ts_launch(qkv_heads_kernel<bf16>, grid, dim3(QH_WARPS * 32), smem, s, (bf16*)proj, stride, positions, (bf16*)k_cache,
              (bf16*)v_cache, slots, a);
  else
    TS_REFUSE(TS_ERR_DTYPE, "ts_qkv_heads_write: dtype %d", dtype);
  TS_LAUNCH_CHECK();
}
