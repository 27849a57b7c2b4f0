// The real-gated linear recurrent unit: a diagonal recurrence whose decay and input are gated by block-diagonal
// products of its own input.  Per channel, in 32-bit, with u the causally filtered branch, S the channel's state and
// rate = 8 softplus(lam) (worked out when the weights are loaded):
//     r = sigmoid(Ra u + ra_b),  i = sigmoid(Ri u + ri_b)         (Ra, Ri block-diagonal: `blocks` square matrices)
//     a = exp(-rate r),   S <- a S + sqrt(1 - a^2) i u,   out = S gelu(y).
// y and the filter's raw input are columns of one fused projection.  The filter's last inputs live behind S in the
// request's state slot, 32-bit: [W | ring of taps x W], the input of the token at position p in place p % taps.  A token reads
// the taps - 1 inputs before its own and writes its own place, which none of those is: nothing moves, and blocks of one
// kernel may read and write in any order.  (Zeroed at admission, so places of positions before 0 read as zero: they are
// not written before the tokens that would read them have run.)  sqrt(1 - a^2) is taken as sqrt(-expm1(-2 rate r)), which keeps
// its digits where the decay is close to one.
//
//   ts_short_filter   u = bias + sum of taps, every channel, rounded to the engine's type; reads the slot's inputs for
//                     the tokens before the step's first, writes nothing to the slot
//   ts_rglru_gates    (a, sqrt(1 - a^2) i u) of every (token, channel), 32-bit pairs: both products of a 64 x 64 tile
//                     share the tile of u (tensor cores for bfloat16: u is bfloat16 already, so operands are exact and
//                     sums 32-bit; FFMA for the 32-bit type and for odd sizes), the gates in the epilogue
//   ts_rglru_scan     the recurrence: a block owns RS_CH channels of one request; RS_SEGS threads a channel take
//                     RS_TOK neighbouring tokens each, fold them into one (decay, sum) pair, pick up the state in front
//                     of them from the pairs before (shared memory), and run through their tokens once more for the
//                     output; then the filter's last inputs into their places
//   ts_rglru_step     all of it in one kernel for a step of single tokens (bfloat16): the filter in shared memory, the
//                     two products by m16n8k16 with the weights streamed from memory once, gates, state, output
#include "activations.cuh"
#include "common.cuh"
#include "mma_utils.cuh"

namespace {

constexpr int RG_MAX_TAPS = 8;

// (decay, addend) of one channel from the two pre-activations.  bfloat16 engine: the hardware's approximate exponential and
// reciprocal (relative errors of a few 2^-22, like the rounding of a 32-bit number; the exact functions cost
// the gates kernel more than its products do), and 1 - a^2 by the series of -expm1(t), t = 2 log a, where a is close to
// one (t > -1/2: seven terms, relative error below 2^-22), by the product 1 - a a elsewhere.
template <typename T> __device__ __forceinline__ float2 rg_pair(float zr, float zi, float rate, float u) {
  const float r = 1.f / (1.f + expf(-zr)), i = 1.f / (1.f + expf(-zi));
  const float la = -rate * r;
  return make_float2(expf(la), sqrtf(-expm1f(2.f * la)) * i * u);
}
template <> __device__ __forceinline__ float2 rg_pair<bf16>(float zr, float zi, float rate, float u) {
  const float r = __fdividef(1.f, 1.f + __expf(-zr)), i = __fdividef(1.f, 1.f + __expf(-zi));
  const float la = -rate * r, t = 2.f * la;
  const float a = __expf(la);
  float p = fmaf(t, 1.f / 5040.f, 1.f / 720.f);
  p = fmaf(t, p, 1.f / 120.f);
  p = fmaf(t, p, 1.f / 24.f);
  p = fmaf(t, p, 1.f / 6.f);
  p = fmaf(t, p, 0.5f);
  p = fmaf(t, p, 1.f);
  const float left = t > -0.5f ? -t * p : fmaf(-a, a, 1.f);
  return make_float2(a, __fsqrt_rn(left) * i * u);
}

// ---------------------------------------------------------------------------------------------------
// V neighbouring channels of a row
template <typename T, int V> struct RgVec;
template <typename T> struct RgVec<T, 1> {
  static __device__ __forceinline__ void load(const T* p, float* f) { f[0] = to_f(p[0]); }
  static __device__ __forceinline__ void store(T* p, const float* f) { p[0] = from_f<T>(f[0]); }
};
template <> struct RgVec<bf16, 4> {
  static __device__ __forceinline__ void load(const bf16* p, float* f) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  }
  static __device__ __forceinline__ void store(bf16* p, const float* f) {
    uint2 v;
    *reinterpret_cast<__nv_bfloat162*>(&v.x) = __floats2bfloat162_rn(f[0], f[1]);
    *reinterpret_cast<__nv_bfloat162*>(&v.y) = __floats2bfloat162_rn(f[2], f[3]);
    *reinterpret_cast<uint2*>(p) = v;
  }
};

// grid (ceil(T / TOK), ceil(W / (V blockDim))): a thread takes V neighbouring channels of TOK neighbouring tokens; the
// window of the filter slides through registers and is refilled (from the rows before, or the slot's memory) only at the
// thread's first token and where another request begins.  NT: the most taps the instance takes.
template <typename T, int TOK, int V, int NT>
__global__ void __launch_bounds__(128)
short_filter_kernel(T* __restrict__ out, int out_stride, const T* __restrict__ x, int x_stride, int x_off,
                    const float* __restrict__ conv_w, const float* __restrict__ conv_b, const float* __restrict__ state,
                    size_t state_stride, size_t ring_off, const int* __restrict__ token_request,
                    const int* __restrict__ q_start, const int* __restrict__ slots, const int* __restrict__ positions, int T_,
                    int W, int taps) {
  pdl_launch_dependents();
  pdl_wait();
  const int t_base = blockIdx.x * TOK;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (c >= W) return;
  const int count = min(TOK, T_ - t_base), keep = taps - 1;
  float v[TOK][V];
#pragma unroll
  for (int k = 0; k < TOK; ++k) {
    if (k < count) {
      RgVec<T, V>::load(x + (size_t)(t_base + k) * x_stride + x_off + c, v[k]);
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) v[k][e] = 0.f;
    }
  }
  float wgt[NT][V], bias[V];                    // wgt[d]: the tap d tokens back
#pragma unroll
  for (int e = 0; e < V; ++e) {
    bias[e] = conv_b != nullptr ? conv_b[c + e] : 0.f;
#pragma unroll
    for (int d = 0; d < NT; ++d) wgt[d][e] = d < taps ? conv_w[(size_t)(c + e) * taps + keep - d] : 0.f;
  }
  float win[NT][V];                             // win[d]: the input d + 1 tokens back
  int t_end = t_base;                                    // the end of the request the window belongs to
#pragma unroll
  for (int k = 0; k < TOK; ++k) {
    if (k < count) {
      const int t = t_base + k;
      if (t >= t_end) {
        const int b = token_request[t];
        const int t0 = q_start[b], i = t - t0;
        t_end = q_start[b + 1];
        const int pos = positions[t];
        const float* ring = state + (size_t)slots[b] * state_stride + ring_off;        // [taps][W]
#pragma unroll
        for (int d = 0; d < NT - 1; ++d)
          if (d < keep) {
            const int rel = i - 1 - d;                   // counted from the step's first token
            const int at = pos - 1 - d;                  // the input's position in the sequence
            if (rel >= 0) {
              RgVec<T, V>::load(x + (size_t)(t0 + rel) * x_stride + x_off + c, win[d]);
            } else {
#pragma unroll
              for (int e = 0; e < V; ++e) win[d][e] = at >= 0 ? ring[(size_t)(at % taps) * W + c + e] : 0.f;
            }
          }
      }
      float acc[V];
#pragma unroll
      for (int e = 0; e < V; ++e) {
        acc[e] = bias[e];
#pragma unroll
        for (int d = NT - 1; d > 0; --d)
          if (d < taps) acc[e] = fmaf(wgt[d][e], win[d - 1][e], acc[e]);
        acc[e] = fmaf(wgt[0][e], v[k][e], acc[e]);
#pragma unroll
        for (int d = NT - 2; d > 0; --d) win[d][e] = win[d - 1][e];
        win[0][e] = v[k][e];
      }
      RgVec<T, V>::store(out + (size_t)t * out_stride + c, acc);
    }
  }
}

// ---------------------------------------------------------------------------------------------------
// Both gate products of a tile of 64 tokens x 64 channels of one part, FFMA, any size and type.
constexpr int RF_M = 64, RF_N = 64, RF_K = 16, RF_PAD = 4;

template <typename T>
__global__ void __launch_bounds__(256)
rglru_gates_kernel(float2* __restrict__ ab, const T* __restrict__ u, const T* __restrict__ ra, const T* __restrict__ ri,
                   const float* __restrict__ ra_b, const float* __restrict__ ri_b, const float* __restrict__ rate, int M,
                   int W, int bs) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ __align__(16) float As[RF_K][RF_M + RF_PAD];
  __shared__ __align__(16) float Rs[RF_K][RF_N + RF_PAD];
  __shared__ __align__(16) float Is[RF_K][RF_N + RF_PAD];
  const int tid = threadIdx.x, part = blockIdx.y;
  const int n0 = blockIdx.x * RF_N, m0 = blockIdx.z * RF_M;
  const int lr = tid >> 2, lk = (tid & 3) * 4, ty = tid >> 4, tx = tid & 15;
  float r_acc[4][4] = {}, i_acc[4][4] = {};
  const T* a_row = m0 + lr < M ? u + (size_t)(m0 + lr) * W + (size_t)part * bs : nullptr;
  const bool n_ok = n0 + lr < bs;
  const T* r_row = ra + ((size_t)part * bs + (n_ok ? n0 + lr : 0)) * bs;
  const T* i_row = ri + ((size_t)part * bs + (n_ok ? n0 + lr : 0)) * bs;
  for (int k0 = 0; k0 < bs; k0 += RF_K) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int k = k0 + lk + i;
      As[lk + i][lr] = (a_row != nullptr && k < bs) ? to_f(a_row[k]) : 0.f;
      Rs[lk + i][lr] = (n_ok && k < bs) ? to_f(r_row[k]) : 0.f;
      Is[lk + i][lr] = (n_ok && k < bs) ? to_f(i_row[k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < RF_K; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&As[k][ty * 4]);
      const float4 r = *reinterpret_cast<const float4*>(&Rs[k][tx * 4]);
      const float4 g = *reinterpret_cast<const float4*>(&Is[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, rv[4] = {r.x, r.y, r.z, r.w}, gv[4] = {g.x, g.y, g.z, g.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          r_acc[i][j] = fmaf(av[i], rv[j], r_acc[i][j]);
          i_acc[i][j] = fmaf(av[i], gv[j], i_acc[i][j]);
        }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= bs) continue;
      const int c = part * bs + n;
      ab[(size_t)m * W + c] = rg_pair<T>(r_acc[i][j] + ra_b[c], i_acc[i][j] + ri_b[c], rate[c], to_f(u[(size_t)m * W + c]));
    }
  }
}

// The same on the tensor cores: bfloat16, parts a multiple of 8 wide on 16-byte boundaries.
constexpr int RM_M = 64, RM_N = 64, RM_K = 64, RM_STAGES = 3, RM_WARPS = 4;

__global__ void __launch_bounds__(RM_WARPS * 32)
rglru_gates_mma_kernel(float2* __restrict__ ab, const bf16* __restrict__ u, const bf16* __restrict__ ra,
                       const bf16* __restrict__ ri, const float* __restrict__ ra_b, const float* __restrict__ ri_b,
                       const float* __restrict__ rate, int M, int W, int bs) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(128) unsigned char rsm[];
  constexpr int TILE = RM_M * RM_K * 2;                  // bytes of one tile (all three are 64 x 64)
  unsigned char* u_s = rsm;
  unsigned char* r_s = u_s + RM_STAGES * TILE;
  unsigned char* i_s = r_s + RM_STAGES * TILE;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int part = blockIdx.y, n0 = blockIdx.x * RM_N, m0 = blockIdx.z * RM_M;
  const bf16* ub = u + (size_t)part * bs;
  const bf16* rb = ra + (size_t)part * bs * bs;
  const bf16* ib = ri + (size_t)part * bs * bs;
  const int k_tiles = (bs + RM_K - 1) / RM_K;
  auto load_tile = [&](int kt, int stage) {
    const int k0 = kt * RM_K;
#pragma unroll
    for (int idx = tid; idx < RM_M * 8; idx += RM_WARPS * 32) {
      const int r = idx >> 3, c = idx & 7, k = k0 + c * 8;
      const bool ok = m0 + r < M && k < bs;
      cp_async_16(u_s + stage * TILE + swz<RM_K>(r, c), ok ? ub + (size_t)(m0 + r) * W + k : u, ok);
      const bool w_ok = n0 + r < bs && k < bs;
      cp_async_16(r_s + stage * TILE + swz<RM_K>(r, c), w_ok ? rb + (size_t)(n0 + r) * bs + k : ra, w_ok);
      cp_async_16(i_s + stage * TILE + swz<RM_K>(r, c), w_ok ? ib + (size_t)(n0 + r) * bs + k : ri, w_ok);
    }
  };
  float r_acc[RM_N / 8][4], i_acc[RM_N / 8][4];
#pragma unroll
  for (int i = 0; i < RM_N / 8; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) r_acc[i][e] = i_acc[i][e] = 0.f;
#pragma unroll
  for (int s = 0; s < RM_STAGES - 1; ++s) {
    if (s < k_tiles) load_tile(s, s);
    cp_async_commit();
  }
  for (int kt = 0; kt < k_tiles; ++kt) {
    if (kt + RM_STAGES - 1 < k_tiles) load_tile(kt + RM_STAGES - 1, (kt + RM_STAGES - 1) % RM_STAGES);
    cp_async_commit();
    cp_async_wait<RM_STAGES - 1>();
    __syncthreads();
    const int st = (kt % RM_STAGES) * TILE;
#pragma unroll
    for (int ks = 0; ks < RM_K / 16; ++ks) {
      const int mat = lane >> 3, r = lane & 7;
      unsigned a[4];
      ldmatrix_x4(a[0], a[1], a[2], a[3], u_s + st + swz<RM_K>(warp * 16 + (mat & 1) * 8 + r, ks * 2 + (mat >> 1)));
#pragma unroll
      for (int np = 0; np < RM_N / 16; ++np) {
        const int at = swz<RM_K>(np * 16 + (mat >> 1) * 8 + r, ks * 2 + (mat & 1));
        unsigned b0, b1, b2, b3;
        ldmatrix_x4(b0, b1, b2, b3, r_s + st + at);
        mma_bf16(r_acc[2 * np], a, b0, b1);
        mma_bf16(r_acc[2 * np + 1], a, b2, b3);
        ldmatrix_x4(b0, b1, b2, b3, i_s + st + at);
        mma_bf16(i_acc[2 * np], a, b0, b1);
        mma_bf16(i_acc[2 * np + 1], a, b2, b3);
      }
    }
    __syncthreads();
  }
  cp_async_wait<0>();
#pragma unroll
  for (int nt = 0; nt < RM_N / 8; ++nt) {
    const int n = n0 + nt * 8 + (lane & 3) * 2;          // (parts are even, so both columns of a pair exist or neither)
    if (n >= bs) continue;
    const int c = part * bs + n;
    const float2 rbias = *reinterpret_cast<const float2*>(ra_b + c), ibias = *reinterpret_cast<const float2*>(ri_b + c);
    const float2 rt = *reinterpret_cast<const float2*>(rate + c);
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int m = m0 + warp * 16 + (lane >> 2) + 8 * h;
      if (m >= M) continue;
      const float2 uv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(u + (size_t)m * W + c));
      const float2 p0 = rg_pair<bf16>(r_acc[nt][2 * h] + rbias.x, i_acc[nt][2 * h] + ibias.x, rt.x, uv.x);
      const float2 p1 = rg_pair<bf16>(r_acc[nt][2 * h + 1] + rbias.y, i_acc[nt][2 * h + 1] + ibias.y, rt.y, uv.y);
      *reinterpret_cast<float4*>(ab + (size_t)m * W + c) = make_float4(p0.x, p0.y, p1.x, p1.y);
    }
  }
}

// ---------------------------------------------------------------------------------------------------
constexpr int RS_CH = 16, RS_SEGS = 32, RS_TOK = 8;

template <typename T>
__global__ void __launch_bounds__(RS_CH * RS_SEGS)
rglru_scan_kernel(T* __restrict__ out, const float2* __restrict__ ab, const T* __restrict__ proj, int proj_stride,
                  int y_off, int x_off, float* __restrict__ state, size_t state_stride, const int* __restrict__ q_start,
                  const int* __restrict__ slots, const int* __restrict__ positions, int W, int taps) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float2 agg[2][RS_SEGS][RS_CH];
  __shared__ float carry_s[2][RS_CH];
  const int b = blockIdx.y;
  const int t0 = q_start[b], n = q_start[b + 1] - t0;
  if (n <= 0) return;
  const int col = threadIdx.x % RS_CH, seg = threadIdx.x / RS_CH;
  const int c = blockIdx.x * RS_CH + col;
  const bool live = c < W;
  float* base = state + (size_t)slots[b] * state_stride;
  const bool one = n <= RS_TOK;                          // the first segment's thread runs through the request alone
  if (one && seg > 0) return;                            // (no barrier is reached then)
  if (seg == 0) carry_s[0][col] = live ? base[c] : 0.f;
  float2 v[RS_TOK];
  T y[RS_TOK];
  auto fetch = [&](int g0) {
    const int first = g0 + seg * RS_TOK;
#pragma unroll
    for (int k = 0; k < RS_TOK; ++k) {
      const bool ok = live && first + k < n;             // (a token that is not there leaves the state as it is)
      v[k] = ok ? __ldcs(ab + (size_t)(t0 + first + k) * W + c) : make_float2(1.f, 0.f);
      y[k] = ok ? proj[(size_t)(t0 + first + k) * proj_stride + y_off + c] : from_f<T>(0.f);
    }
  };
  fetch(0);
  int buf = 0;
  const int segs_last = one ? 0 : RS_SEGS - 1;           // (a segment without tokens passes the state on)
  for (int g0 = 0; g0 < n; g0 += RS_SEGS * RS_TOK, buf ^= 1) {
    float A = 1.f, B = 0.f;
#pragma unroll
    for (int k = 0; k < RS_TOK; ++k) {
      B = fmaf(v[k].x, B, v[k].y);
      A *= v[k].x;
    }
    float S;
    if (one) {
      S = carry_s[0][col];                               // (this thread's own)
    } else {
      agg[buf][seg][col] = make_float2(A, B);
      __syncthreads();
      S = carry_s[buf][col];
    }
#pragma unroll 4
    for (int s = 0; s < seg; ++s) {
      const float2 p = agg[buf][s][col];
      S = fmaf(p.x, S, p.y);
    }
    float o[RS_TOK];
#pragma unroll
    for (int k = 0; k < RS_TOK; ++k) {
      S = fmaf(v[k].x, S, v[k].y);
      o[k] = S * ts_activate_for<T>(to_f(y[k]), TS_ACT_GELU_TANH);
    }
    if (!one && seg == RS_SEGS - 1) carry_s[buf ^ 1][col] = S;
    const int first = g0 + seg * RS_TOK;
    if (g0 + RS_SEGS * RS_TOK < n) fetch(g0 + RS_SEGS * RS_TOK);
#pragma unroll
    for (int k = 0; k < RS_TOK; ++k)
      if (live && first + k < n) out[(size_t)(t0 + first + k) * W + c] = from_f<T>(o[k]);
    if (g0 + RS_SEGS * RS_TOK >= n && seg == segs_last && live) base[c] = S;
  }
  // the filter's last inputs into their places
  if (seg == 0 && live && taps > 1) {
    float* ring = base + W + c;
    const int pos0 = positions[t0];
    for (int i = max(0, n - (taps - 1)); i < n; ++i)
      ring[(size_t)((pos0 + i) % taps) * W] = to_f(proj[(size_t)(t0 + i) * proj_stride + x_off + c]);
  }
}

// ---------------------------------------------------------------------------------------------------
// A step of single tokens.  grid (channel groups of a part, parts, groups of RT_TOK tokens).  Everything that is weights is on
// its way before the wait for the predecessor, everything that is state or projection right after it.
constexpr int RT_TOK = 8, RT_WARPS = 8, RT_UNROLL = 4;

__global__ void __launch_bounds__(RT_WARPS * 32)
rglru_step_kernel(bf16* __restrict__ out, const bf16* __restrict__ proj, int proj_stride, int y_off, int x_off,
                  const float* __restrict__ conv_w, const float* __restrict__ conv_b, const bf16* __restrict__ ra,
                  const bf16* __restrict__ ri, const float* __restrict__ ra_b, const float* __restrict__ ri_b,
                  const float* __restrict__ rate, float* __restrict__ state, size_t state_stride,
                  const int* __restrict__ slots, const int* __restrict__ positions, int M, int W, int bs, int taps) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) unsigned char rtm[];
  bf16* u_s = reinterpret_cast<bf16*>(rtm);              // [RT_TOK][bs + 8]
  __shared__ int slot_s[RT_TOK], pos_s[RT_TOK];
  const int part = blockIdx.y, m0 = blockIdx.z * RT_TOK;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int g = lane >> 2, t = lane & 3;
  const int own0 = blockIdx.x * RT_WARPS * 8;            // this block's channels of the part
  const int n0 = own0 + warp * 8;                        // and this warp's
  const int us = bs + 8, keep = taps - 1;
  const bool n_ok = n0 + g < bs;
  const bf16* r_row = ra + ((size_t)part * bs + (n_ok ? n0 + g : 0)) * bs + t * 8;
  const bf16* i_row = ri + ((size_t)part * bs + (n_ok ? n0 + g : 0)) * bs + t * 8;
  uint4 rw[2][RT_UNROLL], iw[2][RT_UNROLL];
  auto fetch = [&](int k0, int buf) {
#pragma unroll
    for (int q = 0; q < RT_UNROLL; ++q) {
      const int k = k0 + q * 32;
      const bool ok = n_ok && k + t * 8 < bs;
      rw[buf][q] = ok ? *reinterpret_cast<const uint4*>(r_row + k) : make_uint4(0u, 0u, 0u, 0u);
      iw[buf][q] = ok ? *reinterpret_cast<const uint4*>(i_row + k) : make_uint4(0u, 0u, 0u, 0u);
    }
  };
  fetch(0, 0);
  fetch(32 * RT_UNROLL, 1);
  float rb[2] = {0.f, 0.f}, ib[2] = {0.f, 0.f}, rt[2] = {0.f, 0.f};
#pragma unroll
  for (int e = 0; e < 2; ++e)
    if (n0 + 2 * t + e < bs) {
      const int c = part * bs + n0 + 2 * t + e;
      rb[e] = ra_b[c];
      ib[e] = ri_b[c];
      rt[e] = rate[c];
    }
  // (slots and positions come from the host, before the step's first kernel)
  if (threadIdx.x < RT_TOK) {
    const bool there = m0 + (int)threadIdx.x < M;
    slot_s[threadIdx.x] = there ? slots[m0 + threadIdx.x] : -1;
    pos_s[threadIdx.x] = there ? positions[m0 + threadIdx.x] : 0;
  }
  __syncthreads();
  pdl_wait();
  // what the end of this thread's work wants: its state, and the gate branch
  float S_old[2] = {0.f, 0.f}, y_raw[2] = {0.f, 0.f};
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int n = n0 + 2 * t + e;
    if (m0 + g < M && n < bs) {
      S_old[e] = state[(size_t)slot_s[g] * state_stride + part * bs + n];
      y_raw[e] = to_f(proj[(size_t)(m0 + g) * proj_stride + y_off + part * bs + n]);
    }
  }
  // the filter: a thread a channel of all tokens, every load independent of the others
  for (int k = threadIdx.x; k < bs; k += RT_WARPS * 32) {
    const int c = part * bs + k;
    float acc[RT_TOK], x[RT_TOK];
    const float bias = conv_b != nullptr ? conv_b[c] : 0.f, w_now = conv_w[(size_t)c * taps + keep];
#pragma unroll
    for (int m = 0; m < RT_TOK; ++m) {
      x[m] = slot_s[m] >= 0 ? to_f(proj[(size_t)(m0 + m) * proj_stride + x_off + c]) : 0.f;
      acc[m] = bias;
    }
#pragma unroll
    for (int d = RG_MAX_TAPS - 1; d > 0; --d)            // d tokens back
      if (d < taps) {
        const float w = conv_w[(size_t)c * taps + keep - d];
        float v[RT_TOK];
#pragma unroll
        for (int m = 0; m < RT_TOK; ++m) {
          const int at = pos_s[m] - d;
          v[m] = slot_s[m] >= 0 && at >= 0 ? state[(size_t)slot_s[m] * state_stride + W + (size_t)(at % taps) * W + c] : 0.f;
        }
#pragma unroll
        for (int m = 0; m < RT_TOK; ++m) acc[m] = fmaf(w, v[m], acc[m]);
      }
    const bool own = taps > 1 && k >= own0 && k < own0 + RT_WARPS * 8;
#pragma unroll
    for (int m = 0; m < RT_TOK; ++m) {
      u_s[m * us + k] = from_f<bf16>(slot_s[m] >= 0 ? fmaf(w_now, x[m], acc[m]) : 0.f);
      // (its place in the ring: one that no token of this step reads)
      if (own && slot_s[m] >= 0) state[(size_t)slot_s[m] * state_stride + W + (size_t)(pos_s[m] % taps) * W + c] = x[m];
    }
  }
  __syncthreads();
  float zr[4] = {0.f, 0.f, 0.f, 0.f}, zi[4] = {0.f, 0.f, 0.f, 0.f};
  auto multiply = [&](int k0, int buf) {
#pragma unroll
    for (int q = 0; q < RT_UNROLL; ++q) {
      const int k = k0 + q * 32 + t * 8;
      const uint4 uv = k < bs ? *reinterpret_cast<const uint4*>(u_s + g * us + k) : make_uint4(0u, 0u, 0u, 0u);
      // rows 8 .. 15 of the product are zero; its k index is a permutation of the real one, the same for both operands
      const unsigned a1[4] = {uv.x, 0u, uv.y, 0u}, a2[4] = {uv.z, 0u, uv.w, 0u};
      mma_bf16(zr, a1, rw[buf][q].x, rw[buf][q].y);
      mma_bf16(zr, a2, rw[buf][q].z, rw[buf][q].w);
      mma_bf16(zi, a1, iw[buf][q].x, iw[buf][q].y);
      mma_bf16(zi, a2, iw[buf][q].z, iw[buf][q].w);
    }
  };
  constexpr int KSTEP = 32 * RT_UNROLL;
  for (int k0 = 0; k0 < bs; k0 += 2 * KSTEP) {
    multiply(k0, 0);
    if (k0 + 2 * KSTEP < bs) fetch(k0 + 2 * KSTEP, 0);
    if (k0 + KSTEP < bs) multiply(k0 + KSTEP, 1);
    if (k0 + 3 * KSTEP < bs) fetch(k0 + 3 * KSTEP, 1);
  }
  const int m = m0 + g;
  if (m >= M) return;
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int n = n0 + 2 * t + e;
    if (n >= bs) continue;
    const int c = part * bs + n;
    const float2 p = rg_pair<bf16>(zr[e] + rb[e], zi[e] + ib[e], rt[e], to_f(u_s[g * us + n]));
    const float s = fmaf(p.x, S_old[e], p.y);
    state[(size_t)slot_s[g] * state_stride + c] = s;
    out[(size_t)m * W + c] = from_f<bf16>(s * ts_activate_for<bf16>(y_raw[e], TS_ACT_GELU_TANH));
  }
}

}  // namespace

// out [T, out_stride] (W columns); x [T, x_stride], the filtered channels from column x_off; conv_w [W, taps] and conv_b
// [W] 32-bit (conv_b may be null); state [slots, state_stride] 32-bit, the ring of the filter's inputs from ring_off;
// positions [T]: the tokens' places in their sequences.
TS_API int ts_short_filter(void* out, int out_stride, const void* x, int x_stride, int x_off, const float* conv_w,
                           const float* conv_b, const float* state, long long state_stride, long long ring_off,
                           const int* token_request, const int* q_start, const int* slots, const int* positions, int T, int W,
                           int taps, int dtype, void* stream) {
  if (T <= 0 || W <= 0) return 0;
  if (taps < 1 || taps > RG_MAX_TAPS) TS_REFUSE(TS_ERR_LIMIT, "ts_short_filter: a filter of %d taps (1 to %d)", taps, RG_MAX_TAPS);
  cudaStream_t s = (cudaStream_t)stream;
  const bool few = T <= 64;
  // bfloat16 rows on 8-byte boundaries: four channels a thread
  const bool vec = dtype == TS_BF16 && !few && W % 4 == 0 && out_stride % 4 == 0 && x_stride % 4 == 0 && x_off % 4 == 0 &&
                   !(((uintptr_t)out | (uintptr_t)x) & 7);
  const dim3 grid(few ? T : ceil_div(T, 8), ceil_div(W, vec ? 512 : 128));
  if (grid.y > 65535) TS_REFUSE(TS_ERR_LIMIT, "ts_short_filter: %d channels", W);
#define TS_SFT(TT, N, V, NT)                                                                                                \
  ts_launch(short_filter_kernel<TT, N, V, NT>, grid, dim3(128), 0, s, (TT*)out, out_stride, (const TT*)x, x_stride, x_off, conv_w, \
            conv_b, state, (size_t)state_stride, (size_t)ring_off, token_request, q_start, slots, positions, T, W, taps)
#define TS_SF(TT, N, V)                                          \
  do {                                                            \
    if (taps <= 4) TS_SFT(TT, N, V, 4);                           \
    else TS_SFT(TT, N, V, RG_MAX_TAPS);                           \
  } while (0)
  if (dtype == TS_F32) { if (few) TS_SF(float, 1, 1); else TS_SF(float, 8, 1); }
  else if (dtype == TS_BF16) { if (few) TS_SF(bf16, 1, 1); else if (vec) TS_SF(bf16, 8, 4); else TS_SF(bf16, 8, 1); }
  else TS_REFUSE(TS_ERR_DTYPE, "ts_short_filter: dtype %d", dtype);
#undef TS_SF
#undef TS_SFT
  TS_LAUNCH_CHECK();
}

// ab [T, W] pairs of 32-bit floats; u [T, W]; ra, ri [blocks, bs, bs] in `dtype`; ra_b, ri_b, rate [W] 32-bit.
TS_API int ts_rglru_gates(float* ab, const void* u, const void* ra, const void* ri, const float* ra_b, const float* ri_b,
                          const float* rate, int T, int W, int blocks, int dtype, void* stream) {
  if (T <= 0) return 0;
  if (blocks < 1 || W % blocks) TS_REFUSE(TS_ERR_SHAPE, "ts_rglru_gates: %d channels in %d parts", W, blocks);
  const int bs = W / blocks;
  const dim3 grid(ceil_div(bs, RM_N), blocks, ceil_div(T, RM_M));
  if (blocks > 65535 || grid.z > 65535) TS_REFUSE(TS_ERR_LIMIT, "ts_rglru_gates: %d parts, %d tokens", blocks, T);
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == TS_BF16 && bs % 8 == 0 && !(((uintptr_t)u | (uintptr_t)ra | (uintptr_t)ri | (uintptr_t)ab) & 15) &&
      !(((uintptr_t)ra_b | (uintptr_t)ri_b | (uintptr_t)rate) & 7)) {
    const size_t smem = (size_t)3 * RM_STAGES * RM_M * RM_K * 2;
    static bool configured = false;
    if (!configured) {
      cudaError_t e = cudaFuncSetAttribute(rglru_gates_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) TS_REFUSE((int)e, "ts_rglru_gates: shared memory %zu: %s", smem, cudaGetErrorString(e));
      configured = true;
    }
    ts_launch(rglru_gates_mma_kernel, grid, dim3(RM_WARPS * 32), smem, s, (float2*)ab, (const bf16*)u, (const bf16*)ra,
              (const bf16*)ri, ra_b, ri_b, rate, T, W, bs);
    TS_LAUNCH_CHECK();
  }
  if (dtype == TS_F32)
    ts_launch(rglru_gates_kernel<float>, grid, dim3(256), 0, s, (float2*)ab, (const float*)u, (const float*)ra,
              (const float*)ri, ra_b, ri_b, rate, T, W, bs);
  else if (dtype == TS_BF16)
    ts_launch(rglru_gates_kernel<bf16>, grid, dim3(256), 0, s, (float2*)ab, (const bf16*)u, (const bf16*)ra,
              (const bf16*)ri, ra_b, ri_b, rate, T, W, bs);
  else
    TS_REFUSE(TS_ERR_DTYPE, "ts_rglru_gates: dtype %d", dtype);
  TS_LAUNCH_CHECK();
}

// out [T, W]; ab as ts_rglru_gates left it; proj [T, proj_stride]: the gate branch y from column y_off, the filter's raw
// input from x_off; state [slots, state_stride]: [W | ring of taps x W], read and left updated at each request's slot.
// longest: the most tokens a request brings (0: not known); long portions are launched late (see ts_launch_late).
constexpr int RS_LATE_TOKENS = 64;

TS_API int ts_rglru_scan(void* out, const float* ab, const void* proj, int proj_stride, int y_off, int x_off, float* state,
                         long long state_stride, const int* q_start, const int* slots, const int* positions, int B, int W,
                         int taps, int longest, int dtype, void* stream) {
  if (B <= 0) return 0;
  if (taps < 1 || taps > RG_MAX_TAPS) TS_REFUSE(TS_ERR_LIMIT, "ts_rglru_scan: a filter of %d taps (1 to %d)", taps, RG_MAX_TAPS);
  if (B > 65535) TS_REFUSE(TS_ERR_LIMIT, "ts_rglru_scan: %d requests per launch", B);
  cudaStream_t s = (cudaStream_t)stream;
  const dim3 grid(ceil_div(W, RS_CH), B), block(RS_CH * RS_SEGS);
#define TS_RS(TT)                                                                                                      \
  do {                                                                                                                 \
    if (longest >= RS_LATE_TOKENS)                                                                                     \
      ts_launch_late(rglru_scan_kernel<TT>, grid, block, 0, s, (TT*)out, (const float2*)ab, (const TT*)proj, proj_stride, y_off, \
                     x_off, state, (size_t)state_stride, q_start, slots, positions, W, taps);                                     \
    else                                                                                                               \
      ts_launch(rglru_scan_kernel<TT>, grid, block, 0, s, (TT*)out, (const float2*)ab, (const TT*)proj, proj_stride, y_off, \
                x_off, state, (size_t)state_stride, q_start, slots, positions, W, taps);                                          \
  } while (0)
  if (dtype == TS_F32) TS_RS(float);
  else if (dtype == TS_BF16) TS_RS(bf16);
  else TS_REFUSE(TS_ERR_DTYPE, "ts_rglru_scan: dtype %d", dtype);
#undef TS_RS
  TS_LAUNCH_CHECK();
}

TS_API int ts_rglru_step_supported(int W, int blocks, int taps, int dtype) {
  return dtype == TS_BF16 && blocks > 0 && blocks <= 65535 && W % blocks == 0 && (W / blocks) % 8 == 0 && W / blocks <= 2048 &&
         taps >= 1 && taps <= RG_MAX_TAPS;
}

// Every token of the step is a request of its own, token m that of slots[m] at positions[m].  Arguments as of the three kernels above.
TS_API int ts_rglru_step(void* out, const void* proj, int proj_stride, int y_off, int x_off, const float* conv_w,
                         const float* conv_b, const void* ra, const void* ri, const float* ra_b, const float* ri_b,
                         const float* rate, float* state, long long state_stride, const int* slots, const int* positions, int T,
                         int W, int blocks, int taps, int dtype, void* stream) {
  if (T <= 0) return 0;
  if (!ts_rglru_step_supported(W, blocks, taps, dtype) || (((uintptr_t)ra | (uintptr_t)ri) & 15))
    TS_REFUSE(TS_ERR_UNSUPPORTED, "ts_rglru_step: %d channels in %d parts, %d taps", W, blocks, taps);
  const int bs = W / blocks;
  const dim3 grid(ceil_div(bs, 8 * RT_WARPS), blocks, ceil_div(T, RT_TOK));
  if (grid.z > 65535) TS_REFUSE(TS_ERR_LIMIT, "ts_rglru_step: %d tokens", T);
  const size_t smem = (size_t)RT_TOK * (bs + 8) * 2;     // (at most 33 KB)
  ts_launch(rglru_step_kernel, grid, dim3(RT_WARPS * 32), smem, (cudaStream_t)stream, (bf16*)out, (const bf16*)proj, proj_stride,
            y_off, x_off, conv_w, conv_b, (const bf16*)ra, (const bf16*)ri, ra_b, ri_b, rate, state, (size_t)state_stride, slots,
            positions, T, W, bs, taps);
  TS_LAUNCH_CHECK();
}
