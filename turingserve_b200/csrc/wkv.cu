// A time mixer whose matrix state fades channel by channel at rates the token chooses (the sixth generation of RWKV; Peng et
// al., "Eagle and Finch: RWKV with Matrix-Valued States and Dynamic Recurrence").  For every request and head a state S [D, V]
// in 32-bit lives in a state slot between steps; per token, with r, k, v and a decay w in (0, 1) per key channel,
//     o = (S + diag(u) k v^T)^T r,        S <- diag(w) S + k v^T          (the bonus u counts for the present token only).
// r, k, v, the gate and the decay each read a mix of the token's input h and the one before it, h + (h' - h) mu; the decay is
// w = exp(-exp(w2 tanh(w1 mix) + w0)).  The slot holds [H D V values of S | the last input h], all 32-bit.
//
//   ts_token_shift    the mixes of every token, [n, T, hidden]; the row before a request's first token comes from the slot
//   ts_wkv_decay      w [T, H D] in 32-bit from the first product's 32-bit rows (tanh, second product, the two exponentials)
//   ts_wkv_scan       the recurrence, token by token for portions and single tokens alike (cutting a prompt changes no bit);
//                     afterwards the request's blocks store the last input
//   ts_wkv_project    steps in which every token is a request of its own: the mixes and their products in one kernel
//   ts_wkv_step       ... and the decay's second product, the recurrence, the heads' norm and the gate in another
//
// What a predecessor writes is read through pointers that are not __restrict__: the compiler holds the memory behind one that
// is for constant over the whole kernel and may move its loads ahead of the wait for the predecessor.
#include "activations.cuh"
#include "common.cuh"
#include "mma_utils.cuh"

namespace {

__device__ __forceinline__ void wk_cp_async_4(void* smem, const void* gmem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(s), "l"(gmem));
}

// ---------------------------------------------------------------------------------------------------------------------
// A thread owns PER neighbouring channels of TOK neighbouring tokens; the row before slides through registers.
constexpr int SH_MAX = 8;                                     // mixes a launch makes

template <typename T, int PER, int TOK>
__global__ void __launch_bounds__(128)
token_shift_kernel(T* out, const T* h, const T* __restrict__ mu, const float* state,
                   size_t state_stride, size_t prev_off, const int* __restrict__ token_request, const int* __restrict__ q_start,
                   const int* __restrict__ slots, int T_, int hidden, int n) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * PER;
  if (c >= hidden) return;
  const int t_base = blockIdx.x * TOK;
  const int count = min(TOK, T_ - t_base);
  float cur[TOK][PER], before[PER];
#pragma unroll
  for (int k = 0; k < TOK; ++k)
    if (k < count) {
      if constexpr (PER == 8) {
        const uint4 v = *reinterpret_cast<const uint4*>(h + (size_t)(t_base + k) * hidden + c);
        const T* e = reinterpret_cast<const T*>(&v);
#pragma unroll
        for (int j = 0; j < PER; ++j) cur[k][j] = to_f(e[j]);
      } else {
#pragma unroll
        for (int j = 0; j < PER; ++j) cur[k][j] = to_f(h[(size_t)(t_base + k) * hidden + c + j]);
      }
    }
#pragma unroll
  for (int k = 0; k < TOK; ++k) {
    if (k < count) {
      const int t = t_base + k, b = token_request[t];
      if (t == q_start[b]) {
        const float* prev = state + (size_t)slots[b] * state_stride + prev_off + c;
#pragma unroll
        for (int j = 0; j < PER; ++j) before[j] = prev[j];
      } else if (k == 0) {
#pragma unroll
        for (int j = 0; j < PER; ++j) before[j] = to_f(h[(size_t)(t - 1) * hidden + c + j]);
      } else {
#pragma unroll
        for (int j = 0; j < PER; ++j) before[j] = cur[k > 0 ? k - 1 : 0][j];
      }
#pragma unroll
      for (int i = 0; i < SH_MAX; ++i) {
        if (i < n) {
          T* dst = out + ((size_t)i * T_ + t) * hidden + c;
          const T* m = mu + (size_t)i * hidden + c;
          if constexpr (PER == 8) {
            const uint4 mv = __ldg(reinterpret_cast<const uint4*>(m));
            const T* me = reinterpret_cast<const T*>(&mv);
            uint4 o;
            T* oe = reinterpret_cast<T*>(&o);
#pragma unroll
            for (int j = 0; j < PER; ++j) oe[j] = from_f<T>(fmaf(before[j] - cur[k][j], to_f(me[j]), cur[k][j]));
            *reinterpret_cast<uint4*>(dst) = o;
          } else {
#pragma unroll
            for (int j = 0; j < PER; ++j) dst[j] = from_f<T>(fmaf(before[j] - cur[k][j], to_f(m[j]), cur[k][j]));
          }
        }
      }
    }
  }
}

// ---------------------------------------------------------------------------------------------------------------------
// out[t, c] = exp(-exp(sum_r w2[c, r] tanh(z[t, r]) + w0[c])): FFMA tiles of 64 tokens x 64 channels, r in ascending order.
constexpr int DC_M = 64, DC_N = 64, DC_K = 16, DC_PAD = 4;

template <typename T>
__global__ void __launch_bounds__(256)
wkv_decay_kernel(float* out, const float* z, const T* __restrict__ w2, const float* __restrict__ w0,
                 int M, int N, int R) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ __align__(16) float As[DC_K][DC_M + DC_PAD];
  __shared__ __align__(16) float Ws[DC_K][DC_N + DC_PAD];
  const int tid = threadIdx.x;
  const int m0 = blockIdx.y * DC_M, n0 = blockIdx.x * DC_N;
  const int lr = tid >> 2, lk = (tid & 3) * 4;
  const int ty = tid >> 4, tx = tid & 15;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < R; k0 += DC_K) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int k = k0 + lk + i;
      As[lk + i][lr] = (m0 + lr < M && k < R) ? tanhf(z[(size_t)(m0 + lr) * R + k]) : 0.f;
      Ws[lk + i][lr] = (n0 + lr < N && k < R) ? to_f(w2[(size_t)(n0 + lr) * R + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < DC_K; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&As[k][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&Ws[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
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
      if (n < N) out[(size_t)m * N + n] = expf(-expf(acc[i][j] + w0[n]));
    }
  }
}

// The same on the tensor cores for bfloat16 weights: tanh(z) enters as two bfloat16 terms (hi + lo, two products a step), so it
// carries 16 bits of mantissa; 32-bit accumulation.  Tiles of 64 tokens x 128 channels, 8 warps of 16 x 64; the whole rank sits
// in shared memory.  The rank is a multiple of 8, at most DM_MAX_R.
constexpr int DM_M = 64, DM_N = 128, DM_MAX_R = 256;

__global__ void __launch_bounds__(256)
wkv_decay_mma_kernel(float* out, const float* z, const bf16* __restrict__ w2, const float* __restrict__ w0, int M, int N, int R) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) unsigned char dm_smem[];
  const int Rp = (R + 15) / 16 * 16, stride = Rp + 8;
  bf16* zh = reinterpret_cast<bf16*>(dm_smem);                        // [DM_M][stride]
  bf16* zl = zh + DM_M * stride;
  bf16* ws = zl + DM_M * stride;                                      // [DM_N][stride]
  const int m0 = blockIdx.y * DM_M, n0 = blockIdx.x * DM_N;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int wm = (warp & 3) * 16, wn = (warp >> 2) * 64;
  const int chunks = Rp / 8;
  for (int i = threadIdx.x; i < DM_N * chunks; i += blockDim.x) {     // (weights: nobody's output)
    const int row = i / chunks, c = (i % chunks) * 8;
    const bool ok = n0 + row < N && c < R;
    cp_async_16(ws + row * stride + c, ok ? w2 + (size_t)(n0 + row) * R + c : w2, ok);
  }
  cp_async_commit();
  pdl_wait();
  for (int i = threadIdx.x; i < DM_M * Rp; i += blockDim.x) {
    const int row = i / Rp, c = i % Rp;
    const float t = (m0 + row < M && c < R) ? tanhf(z[(size_t)(m0 + row) * R + c]) : 0.f;
    const bf16 hi = __float2bfloat16_rn(t);
    zh[row * stride + c] = hi;
    zl[row * stride + c] = __float2bfloat16_rn(t - __bfloat162float(hi));
  }
  cp_async_wait<0>();
  __syncthreads();
  float acc[8][4];
#pragma unroll
  for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  const int mat = lane >> 3, r8 = lane & 7;
  for (int k0 = 0; k0 < Rp; k0 += 16) {
    unsigned ah[4], al[4];
    const int a_at = (wm + (mat & 1) * 8 + r8) * stride + k0 + (mat >> 1) * 8;
    ldmatrix_x4(ah[0], ah[1], ah[2], ah[3], zh + a_at);
    ldmatrix_x4(al[0], al[1], al[2], al[3], zl + a_at);
#pragma unroll
    for (int np = 0; np < 4; ++np) {
      unsigned b0, b1, b2, b3;
      ldmatrix_x4(b0, b1, b2, b3, ws + (wn + np * 16 + (mat >> 1) * 8 + r8) * stride + k0 + (mat & 1) * 8);
      mma_bf16(acc[2 * np], ah, b0, b1);
      mma_bf16(acc[2 * np], al, b0, b1);
      mma_bf16(acc[2 * np + 1], ah, b2, b3);
      mma_bf16(acc[2 * np + 1], al, b2, b3);
    }
  }
#pragma unroll
  for (int nt = 0; nt < 8; ++nt)
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      const int m = m0 + wm + (lane >> 2) + 8 * hh, c = n0 + wn + nt * 8 + (lane & 3) * 2;
      if (m >= M) continue;
      float* dst = out + (size_t)m * N + c;
      if (c < N) dst[0] = expf(-expf(acc[nt][2 * hh] + w0[c]));
      if (c + 1 < N) dst[1] = expf(-expf(acc[nt][2 * hh + 1] + w0[c + 1]));
    }
}

// ---------------------------------------------------------------------------------------------------------------------
// A warp owns WK_COLS columns of one (head, request) state: lane l holds rows l * RPL .. of them in registers over the step's
// tokens.  A block's WK_WARPS warps take neighbouring columns and share the staged rows: r, k and v as stored, w in 32-bit,
// which a warp brings whole tokens of by cp.async, two or three groups of WK_GROUP tokens ahead; one block-wide barrier a group.  Per token a lane adds its rows' share of (S + diag(u) k v^T)^T r and fades and writes its rows; the lanes' shares of
// a group are added through the warp's own piece of shared memory (lane l adds up the 32 shares of output l: token l / 2,
// column l % 2, in lane order), so nothing crosses lanes inside a token.  Few columns a warp mean many warps a scheduler: one
// warp alone issues an instruction every three or four cycles.
constexpr int WK_GROUP = 16, WK_COLS = 2, WK_WARPS = 8, WK_RED = 36;
static_assert(WK_GROUP * WK_COLS == 32, "a lane adds up one output of a group of tokens");
template <typename T, int RPL> constexpr int wk_stages() { return RPL * (int)sizeof(T) >= 32 ? 3 : 4; }

// N neighbouring values as 32-bit numbers, in loads of up to 16 bytes
template <int N> __device__ __forceinline__ void wk_load(float (&f)[N], const float* p) {
  if constexpr (N >= 4) {
#pragma unroll
    for (int i = 0; i < N; i += 4) {
      const float4 x = *reinterpret_cast<const float4*>(p + i);
      f[i] = x.x; f[i + 1] = x.y; f[i + 2] = x.z; f[i + 3] = x.w;
    }
  } else if constexpr (N == 2) {
    const float2 x = *reinterpret_cast<const float2*>(p);
    f[0] = x.x; f[1] = x.y;
  } else {
    f[0] = p[0];
  }
}
template <int N> __device__ __forceinline__ void wk_load(float (&f)[N], const bf16* p) {
  if constexpr (N == 1) {
    f[0] = to_f(p[0]);
  } else {
    unsigned x[N / 2];
    if constexpr (N == 8) *reinterpret_cast<uint4*>(x) = *reinterpret_cast<const uint4*>(p);
    else if constexpr (N == 4) *reinterpret_cast<uint2*>(x) = *reinterpret_cast<const uint2*>(p);
    else x[0] = *reinterpret_cast<const unsigned*>(p);
#pragma unroll
    for (int i = 0; i < N / 2; ++i) {
      f[2 * i] = __uint_as_float(x[i] << 16);
      f[2 * i + 1] = __uint_as_float(x[i] & 0xffff0000u);
    }
  }
}

template <typename T, int RPL>
__global__ void __launch_bounds__(WK_WARPS * 32, 1)
wkv_scan_kernel(float* out, const T* r, const T* k, const T* v, const float* w, const float* __restrict__ u, const T* h_in,
                float* state, size_t state_stride, const int* __restrict__ q_start, const int* __restrict__ slots, int H, int D,
                int V, int hidden, int fast) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float smem[];
  const int h = blockIdx.y, b = blockIdx.z;
  const int t0 = q_start[b], n = q_start[b + 1] - t0;
  if (n <= 0) return;
  constexpr int WK_STAGES = wk_stages<T, RPL>(), Dp = 32 * RPL, BC = WK_COLS * WK_WARPS, PER = 16 / (int)sizeof(T);     // (rows beyond D hold zeros)
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int b0 = blockIdx.x * BC, c0 = b0 + warp * WK_COLS;            // the block's and this warp's first column
  const int cols_here = min(BC, V - b0);
  float* base = state + (size_t)slots[b] * state_stride;
  float* S = base + (size_t)h * D * V;
  float* w_s = smem;                                                   // [WK_STAGES][WK_GROUP][Dp]
  float* red = w_s + WK_STAGES * WK_GROUP * Dp + warp * 32 * WK_RED;   // [32 outputs][WK_RED]: the lanes' shares
  T* r_s = reinterpret_cast<T*>(w_s + WK_STAGES * WK_GROUP * Dp + WK_WARPS * 32 * WK_RED);   // [WK_STAGES][WK_GROUP][Dp]
  T* k_s = r_s + WK_STAGES * WK_GROUP * Dp;
  T* v_s = k_s + WK_STAGES * WK_GROUP * Dp;                            // [WK_STAGES][WK_GROUP][BC]
  const int HD = H * D, HV = H * V;

  float s[RPL][WK_COLS], uu[RPL];
#pragma unroll
  for (int i = 0; i < RPL; ++i) {
    const int d = lane * RPL + i;
    uu[i] = d < D ? u[h * D + d] : 0.f;
#pragma unroll
    for (int j = 0; j < WK_COLS; ++j) s[i][j] = (d < D && c0 + j < V) ? S[(size_t)d * V + c0 + j] : 0.f;
  }
  if (D < Dp)
    for (int i = threadIdx.x; i < WK_STAGES * WK_GROUP * Dp; i += blockDim.x) {
      w_s[i] = 0.f;
      r_s[i] = from_f<T>(0.f);
      k_s[i] = from_f<T>(0.f);
    }
  if (cols_here < BC)
    for (int i = threadIdx.x; i < WK_STAGES * WK_GROUP * BC; i += blockDim.x) v_s[i] = from_f<T>(0.f);
  __syncthreads();

  // Which 16-byte pieces of a token's rows [r | k | w | v] a lane brings is the same for every token: where they come from, how
  // far apart two tokens' are there and here, and where they go is worked out once.  (`fast`: every piece starts on a 16-byte
  // boundary on both sides; else single values.)
  constexpr int PIECES = (RPL * (2 * (int)sizeof(T) + 4) + 15) / 16 + 1;
  const char* src[PIECES];
  unsigned src_step[PIECES], dst[PIECES], dst_step[PIECES];
  const unsigned smem0 = (unsigned)__cvta_generic_to_shared(smem);
  const int pr = D / PER, pw = D / 4, pv = (cols_here + PER - 1) / PER;
#pragma unroll
  for (int i = 0; i < PIECES; ++i) {
    int at = lane + 32 * i;
    src[i] = nullptr;
    src_step[i] = dst[i] = dst_step[i] = 0u;
    if (!fast) continue;
    if (at < 2 * pr) {
      const bool is_k = at >= pr;
      const int c = (is_k ? at - pr : at) * PER;
      src[i] = reinterpret_cast<const char*>((is_k ? k : r) + (size_t)t0 * HD + h * D + c);
      src_step[i] = HD * (unsigned)sizeof(T);
      dst[i] = smem0 + (unsigned)((const char*)((is_k ? k_s : r_s) + c) - (const char*)smem);
      dst_step[i] = Dp * (unsigned)sizeof(T);
    } else if ((at -= 2 * pr) < pw) {
      src[i] = reinterpret_cast<const char*>(w + (size_t)t0 * HD + h * D + at * 4);
      src_step[i] = HD * 4u;
      dst[i] = smem0 + (unsigned)((const char*)(w_s + at * 4) - (const char*)smem);
      dst_step[i] = Dp * 4u;
    } else if ((at -= pw) < pv) {
      src[i] = reinterpret_cast<const char*>(v + (size_t)t0 * HV + h * V + b0 + at * PER);
      src_step[i] = HV * (unsigned)sizeof(T);
      dst[i] = smem0 + (unsigned)((const char*)(v_s + at * PER) - (const char*)smem);
      dst_step[i] = BC * (unsigned)sizeof(T);
    }
  }
  auto fetch = [&](int g0, int st) {
    const int gn = min(WK_GROUP, n - g0);
    for (int q = warp; q < gn; q += WK_WARPS) {
      const int at = st * WK_GROUP + q;
      if (fast) {
#pragma unroll
        for (int i = 0; i < PIECES; ++i)
          if (src[i] != nullptr)
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(dst[i] + (unsigned)at * dst_step[i]),
                         "l"(src[i] + (size_t)(unsigned)(g0 + q) * src_step[i]));
      } else {
        const size_t t = t0 + g0 + q;
        for (int c = lane; c < D; c += 32) {
          r_s[at * Dp + c] = r[t * HD + h * D + c];
          k_s[at * Dp + c] = k[t * HD + h * D + c];
          wk_cp_async_4(w_s + at * Dp + c, w + t * HD + h * D + c);
        }
        for (int c = lane; c < cols_here; c += 32) v_s[at * BC + c] = v[t * HV + h * V + b0 + c];
      }
    }
  };
#pragma unroll
  for (int st = 0; st < WK_STAGES - 1; ++st) {
    if (st * WK_GROUP < n) fetch(st * WK_GROUP, st);
    cp_async_commit();
  }
  int st = 0;
  for (int g0 = 0; g0 < n; g0 += WK_GROUP, st = (st + 1) % WK_STAGES) {
    const int gn = min(WK_GROUP, n - g0);
    cp_async_wait<WK_STAGES - 2>();
    __syncthreads();                                       // this group is here for all; the one before it is used up
    if (g0 + (WK_STAGES - 1) * WK_GROUP < n) fetch(g0 + (WK_STAGES - 1) * WK_GROUP, (st + WK_STAGES - 1) % WK_STAGES);
    cp_async_commit();
    float o[WK_GROUP][WK_COLS];
    const T* r_l = r_s + st * WK_GROUP * Dp + lane * RPL;
    const T* k_l = k_s + st * WK_GROUP * Dp + lane * RPL;
    const float* w_l = w_s + st * WK_GROUP * Dp + lane * RPL;
    const T* v_l = v_s + st * WK_GROUP * BC + warp * WK_COLS;
    auto token = [&](int q, float (&oq)[WK_COLS]) {
      float rq[RPL], kq[RPL], wq[RPL], vf[WK_COLS], c = 0.f;   // c: this lane's part of the sum of r u k
      wk_load(rq, r_l + q * Dp);
      wk_load(kq, k_l + q * Dp);
      wk_load(wq, w_l + q * Dp);
      wk_load(vf, v_l + q * BC);
#pragma unroll
      for (int j = 0; j < WK_COLS; ++j) oq[j] = 0.f;
#pragma unroll
      for (int i = 0; i < RPL; ++i) {
        c = fmaf(rq[i], uu[i] * kq[i], c);
#pragma unroll
        for (int j = 0; j < WK_COLS; ++j) {
          oq[j] = fmaf(s[i][j], rq[i], oq[j]);
          s[i][j] = fmaf(wq[i], s[i][j], kq[i] * vf[j]);
        }
      }
#pragma unroll
      for (int j = 0; j < WK_COLS; ++j) oq[j] = fmaf(c, vf[j], oq[j]);
    };
    if (gn == WK_GROUP) {
#pragma unroll
      for (int q = 0; q < WK_GROUP; ++q) token(q, o[q]);
    } else {
#pragma unroll
      for (int q = 0; q < WK_GROUP; ++q) {
#pragma unroll
        for (int j = 0; j < WK_COLS; ++j) o[q][j] = 0.f;
        if (q < gn) token(q, o[q]);
      }
    }
#pragma unroll
    for (int q = 0; q < WK_GROUP; ++q)
#pragma unroll
      for (int j = 0; j < WK_COLS; ++j) red[(q * WK_COLS + j) * WK_RED + lane] = o[q][j];
    __syncwarp();
    float total = 0.f;
#pragma unroll
    for (int i = 0; i < 32; i += 4) {
      const float4 p = *reinterpret_cast<const float4*>(red + lane * WK_RED + i);
      total += (p.x + p.y) + (p.z + p.w);
    }
    const int q = lane / WK_COLS, c = c0 + lane % WK_COLS;
    if (q < gn && c < V) out[(size_t)(t0 + g0 + q) * HV + h * V + c] = total;
    // (the next group's shares are written past the next block-wide barrier)
  }
  cp_async_wait<0>();
#pragma unroll
  for (int i = 0; i < RPL; ++i) {
    const int d = lane * RPL + i;
#pragma unroll
    for (int j = 0; j < WK_COLS; ++j)
      if (d < D && c0 + j < V) S[(size_t)d * V + c0 + j] = s[i][j];
  }
  // the request's last input, for its next token; every block of the request takes a share of the channels
  float* prev = base + (size_t)H * D * V;
  const T* last = h_in + (size_t)(t0 + n - 1) * hidden;
  for (int c = (h * gridDim.x + blockIdx.x) * blockDim.x + threadIdx.x; c < hidden; c += H * gridDim.x * blockDim.x)
    prev[c] = to_f(last[c]);
}

// ---------------------------------------------------------------------------------------------------------------------
// Single tokens (bfloat16): out[s, m, :] = W[s] mix_s(m) for the s < n stacked matrices [n, N, K], and z[m, :] = w1 mix_n(m) in
// 32-bit.  A block takes 64 columns of one matrix: it puts the first weights of its warps on their way (they are nobody's
// output), then makes its mix of all rows in shared memory and multiplies on the tensor cores.  KS = 2: two warps share 8 columns, each
// half of k (launches of one wave); KS = 1: a warp takes the whole of k, two blocks an SM.  (The products' k index is a
// permutation of the real one, the same for both operands.)
constexpr int PJ_COLS = 64, PJ_UNROLL = 8, PJ_PAD = 32;

template <int ROWS, int KS>
__global__ void __launch_bounds__(PJ_COLS / 8 * KS * 32)
wkv_project_kernel(bf16* out, float* z, const bf16* h, const bf16* __restrict__ mu, const bf16* __restrict__ w,
                   const bf16* __restrict__ w1, const float* state,
                   size_t state_stride, size_t prev_off, const int* __restrict__ slots, int M, int n, int N, int R, int K) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) unsigned char pj_smem[];
  bf16* x_s = reinterpret_cast<bf16*>(pj_smem);                       // [ROWS][K + PJ_PAD]
  constexpr int THREADS = PJ_COLS / 8 * KS * 32;
  __shared__ float red[PJ_COLS / 8][ROWS][8];
  const int xs = K + PJ_PAD;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int g = lane >> 2, t = lane & 3;
  const int per = (N + PJ_COLS - 1) / PJ_COLS;
  const int s = min((int)blockIdx.x / per, n);                        // which mix; n: the decay's
  const int n_cols = s < n ? N : R;
  const int n0 = ((int)blockIdx.x - s * per) * PJ_COLS + warp / KS * 8;
  const bool n_ok = n0 + g < n_cols;
  const bf16* mat = s < n ? w + (size_t)s * N * K : w1;
  const int steps = (K + 31) / 32, share = (steps + KS - 1) / KS;
  const int st0 = warp % KS * share, st1 = min(st0 + share, steps);
  const bf16* wrow = mat + (size_t)(n_ok ? n0 + g : 0) * K + t * 8;
  uint4 wv[2][PJ_UNROLL];
  auto fetch = [&](int st, int bf) {
#pragma unroll
    for (int q = 0; q < PJ_UNROLL; ++q) {
      const int kk = (st + q) * 32;
      wv[bf][q] = (n_ok && st + q < st1 && kk + t * 8 < K) ? __ldcs(reinterpret_cast<const uint4*>(wrow + kk)) : make_uint4(0u, 0u, 0u, 0u);
    }
  };
  fetch(st0, 0);
  if constexpr (ROWS == 8) fetch(st0 + PJ_UNROLL, 1);
  pdl_wait();
  for (int i = threadIdx.x * 8; i < ROWS * K; i += THREADS * 8) {
    const int m = i / K, c = i - m * K;
    uint4 o = make_uint4(0u, 0u, 0u, 0u);
    if (m < M) {
      const uint4 hv = *reinterpret_cast<const uint4*>(h + (size_t)m * K + c);
      const uint4 mv = *reinterpret_cast<const uint4*>(mu + (size_t)s * K + c);
      const float4* pv = reinterpret_cast<const float4*>(state + (size_t)slots[m] * state_stride + prev_off + c);
      const float4 p0 = pv[0], p1 = pv[1];
      const float pe[8] = {p0.x, p0.y, p0.z, p0.w, p1.x, p1.y, p1.z, p1.w};
      const bf16* he = reinterpret_cast<const bf16*>(&hv);
      const bf16* me = reinterpret_cast<const bf16*>(&mv);
      bf16* oe = reinterpret_cast<bf16*>(&o);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float x = to_f(he[j]);
        oe[j] = from_f<bf16>(fmaf(pe[j] - x, to_f(me[j]), x));
      }
    }
    *reinterpret_cast<uint4*>(x_s + m * xs + c) = o;
  }
  __syncthreads();
  float acc[4] = {0.f, 0.f, 0.f, 0.f};
  auto multiply = [&](int st, int bf) {
#pragma unroll
    for (int q = 0; q < PJ_UNROLL; ++q) {
      const int kk = (st + q) * 32 + t * 8;
      const bool ok = st + q < st1 && kk < K;
      const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
      const uint4 xv = ok ? *reinterpret_cast<const uint4*>(x_s + g * xs + kk) : zero;
      uint4 yv = zero;
      if constexpr (ROWS == 16) yv = ok ? *reinterpret_cast<const uint4*>(x_s + (g + 8) * xs + kk) : zero;
      const unsigned a1[4] = {xv.x, yv.x, xv.y, yv.y}, a2[4] = {xv.z, yv.z, xv.w, yv.w};
      mma_bf16(acc, a1, wv[bf][q].x, wv[bf][q].y);
      mma_bf16(acc, a2, wv[bf][q].z, wv[bf][q].w);
    }
  };
  if constexpr (ROWS == 8) {
    for (int st = st0; st < st1; st += 2 * PJ_UNROLL) {
      multiply(st, 0);
      if (st + 2 * PJ_UNROLL < st1) fetch(st + 2 * PJ_UNROLL, 0);
      if (st + PJ_UNROLL < st1) multiply(st + PJ_UNROLL, 1);
      if (st + 3 * PJ_UNROLL < st1) fetch(st + 3 * PJ_UNROLL, 1);
    }
  } else {
    for (int st = st0; st < st1; st += 2 * PJ_UNROLL) {
      if (st + PJ_UNROLL < st1) fetch(st + PJ_UNROLL, 1);
      multiply(st, 0);
      if (st + 2 * PJ_UNROLL < st1) fetch(st + 2 * PJ_UNROLL, 0);
      if (st + PJ_UNROLL < st1) multiply(st + PJ_UNROLL, 1);
    }
  }
  // (lane (g, t) holds rows g and g + 8 of columns 2 t and 2 t + 1)
  if constexpr (KS == 2) {
    if (warp & 1) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        red[warp >> 1][g][2 * t + e] = acc[e];
        if constexpr (ROWS == 16) red[warp >> 1][g + 8][2 * t + e] = acc[2 + e];
      }
    }
    __syncthreads();
    if (warp & 1) return;
  }
#pragma unroll
  for (int hh = 0; hh < ROWS / 8; ++hh)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int m = g + 8 * hh, c = n0 + 2 * t + e;
      if (m >= M || c >= n_cols) continue;
      const float val = KS == 2 ? acc[2 * hh + e] + red[warp >> 1][m][2 * t + e] : acc[2 * hh + e];
      if (s < n) out[((size_t)s * M + m) * N + c] = from_f<bf16>(val);
      else z[(size_t)m * R + c] = val;
    }
}

// One block a (head, request), every token a request of its own: thread (part, col) holds ST_ROWS rows of state column col,
// fetched before the wait for the predecessor (no kernel but this one writes the state in a step).
constexpr int ST_ROWS = 16;

template <typename T, int THREADS>
__global__ void __launch_bounds__(THREADS, THREADS == 256 ? 3 : 1)
wkv_step_kernel(T* out, const T* rkvg, const float* z, const T* __restrict__ w2,
                const float* __restrict__ w0, const float* __restrict__ u, const float* __restrict__ norm_w, float eps,
                const T* h_in, float* state, size_t state_stride, const int* __restrict__ slots, int M, int H, int D, int R,
                int hidden, int cols, int w2_in_smem) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float st_smem[];
  __shared__ float scratch[32];
  const int h = blockIdx.x, b = blockIdx.y;
  const int col = threadIdx.x % cols, part = threadIdx.x / cols, parts = blockDim.x / cols;
  const int HD = H * D;
  constexpr int PER = 16 / (int)sizeof(T);
  T* w2_s = reinterpret_cast<T*>(st_smem);                 // [D][R] where w2_in_smem
  float* z_s = st_smem + (w2_in_smem ? (D * R * (int)sizeof(T) + 15) / 16 * 4 : 0);   // [R], rounded up to 16 bytes
  float* r_s = z_s + (R + 3) / 4 * 4;                      // [D] each
  float* k_s = r_s + D;
  float* w_s = k_s + D;
  float* c_s = w_s + D;                                    // r u k
  float* o_s = c_s + D;                                    // [parts][cols]
  float* base = state + (size_t)slots[b] * state_stride;
  float* S = base + (size_t)h * D * D;
  const T* w2_h = w2 + (size_t)h * D * R;
  if (w2_in_smem)
    for (int i = threadIdx.x * PER; i < D * R; i += blockDim.x * PER) cp_async_16(w2_s + i, w2_h + i, true);
  cp_async_commit();
  float s[ST_ROWS];
#pragma unroll
  for (int i = 0; i < ST_ROWS; ++i) {
    const int d = part * ST_ROWS + i;
    s[i] = (col < D && d < D) ? S[(size_t)d * D + col] : 0.f;
  }
  const bool mine = threadIdx.x < D;                       // (the block has a thread for every channel)
  const float u_d = mine ? u[h * D + threadIdx.x] : 0.f, n_d = mine ? norm_w[h * D + threadIdx.x] : 0.f;
  if (mine) w_s[threadIdx.x] = w0[h * D + threadIdx.x];
  pdl_wait();
  const T* row = rkvg + (size_t)b * HD + h * D;            // (r, k, v, gate: one matrix of rows each)
  const size_t plane = (size_t)M * HD;
  float r_d = 0.f, k_d = 0.f, vj = 0.f, gate = 0.f;
  if (mine) {
    r_d = to_f(row[threadIdx.x]);
    k_d = to_f(row[plane + threadIdx.x]);
    gate = to_f(row[3 * plane + threadIdx.x]);
  }
  if (col < D) vj = to_f(row[2 * plane + col]);
  for (int i = threadIdx.x; i < R; i += blockDim.x) z_s[i] = tanhf(z[(size_t)b * R + i]);
  if (mine) {
    r_s[threadIdx.x] = r_d;
    k_s[threadIdx.x] = k_d;
    c_s[threadIdx.x] = r_d * u_d * k_d;
  }
  cp_async_wait<0>();
  __syncthreads();
  // the decays: eight lanes a channel; a warp's four channels lie inside or outside [0, D rounded up) together
  for (int d0 = threadIdx.x >> 3; d0 < (D + 3) / 4 * 4; d0 += blockDim.x >> 3) {
    const int sub = threadIdx.x & 7;
    float a = 0.f;
    if (d0 < D) {
      if (w2_in_smem) {
        for (int i = sub * PER; i < R; i += 8 * PER) {
          const uint4 v = *reinterpret_cast<const uint4*>(w2_s + (size_t)d0 * R + i);
          const T* e = reinterpret_cast<const T*>(&v);
#pragma unroll
          for (int j = 0; j < PER; ++j) a = fmaf(to_f(e[j]), z_s[i + j], a);
        }
      } else {
        for (int i = sub; i < R; i += 8) a = fmaf(to_f(w2_h[(size_t)d0 * R + i]), z_s[i], a);
      }
    }
    a += __shfl_xor_sync(0xffffffffu, a, 1);
    a += __shfl_xor_sync(0xffffffffu, a, 2);
    a += __shfl_xor_sync(0xffffffffu, a, 4);
    if (sub == 0 && d0 < D) w_s[d0] = expf(-expf(a + w_s[d0]));
  }
  __syncthreads();
  float o = 0.f;
#pragma unroll
  for (int i = 0; i < ST_ROWS; ++i) {
    const int d = part * ST_ROWS + i;
    if (d < D) {
      o = fmaf(s[i], r_s[d], fmaf(c_s[d], vj, o));
      s[i] = fmaf(w_s[d], s[i], k_s[d] * vj);
      if (col < D) S[(size_t)d * D + col] = s[i];
    }
  }
  o_s[part * cols + col] = o;
  __syncthreads();
  float total = 0.f;
  if (mine)                                                // (column threadIdx.x, whose row part is the first)
    for (int p = 0; p < parts; ++p) total += o_s[p * cols + threadIdx.x];
  const float ss = block_sum(total * total, scratch);
  if (mine) {
    const float rstd = 1.f / sqrtf(ss / (float)D + eps);
    out[(size_t)b * HD + h * D + threadIdx.x] = from_f<T>(total * rstd * n_d * silu_for<T>(gate));
  }
  float* prev = base + (size_t)H * D * D;
  for (int c = h * blockDim.x + threadIdx.x; c < hidden; c += H * blockDim.x) prev[c] = to_f(h_in[(size_t)b * hidden + c]);
}

}  // namespace

// out [n, T, hidden]; h [T, hidden]; mu [n, hidden] (all in `dtype`); state [slots, state_stride] 32-bit with the row before
// the step's first token at prev_off.
TS_API int ts_token_shift(void* out, const void* h, const void* mu, const float* state, long long state_stride,
                          long long prev_off, const int* token_request, const int* q_start, const int* slots, int T, int hidden,
                          int n, int dtype, void* stream) {
  if (T <= 0 || n <= 0 || hidden <= 0) return 0;
  if (n > SH_MAX) TS_REFUSE(TS_ERR_LIMIT, "ts_token_shift: %d mixes (limit %d)", n, SH_MAX);
  cudaStream_t s = (cudaStream_t)stream;
  const bool vec = dtype == TS_BF16 && hidden % 8 == 0 && !(((uintptr_t)out | (uintptr_t)h | (uintptr_t)mu) & 15);
  const bool few = T <= 256;
  const dim3 grid(few ? T : ceil_div(T, 4), ceil_div(hidden, vec ? 1024 : 128));
  if (grid.y > 65535) TS_REFUSE(TS_ERR_LIMIT, "ts_token_shift: rows of %d", hidden);
#define TS_SHIFT(TT, PER, TOK)                                                                                            \
  ts_launch(token_shift_kernel<TT, PER, TOK>, grid, dim3(128), 0, s, (TT*)out, (const TT*)h, (const TT*)mu, state, (size_t)state_stride, \
            (size_t)prev_off, token_request, q_start, slots, T, hidden, n)
  if (dtype == TS_F32) { if (few) TS_SHIFT(float, 1, 1); else TS_SHIFT(float, 1, 4); }
  else if (dtype == TS_BF16) {
    if (vec) { if (few) TS_SHIFT(bf16, 8, 1); else TS_SHIFT(bf16, 8, 4); }
    else { if (few) TS_SHIFT(bf16, 1, 1); else TS_SHIFT(bf16, 1, 4); }
  } else TS_REFUSE(TS_ERR_DTYPE, "ts_token_shift: dtype %d", dtype);
#undef TS_SHIFT
  TS_LAUNCH_CHECK();
}

// out [T, N] 32-bit; z [T, R] 32-bit; w2 [N, R] in `dtype`; w0 [N] 32-bit.
TS_API int ts_wkv_decay(float* out, const float* z, const void* w2, const float* w0, int T, int N, int R, int dtype, void* stream) {
  if (T <= 0 || N <= 0) return 0;
  if (R <= 0) TS_REFUSE(TS_ERR_SHAPE, "ts_wkv_decay: a rank of %d", R);
  const dim3 grid(ceil_div(N, DC_N), ceil_div(T, DC_M));
  if (grid.y > 65535) TS_REFUSE(TS_ERR_LIMIT, "ts_wkv_decay: %d tokens", T);
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == TS_BF16 && R % 8 == 0 && R <= DM_MAX_R && !((uintptr_t)w2 & 15)) {
    const size_t smem = (size_t)(2 * DM_M + DM_N) * ((R + 15) / 16 * 16 + 8) * 2;
    static size_t configured = 0;
    if (smem > 48 * 1024 && smem > configured) {
      cudaError_t e = cudaFuncSetAttribute(wkv_decay_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) TS_REFUSE((int)e, "ts_wkv_decay: shared memory %zu: %s", smem, cudaGetErrorString(e));
      configured = smem;
    }
    ts_launch(wkv_decay_mma_kernel, dim3(ceil_div(N, DM_N), ceil_div(T, DM_M)), dim3(256), smem, s, out, z, (const bf16*)w2, w0, T, N, R);
    TS_LAUNCH_CHECK();
  }
  if (dtype == TS_F32) ts_launch(wkv_decay_kernel<float>, grid, dim3(256), 0, s, out, z, (const float*)w2, w0, T, N, R);
  else if (dtype == TS_BF16) ts_launch(wkv_decay_kernel<bf16>, grid, dim3(256), 0, s, out, z, (const bf16*)w2, w0, T, N, R);
  else TS_REFUSE(TS_ERR_DTYPE, "ts_wkv_decay: dtype %d", dtype);
  TS_LAUNCH_CHECK();
}

// out [T, H V] 32-bit; r, k [T, H D] and v [T, H V] in `dtype`; w [T, H D] and u [H, D] 32-bit; h_in [T, hidden]: the mixer's
// input; state [slots, state_stride]: [H D V | hidden].  longest: the most tokens a request brings (0: not known); long
// portions are launched late (see ts_launch_late).
constexpr int WK_LATE_TOKENS = 64;
// Long portions whose blocks are at most one an SM ask for so much shared memory that no SM takes two of them (left to itself the
// hardware puts two on some SMs while others stay empty, and the scan is as slow as those).
constexpr size_t WK_ALONE_BYTES = 116 * 1024;

TS_API int ts_wkv_scan(float* out, const void* r, const void* k, const void* v, const float* w, const float* u, const void* h_in,
                       float* state, long long state_stride, const int* q_start, const int* slots, int B, int H, int D, int V,
                       int hidden, int longest, int dtype, void* stream) {
  if (B <= 0) return 0;
  if (H <= 0 || D <= 0 || V <= 0) TS_REFUSE(TS_ERR_SHAPE, "ts_wkv_scan: %d heads of %d x %d", H, D, V);
  if (D > 256) TS_REFUSE(TS_ERR_LIMIT, "ts_wkv_scan: keys of %d (limit 256)", D);
  if (B > 65535 || H > 65535) TS_REFUSE(TS_ERR_LIMIT, "ts_wkv_scan: %d requests / %d heads per launch", B, H);
  cudaStream_t s = (cudaStream_t)stream;
  const int elem = dtype == TS_F32 ? 4 : 2, per = 16 / elem;
  const int fast = D % per == 0 && V % per == 0 && D % 4 == 0 &&
                   !(((uintptr_t)r | (uintptr_t)k | (uintptr_t)v | (uintptr_t)w) & 15);
  const dim3 grid(ceil_div(V, WK_COLS * WK_WARPS), H, B);
  const bool alone = longest >= WK_LATE_TOKENS && (long long)grid.x * grid.y * grid.z <= 148;
#define TS_WKR(TT, RPL)                                                                                                  \
  do {                                                                                                                   \
    size_t smem = (size_t)wk_stages<TT, RPL>() * WK_GROUP * (32 * RPL * (sizeof(float) + 2 * sizeof(TT)) + WK_COLS * WK_WARPS * sizeof(TT)) + \
                        sizeof(float) * WK_WARPS * 32 * WK_RED;                                                          \
    if (alone && smem < WK_ALONE_BYTES) smem = WK_ALONE_BYTES;                                                           \
    static bool configured = false;                                                                                      \
    if (!configured) {                                                                                                   \
      cudaError_t e = cudaFuncSetAttribute(wkv_scan_kernel<TT, RPL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(smem < WK_ALONE_BYTES ? WK_ALONE_BYTES : smem)); \
      if (e != cudaSuccess) TS_REFUSE((int)e, "ts_wkv_scan: shared memory %zu: %s", smem, cudaGetErrorString(e));        \
      configured = true;                                                                                                 \
    }                                                                                                                    \
    if (longest >= WK_LATE_TOKENS)                                                                                       \
      ts_launch_late(wkv_scan_kernel<TT, RPL>, grid, dim3(WK_WARPS * 32), smem, s, out, (const TT*)r, (const TT*)k, (const TT*)v, w, u, \
                     (const TT*)h_in, state, (size_t)state_stride, q_start, slots, H, D, V, hidden, fast);               \
    else                                                                                                                 \
      ts_launch(wkv_scan_kernel<TT, RPL>, grid, dim3(WK_WARPS * 32), smem, s, out, (const TT*)r, (const TT*)k, (const TT*)v, w, u, \
                (const TT*)h_in, state, (size_t)state_stride, q_start, slots, H, D, V, hidden, fast);                    \
  } while (0)
#define TS_WK(TT)                  \
  do {                             \
    if (D <= 32) TS_WKR(TT, 1);    \
    else if (D <= 64) TS_WKR(TT, 2);  \
    else if (D <= 128) TS_WKR(TT, 4); \
    else TS_WKR(TT, 8);            \
  } while (0)
  if (dtype == TS_F32) TS_WK(float);
  else if (dtype == TS_BF16) TS_WK(bf16);
  else TS_REFUSE(TS_ERR_DTYPE, "ts_wkv_scan: dtype %d", dtype);
#undef TS_WK
#undef TS_WKR
  TS_LAUNCH_CHECK();
}

// bfloat16; M <= 16 tokens, each a request of its own (that of slots[m]); h [M, K]; mu [n + 1, K] (the last row the decay's);
// w [n, N, K]; w1 [R, K]; out [n, M, N]; z [M, R] 32-bit.
TS_API int ts_wkv_project_supported(int M, int K, int dtype) { return dtype == TS_BF16 && M > 0 && M <= 16 && K % 8 == 0 && K <= 6144; }

TS_API int ts_wkv_project(void* out, float* z, const void* h, const void* mu, const void* w, const void* w1, const float* state,
                          long long state_stride, long long prev_off, const int* slots, int M, int n, int N, int R, int K,
                          void* stream) {
  if (M <= 0 || n <= 0 || N <= 0 || R <= 0) return 0;
  if (!ts_wkv_project_supported(M, K, TS_BF16) || state_stride % 4 || prev_off % 4 ||
      (((uintptr_t)h | (uintptr_t)mu | (uintptr_t)w | (uintptr_t)w1 | (uintptr_t)state) & 15))
    TS_REFUSE(TS_ERR_UNSUPPORTED, "ts_wkv_project: %d tokens, rows of %d", M, K);
  const dim3 grid(n * ceil_div(N, PJ_COLS) + ceil_div(R, PJ_COLS));
  cudaStream_t s = (cudaStream_t)stream;
#define TS_PJ(ROWS, KS)                                                                                                  \
  do {                                                                                                                   \
    const size_t smem = (size_t)ROWS * (K + PJ_PAD) * 2;                                                                 \
    static size_t configured = 0;                                                                                        \
    if (smem > 40 * 1024 && smem > configured) {                                                                         \
      cudaError_t e = cudaFuncSetAttribute(wkv_project_kernel<ROWS, KS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
      if (e != cudaSuccess) TS_REFUSE((int)e, "ts_wkv_project: shared memory %zu: %s", smem, cudaGetErrorString(e));     \
      configured = smem;                                                                                                 \
    }                                                                                                                    \
    ts_launch(wkv_project_kernel<ROWS, KS>, grid, dim3(PJ_COLS / 8 * KS * 32), smem, s, (bf16*)out, z, (const bf16*)h, (const bf16*)mu, \
              (const bf16*)w, (const bf16*)w1, state, (size_t)state_stride, (size_t)prev_off, slots, M, n, N, R, K);     \
  } while (0)
  const bool one_wave = grid.x <= 148;
  if (M <= 8) { if (one_wave) TS_PJ(8, 2); else TS_PJ(8, 1); }
  else { if (one_wave) TS_PJ(16, 2); else TS_PJ(16, 1); }
#undef TS_PJ
  TS_LAUNCH_CHECK();
}

// Heads whose state a block holds in registers: value columns rounded up to whole warps times row parts of 16.
TS_API int ts_wkv_step_supported(int D, int V) {
  return D > 0 && V == D && ceil_div(V, 32) * 32 * ceil_div(D, ST_ROWS) <= 1024;
}

// out [M, H V]; rkvg [4, M, H D] in `dtype`; z [M, R] 32-bit (before the tanh); w2 [H D, R] in `dtype`; w0 [H D], u [H, D] and
// norm_w [H V] 32-bit; every token a request of its own (that of slots[m]).
TS_API int ts_wkv_step(void* out, const void* rkvg, const float* z, const void* w2, const float* w0, const float* u,
                       const float* norm_w, float eps, const void* h_in, float* state, long long state_stride, const int* slots,
                       int M, int H, int D, int R, int hidden, int dtype, void* stream) {
  if (M <= 0) return 0;
  if (!ts_wkv_step_supported(D, D)) TS_REFUSE(TS_ERR_UNSUPPORTED, "ts_wkv_step: heads of %d", D);
  if (M > 65535) TS_REFUSE(TS_ERR_LIMIT, "ts_wkv_step: %d requests per launch", M);
  const int cols = ceil_div(D, 32) * 32, parts = ceil_div(D, ST_ROWS), elem = dtype == TS_F32 ? 4 : 2;
  // (R a multiple of what 16 bytes hold, so that a row's pieces start on 16-byte boundaries)
  const int w2_in_smem = R % (16 / elem) == 0 && !((uintptr_t)w2 & 15) && D * R * elem <= 32 * 1024;
  const size_t smem = (w2_in_smem ? ((size_t)D * R * elem + 15) / 16 * 16 : 0) +
                      sizeof(float) * ((size_t)4 * D + (R + 3) / 4 * 4 + cols * parts);
  if (smem > 47 * 1024) TS_REFUSE(TS_ERR_UNSUPPORTED, "ts_wkv_step: a rank of %d", R);
  cudaStream_t s = (cudaStream_t)stream;
#define TS_ST(TT, TH)                                                                                                      \
  ts_launch(wkv_step_kernel<TT, TH>, dim3(H, M), dim3(cols * parts), smem, s, (TT*)out, (const TT*)rkvg, z, (const TT*)w2, w0, u, \
            norm_w, eps, (const TT*)h_in, state, (size_t)state_stride, slots, M, H, D, R, hidden, cols, w2_in_smem)
  if (dtype == TS_F32) { if (cols * parts <= 256) TS_ST(float, 256); else TS_ST(float, 1024); }
  else if (dtype == TS_BF16) { if (cols * parts <= 256) TS_ST(bf16, 256); else TS_ST(bf16, 1024); }
  else TS_REFUSE(TS_ERR_DTYPE, "ts_wkv_step: dtype %d", dtype);
#undef TS_ST
  TS_LAUNCH_CHECK();
}
