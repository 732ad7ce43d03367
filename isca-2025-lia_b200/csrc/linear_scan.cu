// Linear-attention recurrences with a matrix state per head, for prompts, portions of prompts and single decoded tokens
// alike, and what prepares their inputs.
//
//   DECAY  (a fixed decay per head):     S_t = d_h S_{t-1} + k_t v_t^T                      o_t = S_t^T q_t
//   DELTA  (gated delta rule):           S'  = g_t S_{t-1};  u_t = beta_t (v_t - S'^T k_t);  S_t = S' + k_t u_t^T;  o_t = S_t^T q_t
//   FORGET (keyless: the per-channel forget gate f_t keeps, its complement 1 - f_t writes):
//                                        row d of S:  S[d] <- f[d] S[d] + (1 - f[d]) v      o = sum_d q[d] S[d]
//
// The state is fp32, one [vdim][dim] matrix per (slot, head) -- stored transposed so that the dim-long column a warp owns
// is contiguous.  A warp keeps CW columns in registers for the whole portion, lane l owning rows l, l + 32, ...; a token
// costs one butterfly reduction (CW sums for DECAY; 2 CW + 1 for DELTA, where S'^T k, S'^T q and k . q are reduced together
// and o_t = g S_{t-1}^T q + u (k . q) needs no second pass).  The 8 warps of a block share the q and k of their head through
// a double-buffered shared-memory stage of TB tokens fetched while the previous TB are processed (128-bit loads where the rows
// allow them).  q and k may belong to a
// smaller number of heads than v (head h reads q/k head h / (H / G)); an activation (SiLU) can be applied as the inputs are
// staged, so that a projection's output feeds the recurrence directly.
//
//   conv_prep:         per token, a short causal convolution over time per channel of q | k | v (taps - 1 earlier inputs come
//                      from the rows before it in the same portion, or from the sequence's state), SiLU, q and k made unit
//                      vectors per head (q also scaled), and the per-head gates beta = sigmoid(.), g = exp(-exp(A) softplus(. + dt)).
//   conv_state_update: the last taps - 1 inputs of every portion become the sequence's new convolution state.
//   conv_act:          a short causal convolution over time per channel of ONE column range with an input bias, an output bias and an
//                      activation, the update of its state, and the step sizes and decays of a state-space recurrence beside it.
//
// Two more recurrences, on inputs that conv_act has made fp32:
//   ssd_scan    (state-space duality, a scalar decay per head and token):   S_t = g_t S_{t-1} + dt_t B_t x_t^T,   y_t = S_t^T C_t + D_h x_t.
//               State [vdim][N] per (slot, head) as above, but lanes share columns: a thread owns N / 16 rows of four columns, so one 128-bit
//               read of B or C serves 16 cells, and the sums of several tokens meet in one round of exchanges.
//   rglru_scan  (real-gated linear recurrent unit, one number per channel): S_t = a_t S_{t-1} + sqrt(1 - a_t^2) i_t u_t,  out_t = S_t gelu(y_t).
//               128 tokens at a time: 32 half-warps fold 4 tokens each into one affine map, the maps are chained through shared memory.
#include <math.h>

#include "common.cuh"

namespace {

template <typename T> __device__ __forceinline__ float ldf(const T* p);
template <> __device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf<bf16>(const bf16* p) { return __bfloat162float(*p); }

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }

// ---------------------------------------------------------------------------------------------------- convolution + gates
constexpr int MAX_TAPS = 16;

struct ConvCols {          // where the q, k, v channels sit in a row of the projection's output
  int q_off, k_off, v_off, nq, nk, nv;       // channels of q, of k and of v
  __device__ __forceinline__ int col(int c) const { return c < nq ? q_off + c : (c < nq + nk ? k_off + (c - nq) : v_off + (c - nq - nk)); }
};

// Block per token row.  meta[row] = {slot, position}; rows of one portion are consecutive and so are their positions.
// state [slot][taps-1][C] holds the inputs of the taps - 1 positions before the portion (zero before the sequence's start).
template <typename T>
__global__ void __launch_bounds__(256) conv_prep_kernel(const T* __restrict__ y, int ld, ConvCols cc, const float* __restrict__ wconv,
                                                        const float* __restrict__ state, const int* __restrict__ meta, float* __restrict__ gates,
                                                        const float* __restrict__ a_log, const float* __restrict__ dt_bias, float* __restrict__ qk,
                                                        float* __restrict__ v, int G, int H, int dim, int vdim, int taps, float q_scale,
                                                        float unit_eps) {
  extern __shared__ float ch[];                 // C channels after convolution and SiLU
  const int row = blockIdx.x;
  const int slot = meta[2 * row], pos = meta[2 * row + 1];
  const int C = cc.nq + cc.nk + cc.nv;
  int inside = 1;                               // rows row-1 .. row-(inside-1) belong to this portion
  while (inside < taps && row - inside >= 0 && meta[2 * (row - inside)] == slot && meta[2 * (row - inside) + 1] == pos - inside) ++inside;
  const float* st = state + (size_t)slot * (taps - 1) * C;
  for (int c = threadIdx.x; c < C; c += 256) {
    const int col = cc.col(c);
    float acc = 0.f;
    for (int j = 0; j < taps; ++j) {            // j tokens back
      const float xin = j < inside ? ldf(y + (size_t)(row - j) * ld + col) : st[(size_t)(inside - 1 - j + taps - 1) * C + c];
      acc = fmaf(wconv[(size_t)c * taps + taps - 1 - j], xin, acc);
    }
    acc = silu(acc);
    ch[c] = acc;
    if (c >= cc.nq + cc.nk) v[(size_t)row * cc.nv + c - cc.nq - cc.nk] = acc;
  }
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int hd = warp; hd < 2 * G; hd += 8) {    // q heads, then k heads
    float ss = 0.f;
    for (int i = lane; i < dim; i += 32) ss += ch[hd * dim + i] * ch[hd * dim + i];
    ss = warp_sum(ss);
    const float inv = (hd < G ? q_scale : 1.0f) / sqrtf(ss + unit_eps);
    for (int i = lane; i < dim; i += 32) qk[(size_t)row * (cc.nq + cc.nk) + hd * dim + i] = ch[hd * dim + i] * inv;
  }
  for (int h = threadIdx.x; h < H; h += 256) {
    float* gr = gates + (size_t)row * 2 * H;
    const float zb = gr[h], za = gr[H + h] + dt_bias[h];
    const float softplus = fmaxf(za, 0.f) + log1pf(expf(-fabsf(za)));
    gr[h] = 1.0f / (1.0f + expf(-zb));
    gr[H + h] = expf(-expf(a_log[h]) * softplus);
  }
}

// segs[s] = {slot, first position, first row, rows}.  Thread per channel: the new state's entry i is the input of the
// portion's token len - (taps-1) + i, or, for a portion shorter than taps - 1, entry len + i of the old state.
template <typename T>
__global__ void __launch_bounds__(256) conv_state_update_kernel(const T* __restrict__ y, int ld, ConvCols cc, float* __restrict__ state,
                                                                const int* __restrict__ segs, int taps) {
  const int seg = blockIdx.y;
  const int slot = segs[4 * seg], row0 = segs[4 * seg + 2], len = segs[4 * seg + 3];
  const int C = cc.nq + cc.nk + cc.nv;
  const int c = blockIdx.x * 256 + threadIdx.x;
  if (c >= C) return;
  float* st = state + (size_t)slot * (taps - 1) * C;
  float keep[MAX_TAPS - 1];
#pragma unroll
  for (int i = 0; i < MAX_TAPS - 1; ++i) {
    if (i < taps - 1) {
      const int t = len - (taps - 1) + i;
      keep[i] = t >= 0 ? ldf(y + (size_t)(row0 + t) * ld + cc.col(c)) : st[(size_t)(len + i) * C + c];
    }
  }
#pragma unroll
  for (int i = 0; i < MAX_TAPS - 1; ++i)
    if (i < taps - 1) st[(size_t)i * C + c] = keep[i];
}

// ---------------------------------------------------------------------------------------------------- forget gates
// What turns the q | f | v columns of a projection's output (nq = H * dim channels of q and of f, nv of v) into the FORGET
// recurrence's fp32 inputs, row by row:  q = silu(q),  f = low + (1 - low) * sigmoid(f + f_bias)  (low: the gate's lower
// bound per channel),  v as it is;  out[row] = q | f | v.
template <typename T>
__global__ void forget_gate_prep_kernel(const T* __restrict__ y, int ld, int q_off, int f_off, int v_off, const float* __restrict__ f_bias,
                                        const float* __restrict__ low, float* __restrict__ out, int M, int nq, int nv) {
  const int C = 2 * nq + nv;
  const size_t n = (size_t)M * C;
  for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < n; e += (size_t)gridDim.x * blockDim.x) {
    const size_t m = e / C;
    const int c = (int)(e - m * C);
    const T* row = y + m * ld;
    float val;
    if (c < nq) {
      val = silu(ldf(row + q_off + c));
    } else if (c < 2 * nq) {
      const int i = c - nq;
      const float l = low[i];
      val = l + (1.0f - l) / (1.0f + expf(-(ldf(row + f_off + i) + (f_bias ? f_bias[i] : 0.f))));
    } else {
      val = ldf(row + v_off + (c - 2 * nq));
    }
    out[e] = val;
  }
}

// ---------------------------------------------------------------------------------------------------- the recurrence
// Stage loads return RAW bits and nothing touches them until they are stored to shared memory, so all loads of a stage are
// in flight together while the previous stage is processed.
template <typename T> struct Raw;
template <> struct Raw<float> {
  typedef float type;
  static __device__ __forceinline__ float ld(const float* p) {
    float v;
    asm volatile("ld.global.nc.f32 %0, [%1];" : "=f"(v) : "l"(p));
    return v;
  }
  static __device__ __forceinline__ float to_float(float v) { return v; }
};
template <> struct Raw<bf16> {
  typedef unsigned short type;
  static __device__ __forceinline__ unsigned short ld(const bf16* p) {
    unsigned short u;
    asm volatile("ld.global.nc.u16 %0, [%1];" : "=h"(u) : "l"(p));
    return u;
  }
  static __device__ __forceinline__ float to_float(unsigned short u) { return __uint_as_float((unsigned)u << 16); }
};

// 128-bit stage load (raw bits, same reasoning) and its unpacking into VEC floats
__device__ __forceinline__ uint4 ld_raw128(const void* p) {
  uint4 v;
  asm volatile("ld.global.nc.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}
template <typename T> struct Vec128;
template <> struct Vec128<float> {
  static constexpr int N = 4;
  static __device__ __forceinline__ void unpack(uint4 v, float* f) {
    f[0] = __uint_as_float(v.x); f[1] = __uint_as_float(v.y); f[2] = __uint_as_float(v.z); f[3] = __uint_as_float(v.w);
  }
};
template <> struct Vec128<bf16> {
  static constexpr int N = 8;
  static __device__ __forceinline__ void unpack(uint4 v, float* f) {
    f[0] = __uint_as_float(v.x << 16); f[1] = __uint_as_float(v.x & 0xffff0000u);
    f[2] = __uint_as_float(v.y << 16); f[3] = __uint_as_float(v.y & 0xffff0000u);
    f[4] = __uint_as_float(v.z << 16); f[5] = __uint_as_float(v.z & 0xffff0000u);
    f[6] = __uint_as_float(v.w << 16); f[7] = __uint_as_float(v.w & 0xffff0000u);
  }
};

constexpr int TB = 8;            // tokens per stage
constexpr int CW = 2;            // columns of S per warp
constexpr int NW = 8;            // warps per block
constexpr int CB = CW * NW;      // columns per block

// VL: the stage is fetched with 128-bit loads (the host checked that every q / k / v segment of VEC numbers starts on a
// 16-byte boundary and lies wholly inside or outside its row).
// MODE: 0 DECAY, 1 DELTA, 2 FORGET (the k slot of the stage carries f_t).
template <typename T, int DR, int MODE, bool VL>
__global__ void __launch_bounds__(NW * 32, 2) linear_scan_kernel(const T* __restrict__ q, const T* __restrict__ k, int ldqk, const T* __restrict__ v, int ldv,
                                                              int in_silu, const float* __restrict__ decay, const float* __restrict__ gates,
                                                              float* __restrict__ St, const int* __restrict__ segs, int H, int G, int dim, int vdim,
                                                              float* __restrict__ o) {
  constexpr bool DELTA = MODE == 1, FORGET = MODE == 2;
  constexpr int DP = DR * 32;                    // dim padded to whole warps
  constexpr int ROWF = 2 * DP + CB + 4;          // floats of one staged token: q | k | v (this block's columns) | beta | g | 2 pad
  constexpr int VEC = Vec128<T>::N;
  constexpr int CH = (2 * DP + CB) / VEC;        // 128-bit segments of one staged token
  constexpr int NST = VL ? (TB * CH + NW * 32 - 1) / (NW * 32) : (TB * ROWF + NW * 32 - 1) / (NW * 32);
  extern __shared__ __align__(16) float stage[]; // [2][TB][ROWF]
  const int seg = blockIdx.z, h = blockIdx.y, colb = blockIdx.x * CB;
  const int hk = h / (H / G);
  const int slot = segs[4 * seg], row0 = segs[4 * seg + 2], len = segs[4 * seg + 3];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int col0 = colb + warp * CW;

  float S[DR][CW];
  float* Sp = St + ((size_t)slot * H + h) * vdim * dim;
#pragma unroll
  for (int i = 0; i < DR; ++i) {
    const int r = lane + 32 * i;
#pragma unroll
    for (int c = 0; c < CW; ++c) S[i][c] = (r < dim && col0 + c < vdim) ? Sp[(size_t)(col0 + c) * dim + r] : 0.f;
  }
  const float dec = MODE == 0 ? decay[h] : 0.f;

  typename Raw<T>::type buf[VL ? 1 : NST];
  uint4 vbuf[VL ? NST : 1];
  float gbuf = 0.f;
  auto fetch = [&](int g) {
    if constexpr (VL) {
#pragma unroll
      for (int s = 0; s < NST; ++s) {
        const int e = threadIdx.x + s * NW * 32;
        const T* p = nullptr;
        if (e < TB * CH) {
          const int t = e / CH, j = (e - t * CH) * VEC;
          const int tok = g * TB + t;
          if (tok < len) {
            const size_t row = (size_t)(row0 + tok);
            if (j < DP) { if (j < dim) p = q + row * ldqk + hk * dim + j; }
            else if (j < 2 * DP) { if (j - DP < dim) p = k + row * ldqk + hk * dim + (j - DP); }
            else if (colb + j - 2 * DP < vdim) p = v + row * ldv + h * vdim + colb + (j - 2 * DP);
          }
        }
        vbuf[s] = make_uint4(0u, 0u, 0u, 0u);
        if (p != nullptr) vbuf[s] = ld_raw128(p);
      }
    } else {
#pragma unroll
    for (int s = 0; s < NST; ++s) {
      const int e = threadIdx.x + s * NW * 32;
      const T* p = nullptr;
      if (e < TB * ROWF) {
        const int t = e / ROWF, j = e - t * ROWF;
        const int tok = g * TB + t;
        if (tok < len) {
          const size_t row = (size_t)(row0 + tok);
          if (j < dim) p = q + row * ldqk + hk * dim + j;
          else if (j >= DP && j - DP < dim) p = k + row * ldqk + hk * dim + (j - DP);
          else if (j >= 2 * DP && j < 2 * DP + CB && colb + j - 2 * DP < vdim) p = v + row * ldv + h * vdim + colb + (j - 2 * DP);
        }
      }
      buf[s] = typename Raw<T>::type(0);
      if (p != nullptr) buf[s] = Raw<T>::ld(p);
    }
    }
    if (DELTA && threadIdx.x < 2 * TB) {
      const int tok = g * TB + (threadIdx.x >> 1);
      gbuf = 0.f;
      if (tok < len) gbuf = Raw<float>::ld(gates + (size_t)(row0 + tok) * 2 * H + (threadIdx.x & 1) * H + h);
    }
  };
  auto put = [&](int b) {
    if constexpr (VL) {
#pragma unroll
      for (int s = 0; s < NST; ++s) {
        const int e = threadIdx.x + s * NW * 32;
        if (e < TB * CH) {
          const int t = e / CH, j = (e - t * CH) * VEC;
          float f[VEC];
          Vec128<T>::unpack(vbuf[s], f);
          if (in_silu) {
#pragma unroll
            for (int i = 0; i < VEC; ++i) f[i] = silu(f[i]);
          }
          float* dst = stage + b * TB * ROWF + t * ROWF + j;
#pragma unroll
          for (int i = 0; i < VEC; i += 4) *reinterpret_cast<float4*>(dst + i) = make_float4(f[i], f[i + 1], f[i + 2], f[i + 3]);
        }
      }
    } else {
#pragma unroll
    for (int s = 0; s < NST; ++s) {
      const int e = threadIdx.x + s * NW * 32;
      if (e < TB * ROWF) {
        const int j = e % ROWF;
        if (j < 2 * DP + CB) {
          const float x = Raw<T>::to_float(buf[s]);
          stage[b * TB * ROWF + e] = in_silu ? silu(x) : x;
        }
      }
    }
    }
    if (DELTA && threadIdx.x < 2 * TB) stage[b * TB * ROWF + (threadIdx.x >> 1) * ROWF + 2 * DP + CB + (threadIdx.x & 1)] = gbuf;
  };

  const int groups = (len + TB - 1) / TB;
  fetch(0);
  put(0);
  __syncthreads();
  for (int g = 0; g < groups; ++g) {
    if (g + 1 < groups) fetch(g + 1);            // in flight while this group is processed
    const float* st = stage + (g & 1) * TB * ROWF;
    const int nt = min(TB, len - g * TB);
    for (int t = 0; t < nt; ++t) {
      const float* tk = st + t * ROWF;
      float vc[CW], out[CW];
#pragma unroll
      for (int c = 0; c < CW; ++c) vc[c] = tk[2 * DP + warp * CW + c];
      if constexpr (DELTA) {
        const float beta = tk[2 * DP + CB], gt = tk[2 * DP + CB + 1];
        float pk[CW], pq[CW], kq = 0.f;
#pragma unroll
        for (int c = 0; c < CW; ++c) pk[c] = pq[c] = 0.f;
#pragma unroll
        for (int i = 0; i < DR; ++i) {
          const float qv = tk[lane + 32 * i], kv = tk[DP + lane + 32 * i];
          kq = fmaf(kv, qv, kq);
#pragma unroll
          for (int c = 0; c < CW; ++c) {
            pk[c] = fmaf(S[i][c], kv, pk[c]);
            pq[c] = fmaf(S[i][c], qv, pq[c]);
          }
        }
        kq = warp_sum(kq);
        float u[CW];
#pragma unroll
        for (int c = 0; c < CW; ++c) {
          pk[c] = warp_sum(pk[c]);
          pq[c] = warp_sum(pq[c]);
          u[c] = beta * (vc[c] - gt * pk[c]);
          out[c] = fmaf(u[c], kq, gt * pq[c]);
        }
#pragma unroll
        for (int i = 0; i < DR; ++i) {
          const float kv = tk[DP + lane + 32 * i];
#pragma unroll
          for (int c = 0; c < CW; ++c) S[i][c] = fmaf(gt, S[i][c], kv * u[c]);
        }
      } else {
#pragma unroll
        for (int c = 0; c < CW; ++c) out[c] = 0.f;
#pragma unroll
        for (int i = 0; i < DR; ++i) {
          const float qv = tk[lane + 32 * i], kv = tk[DP + lane + 32 * i];
#pragma unroll
          for (int c = 0; c < CW; ++c) {
            if constexpr (FORGET) S[i][c] = fmaf(kv, S[i][c], (1.0f - kv) * vc[c]);     // kv is f_t here; padded rows stay unread
            else S[i][c] = fmaf(dec, S[i][c], kv * vc[c]);
            out[c] = fmaf(S[i][c], qv, out[c]);
          }
        }
#pragma unroll
        for (int c = 0; c < CW; ++c) out[c] = warp_sum(out[c]);
      }
      float mine = out[0];
#pragma unroll
      for (int c = 1; c < CW; ++c) mine = (lane == c) ? out[c] : mine;
      if (lane < CW && col0 + lane < vdim) o[(size_t)(row0 + g * TB + t) * H * vdim + h * vdim + col0 + lane] = mine;
    }
    if (g + 1 < groups) put((g + 1) & 1);        // the other buffer: last read two groups ago, before the barrier below
    __syncthreads();
  }

#pragma unroll
  for (int i = 0; i < DR; ++i) {
    const int r = lane + 32 * i;
    if (r < dim) {
#pragma unroll
      for (int c = 0; c < CW; ++c)
        if (col0 + c < vdim) Sp[(size_t)(col0 + c) * dim + r] = S[i][c];
    }
  }
}

template <typename T, int DR, int MODE, bool VL>
int launch_scan_mode(const void* q, const void* k, int ldqk, const void* v, int ldv, int in_silu, const float* decay, const float* gates, float* St,
                     const int* segs, int nseg, int H, int G, int dim, int vdim, float* o, cudaStream_t stream) {
  const size_t smem = (size_t)2 * TB * (2 * DR * 32 + CB + 4) * sizeof(float);
  dim3 grid((vdim + CB - 1) / CB, H, nseg);
  if (smem > 48 * 1024) LIA_CUDA(cudaFuncSetAttribute(linear_scan_kernel<T, DR, MODE, VL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  linear_scan_kernel<T, DR, MODE, VL><<<grid, NW * 32, smem, stream>>>(reinterpret_cast<const T*>(q), reinterpret_cast<const T*>(k), ldqk,
                                                                       reinterpret_cast<const T*>(v), ldv, in_silu, decay, gates, St, segs, H, G, dim, vdim, o);
  LIA_LAUNCH_CHECK();
  return LIA_OK;
}

// gates given: DELTA; decay given: DECAY; neither: FORGET
template <typename T, int DR, bool VL>
int launch_scan_as(const void* q, const void* k, int ldqk, const void* v, int ldv, int in_silu, const float* decay, const float* gates, float* St,
                   const int* segs, int nseg, int H, int G, int dim, int vdim, float* o, cudaStream_t stream) {
  if (gates != nullptr) return launch_scan_mode<T, DR, 1, VL>(q, k, ldqk, v, ldv, in_silu, decay, gates, St, segs, nseg, H, G, dim, vdim, o, stream);
  if (decay != nullptr) return launch_scan_mode<T, DR, 0, VL>(q, k, ldqk, v, ldv, in_silu, decay, gates, St, segs, nseg, H, G, dim, vdim, o, stream);
  return launch_scan_mode<T, DR, 2, VL>(q, k, ldqk, v, ldv, in_silu, decay, gates, St, segs, nseg, H, G, dim, vdim, o, stream);
}

template <typename T, int DR>
int launch_scan(const void* q, const void* k, int ldqk, const void* v, int ldv, int in_silu, const float* decay, const float* gates, float* St,
                const int* segs, int nseg, int H, int G, int dim, int vdim, float* o, cudaStream_t stream) {
  constexpr int VEC = Vec128<T>::N;
  const bool aligned = ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) % 16 == 0) &&
                       ldqk % VEC == 0 && ldv % VEC == 0 && dim % VEC == 0 && vdim % VEC == 0;
  if (aligned) return launch_scan_as<T, DR, true>(q, k, ldqk, v, ldv, in_silu, decay, gates, St, segs, nseg, H, G, dim, vdim, o, stream);
  return launch_scan_as<T, DR, false>(q, k, ldqk, v, ldv, in_silu, decay, gates, St, segs, nseg, H, G, dim, vdim, o, stream);
}

template <typename T>
int dispatch_scan(const void* q, const void* k, int ldqk, const void* v, int ldv, int in_silu, const float* decay, const float* gates, float* St,
                  const int* segs, int nseg, int H, int G, int dim, int vdim, float* o, cudaStream_t stream) {
  if (dim <= 32) return launch_scan<T, 1>(q, k, ldqk, v, ldv, in_silu, decay, gates, St, segs, nseg, H, G, dim, vdim, o, stream);
  if (dim <= 64) return launch_scan<T, 2>(q, k, ldqk, v, ldv, in_silu, decay, gates, St, segs, nseg, H, G, dim, vdim, o, stream);
  if (dim <= 128) return launch_scan<T, 4>(q, k, ldqk, v, ldv, in_silu, decay, gates, St, segs, nseg, H, G, dim, vdim, o, stream);
  if (dim <= 256) return launch_scan<T, 8>(q, k, ldqk, v, ldv, in_silu, decay, gates, St, segs, nseg, H, G, dim, vdim, o, stream);
  return launch_scan<T, 16>(q, k, ldqk, v, ldv, in_silu, decay, gates, St, segs, nseg, H, G, dim, vdim, o, stream);
}

// ---------------------------------------------------------------------------------------------------- convolution of one column range
// Thread per channel, walking down a strip of rows with the last taps - 1 inputs in registers.  Input = y[row][col0 + c] + in_bias[c] (zero,
// without the bias, before the sequence's start); out[row][c] = act(sum_j w[c][taps - 1 - j] * input j tokens back + bias[c]).
// state [slot][taps-1][C] holds the inputs before their bias.  single: every portion is one row, so the thread that reads a sequence's
// state is the only one that does and also moves it on.
// Threads C .. C + H - 1 (H > 0) make the recurrence's per-token numbers instead: gates[row] = dt | g with
// dt = softplus(y[row][dt_col + h] + dt_bias[h]),  g = exp(-exp(a_log[h]) dt).
struct ConvActArgs {
  int ld, col0, C, taps, act, single, ldo, M, strip;
  int dt_col, H;
};

constexpr int CONV_STRIP = 8;

__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.0f + expf(-z)); }
__device__ __forceinline__ float gelu_tanh(float z) { return 0.5f * z * (1.0f + tanhf(0.79788456080286535588f * (z + 0.044715f * z * z * z))); }

template <typename T, int TM>
__global__ void __launch_bounds__(256) conv_act_kernel(const T* __restrict__ y, const float* __restrict__ in_bias, const float* __restrict__ wconv,
                                                       const float* __restrict__ bias, float* __restrict__ state, const int* __restrict__ meta,
                                                       float* __restrict__ out, const float* __restrict__ dt_bias, const float* __restrict__ a_log,
                                                       float* __restrict__ gates, ConvActArgs a) {
  const int c = blockIdx.x * 256 + threadIdx.x;
  const int r0 = blockIdx.y * a.strip, r1 = min(a.M, r0 + a.strip);
  if (c >= a.C + a.H) return;
  if (c >= a.C) {
    const int h = c - a.C;
    const float rate = -expf(a_log[h]), b = dt_bias[h];
    for (int r = r0; r < r1; ++r) {
      const float z = ldf(y + (size_t)r * a.ld + a.dt_col + h) + b;
      const float dt = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
      gates[(size_t)r * 2 * a.H + h] = dt;
      gates[(size_t)r * 2 * a.H + a.H + h] = expf(rate * dt);
    }
    return;
  }
  const T* col = y + a.col0 + c;
  const float ib = in_bias ? in_bias[c] : 0.f, ob = bias ? bias[c] : 0.f;
  float w[TM], win[TM];                          // by tokens back
#pragma unroll
  for (int j = 0; j < TM; ++j) {
    w[j] = j < a.taps ? wconv[(size_t)c * a.taps + a.taps - 1 - j] : 0.f;
    win[j] = 0.f;
  }
  if (r1 - r0 == CONV_STRIP && r0 >= TM - 1) {
    // a whole strip in the middle of a portion: all its inputs are rows of y, fetched together
    const int slot = meta[2 * r0], pos = meta[2 * r0 + 1];
    if (meta[2 * (r1 - 1)] == slot && meta[2 * (r1 - 1) + 1] == pos + CONV_STRIP - 1 && meta[2 * (r0 - TM + 1)] == slot && meta[2 * (r0 - TM + 1) + 1] == pos - TM + 1) {
      float in[CONV_STRIP + TM - 1];
#pragma unroll
      for (int i = 0; i < CONV_STRIP + TM - 1; ++i) in[i] = ldf(col + (size_t)(r0 - TM + 1 + i) * a.ld);
#pragma unroll
      for (int i = 0; i < CONV_STRIP; ++i) {
        float acc = ob;
#pragma unroll
        for (int j = 0; j < TM; ++j) acc = fmaf(w[j], in[i + TM - 1 - j] + ib, acc);       // (weights beyond the taps are zero)
        if (a.act == LIA_ACT_SILU) acc = silu_fast(acc);
        out[(size_t)(r0 + i) * a.ldo + c] = acc;
      }
      return;
    }
  }
  int pslot = -1, ppos = -1;
  for (int r = r0; r < r1; ++r) {
    const int slot = meta[2 * r], pos = meta[2 * r + 1];
    float* st = state ? state + (size_t)slot * (a.taps - 1) * a.C + c : nullptr;
    if (r > r0 && slot == pslot && pos == ppos + 1) {
#pragma unroll
      for (int j = TM - 1; j > 0; --j) win[j] = win[j - 1];
    } else {
      int inside = 1;                            // rows r-1 .. r-(inside-1) belong to this portion
      while (inside < a.taps && r - inside >= 0 && meta[2 * (r - inside)] == slot && meta[2 * (r - inside) + 1] == pos - inside) ++inside;
#pragma unroll
      for (int j = 1; j < TM; ++j) {
        win[j] = 0.f;
        if (j < a.taps && j <= pos)
          win[j] = j < inside ? ldf(col + (size_t)(r - j) * a.ld) : st[(size_t)(inside - 1 - j + a.taps - 1) * a.C];
      }
    }
    win[0] = ldf(col + (size_t)r * a.ld);
    float acc = 0.f;
#pragma unroll
    for (int j = 0; j < TM; ++j)
      if (j < a.taps && j <= pos) acc = fmaf(w[j], win[j] + ib, acc);
    acc += ob;
    if (a.act == LIA_ACT_SILU) acc = silu_fast(acc);
    out[(size_t)r * a.ldo + c] = acc;
    if (a.single) {
#pragma unroll
      for (int j = 0; j < TM - 1; ++j)
        if (j < a.taps - 1) st[(size_t)(a.taps - 2 - j) * a.C] = win[j];
    }
    pslot = slot;
    ppos = pos;
  }
}

// ---------------------------------------------------------------------------------------------------- state-space duality
__device__ __forceinline__ void cp_async4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

constexpr int SSD_TB = 16;        // tokens per stage

// Block: 4 warps x 4 * 32 / RG columns of one head of one portion.  Lane: row group rg = lane % RG owns rows 4 RG j + 4 rg .. + 3 (j < NJ, N <= 4 RG NJ)
// of the four columns of column group lane / RG.  TG tokens exchange their sums together (the unrolled body of TG tokens must stay small
// enough for the instruction cache: there is one warp per scheduler to hide a miss).  Stages of SSD_TB tokens (B | C | x of this block's columns | dt | g) arrive by cp.async
// one stage ahead.
template <int NJ, int RG, int TG, bool VL>
__global__ void __launch_bounds__(128, TG > 1 ? 1 : (NJ <= 2 ? 5 : (NJ <= 4 ? 3 : 1))) ssd_scan_kernel(const float* __restrict__ B, const float* __restrict__ C, const float* __restrict__ x, int ld,
                                                       const float* __restrict__ gates, const float* __restrict__ D, float* __restrict__ St,
                                                       const int* __restrict__ segs, int H, int G, int N, int vdim, float* __restrict__ o) {
  constexpr int SSD_COLS = 4 * 4 * 32 / RG, NP = NJ * 4 * RG, ROWF = 2 * NP + SSD_COLS + 4;
  extern __shared__ __align__(16) float stage[];       // [2][SSD_TB][ROWF]
  const int seg = blockIdx.z, h = blockIdx.y, colb = blockIdx.x * SSD_COLS, g = h / (H / G);
  const int slot = segs[4 * seg], row0 = segs[4 * seg + 2], len = segs[4 * seg + 3];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, rg = lane % RG;
  const int cl = warp * (SSD_COLS / 4) + (lane / RG) * 4, col0 = colb + cl;
  const int ncol = min(SSD_COLS, vdim - colb);

  if (N < NP || ncol < SSD_COLS)                       // rows N .. NP-1 of B and C and the columns beyond vdim stay zero
    for (int i = threadIdx.x; i < min(2 * SSD_TB, len) * ROWF; i += 128) stage[i] = 0.f;
  float S[4][NJ * 4];
#pragma unroll
  for (int c = 0; c < 4; ++c) {
    const float* Sp = St + (((size_t)slot * H + h) * vdim + col0 + c) * N;
    const bool live = col0 + c < vdim;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int r = 4 * RG * j + 4 * rg;
      if (VL) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (live && r < N) v = *reinterpret_cast<const float4*>(Sp + r);
        S[c][4 * j] = v.x; S[c][4 * j + 1] = v.y; S[c][4 * j + 2] = v.z; S[c][4 * j + 3] = v.w;
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) S[c][4 * j + e] = (live && r + e < N) ? Sp[r + e] : 0.f;
      }
    }
  }
  __syncthreads();

  constexpr int U = VL ? 4 : 1;                        // floats per copy
  constexpr int SLOTS = (SSD_TB * (2 * NP + SSD_COLS) / 4 + 127) / 128;            // copies of 4 floats per thread and stage
  const int n_u = N / U, x_u = ncol / U, per_tok = 2 * n_u + x_u;
  // copy e of a stage: token e / per_tok, then B | C | x in order
  auto place = [&](int e, int& t, size_t& src, int& which, int& dst) {
    t = e / per_tok;
    const int j = e - t * per_tok;
    which = j < n_u ? 0 : (j < 2 * n_u ? 1 : 2);
    const int k = (j - which * n_u) * U;
    src = (size_t)(row0 + t) * ld + (which == 2 ? h * vdim + colb : g * N) + k;
    dst = t * ROWF + which * NP + k;
  };
  const float* slot_src[VL ? SLOTS : 1];               // the copies of this thread, moved on stage by stage
  int slot_dst[VL ? SLOTS : 1];
  if constexpr (VL) {
#pragma unroll
    for (int i = 0; i < SLOTS; ++i) {
      int t, which;
      size_t src;
      place(threadIdx.x + i * 128, t, src, which, slot_dst[i]);
      slot_src[i] = (which == 0 ? B : (which == 1 ? C : x)) + src;
      if (t >= SSD_TB) slot_dst[i] = -1;
    }
  }
  auto fetch = [&](int gidx) {
    const int t0 = gidx * SSD_TB, nt = min(SSD_TB, len - t0);
    float* st = stage + (gidx & 1) * SSD_TB * ROWF;
    if constexpr (VL) {
#pragma unroll
      for (int i = 0; i < SLOTS; ++i) {
        if (slot_dst[i] >= 0 && slot_dst[i] < nt * ROWF) cp_async16(st + slot_dst[i], slot_src[i]);
        slot_src[i] += (size_t)SSD_TB * ld;
      }
    } else {
      for (int e = threadIdx.x; e < nt * per_tok; e += 128) {
        int t, which, dst;
        size_t src;
        place(e, t, src, which, dst);
        cp_async4(st + dst, (which == 0 ? B : (which == 1 ? C : x)) + src + (size_t)t0 * ld);
      }
    }
    if (threadIdx.x < 2 * nt) {
      const int t = threadIdx.x >> 1, which = threadIdx.x & 1;
      cp_async4(st + t * ROWF + 2 * NP + SSD_COLS + which, gates + (size_t)(row0 + t0 + t) * 2 * H + which * H + h);
    }
  };
  // one token: the state moves on; s = this thread's part of the four columns' sums
  auto token = [&](const float* tk, float4 xv, float* s) {
    const float2 dg = *reinterpret_cast<const float2*>(tk + 2 * NP + SSD_COLS);
    const float u[4] = {dg.x * xv.x, dg.x * xv.y, dg.x * xv.z, dg.x * xv.w};
    float hi[4];
#pragma unroll
    for (int c = 0; c < 4; ++c) s[c] = hi[c] = 0.f;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const float4 k = *reinterpret_cast<const float4*>(tk + 4 * RG * j + 4 * rg);
      const float4 q = *reinterpret_cast<const float4*>(tk + NP + 4 * RG * j + 4 * rg);
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        float* Sc = S[c] + 4 * j;
        Sc[0] = fmaf(dg.y, Sc[0], k.x * u[c]);
        Sc[1] = fmaf(dg.y, Sc[1], k.y * u[c]);
        Sc[2] = fmaf(dg.y, Sc[2], k.z * u[c]);
        Sc[3] = fmaf(dg.y, Sc[3], k.w * u[c]);
        s[c] = fmaf(Sc[1], q.y, fmaf(Sc[0], q.x, s[c]));
        hi[c] = fmaf(Sc[3], q.w, fmaf(Sc[2], q.z, hi[c]));
      }
    }
#pragma unroll
    for (int c = 0; c < 4; ++c) s[c] += hi[c];
  };
  const float dh = D[h];
  const int groups = (len + SSD_TB - 1) / SSD_TB;
  fetch(0);
  cp_async_commit();
  for (int gi = 0; gi < groups; ++gi) {
    if (gi + 1 < groups) fetch(gi + 1);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const float* st = stage + (gi & 1) * SSD_TB * ROWF;
    const int nt = min(SSD_TB, len - gi * SSD_TB);
    float* orow = o + (size_t)(row0 + gi * SSD_TB) * H * vdim + (size_t)h * vdim + colb;
    // lane rg ends with the sums e, e + 1, .. of n: every exchange of the loop halves what a lane holds until one is left
    auto exchange = [&](float* s, int n) {
#pragma unroll
      for (int w = RG / 2; w > 0; w >>= 1) {
        n >>= 1;
        const bool up = rg & w;
#pragma unroll
        for (int i = 0; i < n; ++i) {
          const float keep = up ? s[i + n] : s[i], give = up ? s[i] : s[i + n];
          s[i] = keep + __shfl_xor_sync(0xffffffffu, give, w);
        }
        if (n == 0) s[0] += __shfl_xor_sync(0xffffffffu, s[0], w);
      }
    };
    auto put = [&](int t, int c, float sum) {
      if (c < ncol) orow[(size_t)t * H * vdim + c] = fmaf(dh, st[t * ROWF + 2 * NP + c], sum);
    };
    int t0 = 0;
#pragma unroll 1
    for (; t0 + TG <= nt; t0 += TG) {
      float s[TG * 4];
#pragma unroll
      for (int t = 0; t < TG; ++t) token(st + (t0 + t) * ROWF, *reinterpret_cast<const float4*>(st + (t0 + t) * ROWF + 2 * NP + cl), s + 4 * t);
      exchange(s, TG * 4);
      constexpr int PER = TG * 4 / RG > 0 ? TG * 4 / RG : 1, REP = RG / (TG * 4) > 0 ? RG / (TG * 4) : 1;     // sums per lane, lanes per sum
#pragma unroll
      for (int i = 0; i < PER; ++i) {
        const int e = rg / REP * PER + i;
        if (rg % REP == 0) put(t0 + e / 4, cl + e % 4, s[i]);
      }
    }
#pragma unroll 1
    for (; t0 < nt; ++t0) {
      float s[4];
      token(st + t0 * ROWF, *reinterpret_cast<const float4*>(st + t0 * ROWF + 2 * NP + cl), s);
      exchange(s, 4);
      if (rg % (RG / 4) == 0) put(t0, cl + rg / (RG / 4), s[0]);
    }
    __syncthreads();                                   // the stage after next goes where this one was
  }
#pragma unroll
  for (int c = 0; c < 4; ++c) {
    if (col0 + c >= vdim) continue;
    float* Sp = St + (((size_t)slot * H + h) * vdim + col0 + c) * N;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int r = 4 * RG * j + 4 * rg;
      if (VL) {
        if (r < N) *reinterpret_cast<float4*>(Sp + r) = make_float4(S[c][4 * j], S[c][4 * j + 1], S[c][4 * j + 2], S[c][4 * j + 3]);
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (r + e < N) Sp[r + e] = S[c][4 * j + e];
      }
    }
  }
}

template <int NJ, int RG, int TG, bool VL>
int launch_ssd_as(const float* B, const float* C, const float* x, int ld, const float* gates, const float* D, float* St, const int* segs, int nseg, int H,
                  int G, int N, int vdim, float* o, cudaStream_t stream) {
  constexpr int COLS = 16 * 32 / RG;
  const size_t smem = (size_t)2 * SSD_TB * (2 * NJ * 4 * RG + COLS + 4) * sizeof(float);
  if (smem > 48 * 1024) LIA_CUDA(cudaFuncSetAttribute(ssd_scan_kernel<NJ, RG, TG, VL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  dim3 grid((vdim + COLS - 1) / COLS, H, nseg);
  ssd_scan_kernel<NJ, RG, TG, VL><<<grid, 128, smem, stream>>>(B, C, x, ld, gates, D, St, segs, H, G, N, vdim, o);
  LIA_LAUNCH_CHECK();
  return LIA_OK;
}

// 128-bit copies and state accesses: every B, C, x segment and every state column starts on a 16-byte boundary
// single: every portion is one token (decoding) -- the variant without token groups needs fewer registers, so more blocks share an SM
template <int NJ, int RG, int TG>
int launch_ssd(bool single, const float* B, const float* C, const float* x, int ld, const float* gates, const float* D, float* St, const int* segs,
               int nseg, int H, int G, int N, int vdim, float* o, cudaStream_t stream) {
  const bool aligned = ((reinterpret_cast<uintptr_t>(B) | reinterpret_cast<uintptr_t>(C) | reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(St)) % 16 == 0) &&
                       ld % 4 == 0 && N % 4 == 0 && vdim % 4 == 0;
  if (aligned && single) return launch_ssd_as<NJ, RG, 1, true>(B, C, x, ld, gates, D, St, segs, nseg, H, G, N, vdim, o, stream);
  if (aligned) return launch_ssd_as<NJ, RG, TG, true>(B, C, x, ld, gates, D, St, segs, nseg, H, G, N, vdim, o, stream);
  return launch_ssd_as<NJ, RG, TG, false>(B, C, x, ld, gates, D, St, segs, nseg, H, G, N, vdim, o, stream);
}

// ---------------------------------------------------------------------------------------------------- gated linear recurrent unit
constexpr int LRU_T = 4, LRU_CH = 16;          // tokens per thread and sweep, channels per block

__device__ __forceinline__ float sigmoid_fast(float z) { return __fdividef(1.0f, 1.0f + expf(-z)); }

// Block: 16 channels of one portion, LRU_W warps (16; 1 in a step of single tokens); a half-warp takes LRU_T consecutive tokens of a sweep.  z [rows][blocks][2 n] holds every channel block's gate
// projections r | i (n = width / blocks), z_bias [blocks][2 n] their biases, c[ch] = -8 softplus(lam): log a = c sigmoid(r).
template <typename T, int LRU_W>
__global__ void __launch_bounds__(LRU_W * 32) rglru_scan_kernel(const float* __restrict__ u, const float* __restrict__ z, const float* __restrict__ z_bias,
                                                                const float* __restrict__ c, const T* __restrict__ y, int ldy, const float* __restrict__ y_bias,
                                                                float* __restrict__ St, const int* __restrict__ segs, int width, int n, T* __restrict__ out) {
  constexpr int SWEEP = LRU_W * 2 * LRU_T;
  __shared__ float2 maps[2][LRU_W][LRU_CH];   // a warp's eight tokens as S -> x S + y
  const int seg = blockIdx.y, slot = segs[4 * seg], row0 = segs[4 * seg + 2], len = segs[4 * seg + 3];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, cl = lane & (LRU_CH - 1), ch = blockIdx.x * LRU_CH + cl;
  const bool upper = lane >= LRU_CH;
  const int first = (threadIdx.x / LRU_CH) * LRU_T;
  const bool live = ch < width;
  const int blk = live ? ch / n : 0, zc = blk * 2 * n + (live ? ch - blk * n : 0);
  const float cc = live ? c[ch] : 0.f, rb = live ? z_bias[zc] : 0.f, ib = live ? z_bias[zc + n] : 0.f, yb = (live && y_bias) ? y_bias[ch] : 0.f;
  float S = live ? St[(size_t)slot * width + ch] : 0.f;
  float ur[LRU_T], zr[LRU_T], zi[LRU_T], yr[LRU_T];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int k = 0; k < LRU_T; ++k) {
      const int t = t0 + first + k;
      ur[k] = zr[k] = zi[k] = yr[k] = 0.f;
      if (live && t < len) {
        const size_t row = (size_t)(row0 + t);
        ur[k] = u[row * width + ch];
        zr[k] = z[row * 2 * width + zc];
        zi[k] = z[row * 2 * width + zc + n];
        yr[k] = ldf(y + row * ldy + ch);
      }
    }
  };
  fetch(0);
  int buf = 0;
  for (int t0 = 0; t0 < len; t0 += SWEEP) {
    float a[LRU_T], b[LRU_T], g[LRU_T], pa = 1.f, pb = 0.f;
#pragma unroll
    for (int k = 0; k < LRU_T; ++k) {
      a[k] = 1.f;
      b[k] = g[k] = 0.f;
      if (t0 + first + k < len) {
        const float la = cc * sigmoid_fast(zr[k] + rb);
        a[k] = expf(la);
        b[k] = sqrtf(-expm1f(2.0f * la)) * ur[k] * sigmoid_fast(zi[k] + ib);
        g[k] = gelu_tanh(yr[k] + yb);
      }
      pa *= a[k];
      pb = fmaf(a[k], pb, b[k]);
    }
    const float la = __shfl_sync(0xffffffffu, pa, cl), lb = __shfl_sync(0xffffffffu, pb, cl);      // the lower half's map
    if (upper) maps[buf][warp][cl] = make_float2(pa * la, fmaf(pa, lb, pb));
    if (t0 + SWEEP < len) fetch(t0 + SWEEP);
    __syncthreads();
    float s = S;
#pragma unroll
    for (int w = 0; w < LRU_W; ++w) {
      if (w == warp) s = S;
      const float2 m = maps[buf][w][cl];
      S = fmaf(m.x, S, m.y);
    }
    if (upper) s = fmaf(la, s, lb);
#pragma unroll
    for (int k = 0; k < LRU_T; ++k) {
      const int t = t0 + first + k;
      s = fmaf(a[k], s, b[k]);
      if (live && t < len) out[(size_t)(row0 + t) * width + ch] = T(s * g[k]);
    }
    buf ^= 1;                                 // the other half: last read before the barrier above
  }
  if (threadIdx.x < LRU_CH && live) St[(size_t)slot * width + ch] = S;
}

}  // namespace

extern "C" int lia_conv_prep(const void* y, int y_f32, int ld, int q_off, int k_off, int v_off, const float* wconv, const float* conv_state,
                             const int* meta, float* gates, const float* a_log, const float* dt_bias, float* qk, float* v, int M, int G, int H,
                             int dim, int vdim, int taps, float q_scale, float unit_eps, lia_stream_t stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LIA_CHECK_ARG(y && wconv && conv_state && meta && gates && a_log && dt_bias && qk && v, "lia_conv_prep: null pointer");
  LIA_CHECK_ARG(M > 0 && G > 0 && H > 0 && H % G == 0 && dim > 0 && vdim > 0 && taps >= 1 && taps <= MAX_TAPS, "lia_conv_prep: bad shape G=%d H=%d dim=%d vdim=%d taps=%d", G, H, dim, vdim, taps);
  ConvCols cc{q_off, k_off, v_off, G * dim, G * dim, H * vdim};
  const size_t smem = (size_t)(cc.nq + cc.nk + cc.nv) * sizeof(float);
  LIA_CHECK_ARG(smem <= 160 * 1024, "lia_conv_prep: %d channels do not fit shared memory", cc.nq + cc.nk + cc.nv);
  if (y_f32) {
    if (smem > 48 * 1024) LIA_CUDA(cudaFuncSetAttribute(conv_prep_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    conv_prep_kernel<float><<<M, 256, smem, stream>>>(reinterpret_cast<const float*>(y), ld, cc, wconv, conv_state, meta, gates, a_log, dt_bias, qk, v, G, H, dim, vdim, taps, q_scale, unit_eps);
  } else {
    if (smem > 48 * 1024) LIA_CUDA(cudaFuncSetAttribute(conv_prep_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    conv_prep_kernel<bf16><<<M, 256, smem, stream>>>(reinterpret_cast<const bf16*>(y), ld, cc, wconv, conv_state, meta, gates, a_log, dt_bias, qk, v, G, H, dim, vdim, taps, q_scale, unit_eps);
  }
  LIA_LAUNCH_CHECK();
  return LIA_OK;
}

extern "C" int lia_conv_state_update(const void* y, int y_f32, int ld, int q_off, int k_off, int v_off, int nq, int nk, int nv, float* conv_state,
                                     const int* segs, int nseg, int taps, lia_stream_t stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LIA_CHECK_ARG(y && conv_state && segs && nseg > 0 && nseg <= 65535 && nq > 0 && nk > 0 && nv > 0 && taps >= 1 && taps <= MAX_TAPS, "lia_conv_state_update: bad arguments");
  if (taps == 1) return LIA_OK;
  ConvCols cc{q_off, k_off, v_off, nq, nk, nv};
  dim3 grid((nq + nk + nv + 255) / 256, nseg);
  if (y_f32) conv_state_update_kernel<float><<<grid, 256, 0, stream>>>(reinterpret_cast<const float*>(y), ld, cc, conv_state, segs, taps);
  else conv_state_update_kernel<bf16><<<grid, 256, 0, stream>>>(reinterpret_cast<const bf16*>(y), ld, cc, conv_state, segs, taps);
  LIA_LAUNCH_CHECK();
  return LIA_OK;
}

// gates == NULL: the DECAY recurrence with decay[H]; otherwise DELTA with gates[rows][2H] = beta | g.
extern "C" int lia_linear_scan(const void* q, const void* k, int ldqk, const void* v, int ldv, int act_f32, int in_silu, const float* decay,
                               const float* gates, float* state_S, const int* segs, int nseg, int H, int G, int dim, int vdim, float* o,
                               lia_stream_t stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LIA_CHECK_ARG(q && k && v && state_S && segs && o && (decay || gates), "lia_linear_scan: null pointer");
  LIA_CHECK_ARG(nseg > 0 && nseg <= 65535 && H > 0 && H <= 65535 && G > 0 && H % G == 0 && dim > 0 && dim <= 512 && vdim > 0,
                "lia_linear_scan: bad shape nseg=%d H=%d G=%d dim=%d vdim=%d", nseg, H, G, dim, vdim);
  if (act_f32) return dispatch_scan<float>(q, k, ldqk, v, ldv, in_silu, decay, gates, state_S, segs, nseg, H, G, dim, vdim, o, stream);
  return dispatch_scan<bf16>(q, k, ldqk, v, ldv, in_silu, decay, gates, state_S, segs, nseg, H, G, dim, vdim, o, stream);
}

extern "C" int lia_forget_gate_prep(const void* y, int y_f32, int ld, int q_off, int f_off, int v_off, const float* f_bias, const float* low,
                                    float* out, int M, int nq, int nv, lia_stream_t stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LIA_CHECK_ARG(y && low && out && M > 0 && nq > 0 && nv > 0 && ld >= nq && q_off >= 0 && f_off >= 0 && v_off >= 0, "lia_forget_gate_prep: bad arguments");
  const size_t n = (size_t)M * (2 * nq + nv);
  size_t blocks = (n + 255) / 256;
  const size_t capb = (size_t)lia_sm_count() * 16;
  if (blocks > capb) blocks = capb;
  if (y_f32) forget_gate_prep_kernel<float><<<(unsigned)blocks, 256, 0, stream>>>(reinterpret_cast<const float*>(y), ld, q_off, f_off, v_off, f_bias, low, out, M, nq, nv);
  else forget_gate_prep_kernel<bf16><<<(unsigned)blocks, 256, 0, stream>>>(reinterpret_cast<const bf16*>(y), ld, q_off, f_off, v_off, f_bias, low, out, M, nq, nv);
  LIA_LAUNCH_CHECK();
  return LIA_OK;
}

// The FORGET recurrence: q, f fp32 column slices with one row stride (H heads of dim), v fp32 (H heads of vdim).
extern "C" int lia_forget_scan(const float* q, const float* f, int ldqf, const float* v, int ldv, float* state_S, const int* segs, int nseg, int H,
                               int dim, int vdim, float* o, lia_stream_t stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LIA_CHECK_ARG(q && f && v && state_S && segs && o, "lia_forget_scan: null pointer");
  LIA_CHECK_ARG(nseg > 0 && nseg <= 65535 && H > 0 && H <= 65535 && dim > 0 && dim <= 512 && vdim > 0,
                "lia_forget_scan: bad shape nseg=%d H=%d dim=%d vdim=%d", nseg, H, dim, vdim);
  return dispatch_scan<float>(q, f, ldqf, v, ldv, 0, nullptr, nullptr, state_S, segs, nseg, H, H, dim, vdim, o, stream);
}

/* see lia_b200.h */
extern "C" int lia_conv_act(const void* y, int y_f32, int ld, int col0, int C, const float* in_bias, const float* wconv, const float* bias, int taps,
                            int act, float* state, const int* meta, const int* segs, int nseg, float* out, int ldo, int M, int dt_col, int H,
                            const float* dt_bias, const float* a_log, float* gates, lia_stream_t stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LIA_CHECK_ARG(y && wconv && meta && segs && out && M > 0 && C > 0 && nseg > 0 && nseg <= 65535 && nseg <= M, "lia_conv_act: bad arguments");
  LIA_CHECK_ARG(taps >= 1 && taps <= MAX_TAPS && (taps == 1 || state) && ldo >= C && ld >= col0 + C && col0 >= 0, "lia_conv_act: bad shape C=%d taps=%d", C, taps);
  LIA_CHECK_ARG(act == LIA_ACT_NONE || act == LIA_ACT_SILU, "lia_conv_act: unknown activation %d", act);
  LIA_CHECK_ARG(H >= 0 && (H == 0 || (dt_bias && a_log && gates && dt_col >= 0 && ld >= dt_col + H)), "lia_conv_act: bad step sizes (H=%d)", H);
  const int single = nseg == M && taps > 1;      // every portion is one row
  ConvActArgs a{ld, col0, C, taps, act, single, ldo, M, M <= 64 ? 1 : CONV_STRIP, dt_col, H};
  dim3 grid((C + H + 255) / 256, (M + a.strip - 1) / a.strip);
  LIA_CHECK_ARG(grid.y <= 65535, "lia_conv_act: too many rows (%d)", M);
#define LIA_CA(T, TM) conv_act_kernel<T, TM><<<grid, 256, 0, stream>>>(reinterpret_cast<const T*>(y), in_bias, wconv, bias, state, meta, out, dt_bias, a_log, gates, a)
  if (y_f32) {
    if (taps <= 4) LIA_CA(float, 4);
    else LIA_CA(float, MAX_TAPS);
  } else {
    if (taps <= 4) LIA_CA(bf16, 4);
    else LIA_CA(bf16, MAX_TAPS);
  }
#undef LIA_CA
  LIA_LAUNCH_CHECK();
  if (taps > 1 && !single) {
    ConvCols cc{col0, 0, 0, C, 0, 0};
    dim3 g2((C + 255) / 256, nseg);
    if (y_f32) conv_state_update_kernel<float><<<g2, 256, 0, stream>>>(reinterpret_cast<const float*>(y), ld, cc, state, segs, taps);
    else conv_state_update_kernel<bf16><<<g2, 256, 0, stream>>>(reinterpret_cast<const bf16*>(y), ld, cc, state, segs, taps);
    LIA_LAUNCH_CHECK();
  }
  return LIA_OK;
}

extern "C" int lia_ssd_scan(const float* B, const float* C, const float* x, int ld, const float* gates, const float* D, float* state_S, const int* segs,
                            int nseg, int rows, int H, int G, int N, int vdim, float* o, lia_stream_t stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  const bool single = rows == nseg;
  LIA_CHECK_ARG(rows >= nseg, "lia_ssd_scan: fewer rows (%d) than portions (%d)", rows, nseg);
  LIA_CHECK_ARG(B && C && x && gates && D && state_S && segs && o, "lia_ssd_scan: null pointer");
  LIA_CHECK_ARG(nseg > 0 && nseg <= 65535 && H > 0 && H <= 65535 && G > 0 && H % G == 0 && N > 0 && N <= 512 && vdim > 0,
                "lia_ssd_scan: bad shape nseg=%d H=%d G=%d N=%d vdim=%d", nseg, H, G, N, vdim);
  if (N <= 64) return launch_ssd<1, 16, 8>(single, B, C, x, ld, gates, D, state_S, segs, nseg, H, G, N, vdim, o, stream);
  if (N <= 128) return launch_ssd<2, 16, 4>(single, B, C, x, ld, gates, D, state_S, segs, nseg, H, G, N, vdim, o, stream);
  if (N <= 256) return launch_ssd<4, 16, 2>(single, B, C, x, ld, gates, D, state_S, segs, nseg, H, G, N, vdim, o, stream);
  return launch_ssd<8, 16, 1>(single, B, C, x, ld, gates, D, state_S, segs, nseg, H, G, N, vdim, o, stream);
}

extern "C" int lia_rglru_scan(const float* u, const float* z, const float* z_bias, const float* c, const void* y, int y_f32, int ldy, const float* y_bias,
                              float* state, const int* segs, int nseg, int rows, int width, int blocks, void* out, lia_stream_t stream_) {
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  LIA_CHECK_ARG(u && z && z_bias && c && y && state && segs && out, "lia_rglru_scan: null pointer");
  LIA_CHECK_ARG(nseg > 0 && nseg <= 65535 && rows >= nseg && width > 0 && blocks > 0 && width % blocks == 0 && ldy >= width, "lia_rglru_scan: bad shape width=%d blocks=%d", width, blocks);
  dim3 grid((width + LRU_CH - 1) / LRU_CH, nseg);
#define LIA_RS(T, W_) rglru_scan_kernel<T, W_><<<grid, W_ * 32, 0, stream>>>(u, z, z_bias, c, reinterpret_cast<const T*>(y), ldy, y_bias, state, segs, width, width / blocks, reinterpret_cast<T*>(out))
  if (y_f32 && rows == nseg) LIA_RS(float, 1);
  else if (y_f32) LIA_RS(float, 16);
  else if (rows == nseg) LIA_RS(bf16, 1);
  else LIA_RS(bf16, 16);
#undef LIA_RS
  LIA_LAUNCH_CHECK();
  return LIA_OK;
}
