// HGRN2 linear attention between its projections.  Per head, with state S ∈ R^{dim × vdim} in fp32:
//
//   q = silu(q_raw),  k = (1 − lower) σ(−(f_raw + bias)) = 1 − forget gate,  S ← S + k ⊙ (v − S)  (rows by k),  o = Sᵀ q,
//   output = o / rms(o) · weight                                        (rms over the head's vdim)
//
// Forming k instead of the forget gate keeps the digits of gates close to one, and the update above needs no decay beside it.
//
//   hgrn2_prefill  packed prompts; a block owns one head of one sequence (or of one time segment of it), the state is in registers.
//     bf16: sixteen tokens per step on the tensor cores (``hgrn2_chunk_kernel``).  With P_t the product of the forget gates from
//           the step's start through t, R_j the product behind j, and D the whole step's:
//               o_t = Σ_{j ≤ t} A_tj v_j + Sᵀ (q_t P_t),   A_tj = Σ_d q_td k_jd Π_{j < s ≤ t} f_sd,   S ← D S + Σ_j (k_j R_j) v_jᵀ
//           Only products of gates occur, never a quotient or a logarithm, so nothing overflows however fast a channel forgets.
//           Operands that are not bf16 already (state, q P, k R, A) go in as a bf16 value plus the bf16 of what it left over:
//           products keep 16 bits and more, sums are fp32, and the state itself is never rounded.
//     else: token by token in fp32 (``hgrn2_prefill_kernel``): RS neighbouring lanes share two columns, each with RPT of the rows, so a
//           token costs three operations per state element, two 16-byte shared-memory broadcasts per twelve of them and a shuffle
//           per column.
//     Tokens are brought in by asynchronous copies while those before are worked on.  When sequences × heads do not fill the
//     device, sequences are cut into time segments: a first pass forms each segment's own contribution and decay, a scan over
//     segments gives every segment its starting state.
//   hgrn2_step     one token of every sequence: the state passes once through the block, 16 bytes per access.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/types.h>

#include "common.cuh"
#include "host.h"
#include "mma16.cuh"

namespace tk {

using bf16 = __nv_bfloat16;
using OptT = c10::optional<torch::Tensor>;

namespace hg {
constexpr int CH = 16;          // tokens per round

__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(bf16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float silu(float z) { return z / (1.f + __expf(-z)); }
__device__ __forceinline__ float let_in(float z, float low) { return (1.f - low) / (1.f + __expf(z)); }
}  // namespace hg

template <typename T>
struct Hgrn2 {
  const T *q, *f, *v;              // column ranges of the projection, row stride ld
  long ld;
  const T *bias, *lower, *weight;  // [H·dim], [H·dim], [vdim]
  T* o;                            // [rows, H·vdim]
  float* raw;                      // [rows, H·vdim]: outputs before their norm, when a block does not hold a whole head
  const int* cu;                   // [n+1]
  float* pool;                     // [slots, H, dim, vdim] (null: last states are not kept)
  const int* slot;                 // [rows]
  float *part, *decay;             // [n, segments − 1, H, dim, vdim], [n, segments − 1, H, dim]
  int H, dim, vdim, seg_len, segments, slices, cols;
  float eps;
};

// PART: only the state a segment builds up from nothing and its decay; otherwise outputs.
template <typename T, int RPT, int RS, bool VEC, bool PART>
__global__ void __launch_bounds__(256) hgrn2_prefill_kernel(const Hgrn2<T> p) {
  using namespace hg;
  extern __shared__ __align__(16) uint8_t sm_raw[];
  constexpr int DP = RPT * RS;
  const int head = blockIdx.x / p.slices, slice = blockIdx.x - head * p.slices, seg = blockIdx.y, seq = blockIdx.z;
  const int s0 = p.cu[seq], len = p.cu[seq + 1] - s0;
  const int a = seg * p.seg_len, b = min(len, a + p.seg_len);
  if (a >= len || (PART && b >= len)) return;         // the last segment of a sequence is nobody's past
  const int col0 = slice * p.cols, ncol = min(p.cols, p.vdim - col0);
  const int VP = p.cols;
  float* s_q = reinterpret_cast<float*>(sm_raw);      // [CH][DP]
  float* s_k = s_q + CH * DP;                         // [CH][DP]
  float* s_v = s_k + CH * DP;                         // [CH][VP]: values, then outputs
  float* s_low = s_v + CH * VP;                       // [DP] lower bound, [DP] bias
  float* s_bias = s_low + DP;
  T* r_q = reinterpret_cast<T*>(s_bias + DP);         // the next tokens as they lie in memory: [CH][dim], [CH][dim], [CH][ncol]
  T* r_f = r_q + CH * p.dim;
  T* r_v = r_f + CH * p.dim;
  const int tid = threadIdx.x, rs = tid % RS, c0 = tid / RS * 2;
  const bool mine = c0 < ncol, two = c0 + 1 < ncol;
  for (int i = tid; i < DP; i += blockDim.x) {
    s_low[i] = i < p.dim ? ld(p.lower + static_cast<size_t>(head) * p.dim + i) : 1.f;
    s_bias[i] = i < p.dim ? ld(p.bias + static_cast<size_t>(head) * p.dim + i) : 0.f;
  }
  for (int i = tid; i < CH * DP; i += blockDim.x) {   // rows that fill up the head's width stay zero
    s_q[i] = 0.f;
    s_k[i] = 0.f;
  }
  const T* gq = p.q + static_cast<size_t>(s0) * p.ld + static_cast<size_t>(head) * p.dim;
  const T* gf = p.f + static_cast<size_t>(s0) * p.ld + static_cast<size_t>(head) * p.dim;
  const T* gv = p.v + static_cast<size_t>(s0) * p.ld + static_cast<size_t>(head) * p.vdim + col0;
  auto fetch = [&](int t0) {
    if constexpr (VEC) {
      constexpr int E = 16 / sizeof(T);
      const int n = min(CH, b - t0), dv = p.dim / E, vv = ncol / E;
      for (int i = tid; i < n * dv; i += blockDim.x) {
        const int t = i / dv, c = (i - t * dv) * E;
        const size_t g = static_cast<size_t>(t0 + t) * p.ld + c;
        if constexpr (!PART) copy16(r_q + t * p.dim + c, gq + g);
        copy16(r_f + t * p.dim + c, gf + g);
      }
      for (int i = tid; i < n * vv; i += blockDim.x) {
        const int t = i / vv, c = (i - t * vv) * E;
        copy16(r_v + t * ncol + c, gv + static_cast<size_t>(t0 + t) * p.ld + c);
      }
      copies_commit();
    }
  };
  float S0[RPT], S1[RPT];
  const size_t head_state = static_cast<size_t>(p.dim) * p.vdim;
  // row of register i: RS lanes take turns in groups of four
  auto row_of = [&](int i) { return ((i >> 2) * RS + rs) * 4 + (i & 3); };
  {
    const float* init = (!PART && seg > 0) ? p.part + ((static_cast<size_t>(seq) * (p.segments - 1) + seg - 1) * p.H + head) * head_state + col0 : nullptr;
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int r = row_of(i);
      S0[i] = init != nullptr && mine && r < p.dim ? init[static_cast<size_t>(r) * p.vdim + c0] : 0.f;
      S1[i] = init != nullptr && two && r < p.dim ? init[static_cast<size_t>(r) * p.vdim + c0 + 1] : 0.f;
    }
  }
  float keep[(DP + 31) / 32];                         // PART: decay of the rows this thread follows (blocks have at least 32 threads)
  if constexpr (PART) {
#pragma unroll
    for (int i = 0; i < (DP + 31) / 32; ++i) keep[i] = 1.f;
  }
  fetch(a);
  for (int t0 = a; t0 < b; t0 += CH) {
    const int n = min(CH, b - t0);
    if constexpr (VEC) copies_wait();
    __syncthreads();
    for (int i = tid; i < n * p.dim; i += blockDim.x) {
      const int t = i / p.dim, c = i - t * p.dim;
      const size_t g = static_cast<size_t>(t0 + t) * p.ld + c;
      if constexpr (!PART) s_q[t * DP + c] = silu(ld(VEC ? r_q + i : gq + g));
      s_k[t * DP + c] = let_in(ld(VEC ? r_f + i : gf + g) + s_bias[c], s_low[c]);
    }
    for (int i = tid; i < n * ncol; i += blockDim.x) {
      const int t = i / ncol, c = i - t * ncol;
      s_v[t * VP + c] = ld(VEC ? r_v + i : gv + static_cast<size_t>(t0 + t) * p.ld + c);
    }
    __syncthreads();
    if (t0 + CH < b) fetch(t0 + CH);
    for (int t = 0; t < n; ++t) {
      const float v0 = mine ? s_v[t * VP + c0] : 0.f, v1 = two ? s_v[t * VP + c0 + 1] : 0.f;
      float o0 = 0.f, o1 = 0.f, u0 = 0.f, u1 = 0.f;
#pragma unroll
      for (int i = 0; i < RPT; i += 4) {
        const float4 kk = *reinterpret_cast<const float4*>(s_k + t * DP + ((i >> 2) * RS + rs) * 4);
        S0[i] = fmaf(kk.x, v0 - S0[i], S0[i]);
        S1[i] = fmaf(kk.x, v1 - S1[i], S1[i]);
        S0[i + 1] = fmaf(kk.y, v0 - S0[i + 1], S0[i + 1]);
        S1[i + 1] = fmaf(kk.y, v1 - S1[i + 1], S1[i + 1]);
        S0[i + 2] = fmaf(kk.z, v0 - S0[i + 2], S0[i + 2]);
        S1[i + 2] = fmaf(kk.z, v1 - S1[i + 2], S1[i + 2]);
        S0[i + 3] = fmaf(kk.w, v0 - S0[i + 3], S0[i + 3]);
        S1[i + 3] = fmaf(kk.w, v1 - S1[i + 3], S1[i + 3]);
        if constexpr (!PART) {
          const float4 qq = *reinterpret_cast<const float4*>(s_q + t * DP + ((i >> 2) * RS + rs) * 4);
          o0 = fmaf(qq.x, S0[i], o0); o1 = fmaf(qq.x, S1[i], o1);
          u0 = fmaf(qq.y, S0[i + 1], u0); u1 = fmaf(qq.y, S1[i + 1], u1);
          o0 = fmaf(qq.z, S0[i + 2], o0); o1 = fmaf(qq.z, S1[i + 2], o1);
          u0 = fmaf(qq.w, S0[i + 3], u0); u1 = fmaf(qq.w, S1[i + 3], u1);
        }
      }
      if constexpr (!PART) {
        o0 += u0;
        o1 += u1;
#pragma unroll
        for (int o = 1; o < RS; o <<= 1) {
          o0 += __shfl_xor_sync(0xffffffffu, o0, o);
          o1 += __shfl_xor_sync(0xffffffffu, o1, o);
        }
        // every lane that shares the columns has read its values by now: outputs take their place
        if (rs == 0 && mine) s_v[t * VP + c0] = o0;
        if (rs == RS - 1 && two) s_v[t * VP + c0 + 1] = o1;
      }
    }
    if constexpr (PART) {
#pragma unroll
      for (int i = 0; i < (DP + 31) / 32; ++i) {
        const int r = i * blockDim.x + tid;
        if (r < p.dim)
          for (int t = 0; t < n; ++t) keep[i] *= 1.f - s_k[t * DP + r];
      }
    } else {
      __syncthreads();
      const int warp = tid >> 5, lane = tid & 31;
      for (int t = warp; t < n; t += blockDim.x >> 5) {
        const size_t at = static_cast<size_t>(s0 + t0 + t) * p.H * p.vdim + static_cast<size_t>(head) * p.vdim + col0;
        if (p.raw != nullptr) {
          for (int c = lane; c < ncol; c += 32) p.raw[at + c] = s_v[t * VP + c];
          continue;
        }
        float ss = 0.f;
        for (int c = lane; c < ncol; c += 32) ss += s_v[t * VP + c] * s_v[t * VP + c];
        const float r = rsqrtf(warp_sum(ss) / p.vdim + p.eps);
        for (int c = lane; c < ncol; c += 32) st(p.o + at + c, s_v[t * VP + c] * r * ld(p.weight + c));
      }
    }
  }
  float* out = nullptr;
  if constexpr (PART) {
    out = p.part + ((static_cast<size_t>(seq) * (p.segments - 1) + seg) * p.H + head) * head_state + col0;
    if (slice == 0) {
      float* d = p.decay + ((static_cast<size_t>(seq) * (p.segments - 1) + seg) * p.H + head) * p.dim;
#pragma unroll
      for (int i = 0; i < (DP + 31) / 32; ++i) {
        const int r = i * blockDim.x + tid;
        if (r < p.dim) d[r] = keep[i];
      }
    }
  } else if (p.pool != nullptr && b == len) {
    const int sl = p.slot[s0];
    if (sl > 0) out = p.pool + (static_cast<size_t>(sl) * p.H + head) * head_state + col0;
  }
  if (out != nullptr) {
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int r = row_of(i);
      if (r < p.dim) {
        if (mine) out[static_cast<size_t>(r) * p.vdim + c0] = S0[i];
        if (two) out[static_cast<size_t>(r) * p.vdim + c0 + 1] = S1[i];
      }
    }
  }
}

// ------------------------------------------------------------------ sixteen tokens per step on the tensor cores
namespace hg {
constexpr int TOK = 32;         // tokens per round: two steps

// shared memory of a block, in bytes from its start
struct Layout {
  int q, k, qh, ql, kh, kl, a, v, rq, rf, d, low, ss, total, po;
  __host__ __device__ Layout(int DP, int VP) {
    const int pitch = DP + 8;
    po = VP + 4;                                         // row pitch of the outputs, which take the place of q and k
    q = 0;
    k = q + TOK * DP * 4;
    int at = k + TOK * DP * 4;
    if (at < TOK * po * 4) at = TOK * po * 4;
    qh = at; ql = qh + TOK * pitch * 2; kh = ql + TOK * pitch * 2; kl = kh + TOK * pitch * 2;
    a = kl + TOK * pitch * 2;                            // [2 steps][hi, lo][16][24]
    v = a + 2 * 2 * 16 * 24 * 2;                         // [2][TOK][VP + 8]
    rq = v + 2 * TOK * (VP + 8) * 2; rf = rq + TOK * DP * 2;
    d = rf + TOK * DP * 2;                               // [2 steps][DP]
    low = d + 2 * DP * 4;                                // [DP] lower bound, [DP] bias
    ss = low + 2 * DP * 4;                               // [8 warps][TOK]
    total = ss + 8 * TOK * 4;
  }
};
}  // namespace hg

// A warp owns 16 columns of the head's values: Sᵀ [16, DP] lies in its registers as accumulators of Vᵀ (k R) and, packed, as the
// left operand of Sᵀ (q P)ᵀ.  PART: only the state a segment builds up from nothing and its decay.
template <int DP, bool PART>
__global__ void __launch_bounds__(256, 2) hgrn2_chunk_kernel(const Hgrn2<bf16> p) {
  using namespace hg;
  extern __shared__ __align__(16) uint8_t sm_chunk[];
  constexpr int PITCH = DP + 8, NT = DP / 8, DS = DP / 8;     // DS: lanes that share the sum over a head's width
  const int head = blockIdx.x / p.slices, slice = blockIdx.x - head * p.slices, seg = blockIdx.y, seq = blockIdx.z;
  const int s0 = p.cu[seq], len = p.cu[seq + 1] - s0;
  const int a = seg * p.seg_len, b = min(len, a + p.seg_len);
  if (a >= len || (PART && b >= len)) return;
  const int col0 = slice * p.cols, ncol = min(p.cols, p.vdim - col0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, warps = blockDim.x >> 5, VP = warps * 16, VPITCH = VP + 8;
  const Layout L(DP, VP);
  float *s_q = reinterpret_cast<float*>(sm_chunk + L.q), *s_k = reinterpret_cast<float*>(sm_chunk + L.k), *s_o = s_q;
  bf16 *s_qh = reinterpret_cast<bf16*>(sm_chunk + L.qh), *s_ql = reinterpret_cast<bf16*>(sm_chunk + L.ql), *s_kh = reinterpret_cast<bf16*>(sm_chunk + L.kh),
       *s_kl = reinterpret_cast<bf16*>(sm_chunk + L.kl), *s_a = reinterpret_cast<bf16*>(sm_chunk + L.a), *s_v = reinterpret_cast<bf16*>(sm_chunk + L.v),
       *r_q = reinterpret_cast<bf16*>(sm_chunk + L.rq), *r_f = reinterpret_cast<bf16*>(sm_chunk + L.rf);
  float *s_d = reinterpret_cast<float*>(sm_chunk + L.d), *s_low = reinterpret_cast<float*>(sm_chunk + L.low), *s_bias = s_low + DP,
        *s_ss = reinterpret_cast<float*>(sm_chunk + L.ss);
  for (int i = tid; i < DP; i += blockDim.x) {
    s_low[i] = i < p.dim ? ld(p.lower + static_cast<size_t>(head) * p.dim + i) : 1.f;
    s_bias[i] = i < p.dim ? ld(p.bias + static_cast<size_t>(head) * p.dim + i) : 0.f;
  }
  for (int i = tid; i < TOK * DP; i += blockDim.x) r_q[i] = r_f[i] = __float2bfloat16(0.f);      // columns past the head's width
  for (int i = tid; i < 2 * TOK * VPITCH; i += blockDim.x) s_v[i] = __float2bfloat16(0.f);
  __syncthreads();
  const bf16* gq = p.q + static_cast<size_t>(s0) * p.ld + static_cast<size_t>(head) * p.dim;
  const bf16* gf = p.f + static_cast<size_t>(s0) * p.ld + static_cast<size_t>(head) * p.dim;
  const bf16* gv = p.v + static_cast<size_t>(s0) * p.ld + static_cast<size_t>(head) * p.vdim + col0;
  auto fetch = [&](int t0, int buf) {
    const int n = min(TOK, b - t0), dv = p.dim >> 3, vv = ncol >> 3;
    for (int i = tid; i < n * dv; i += blockDim.x) {
      const int t = i / dv, c = (i - t * dv) * 8;
      const size_t g = static_cast<size_t>(t0 + t) * p.ld + c;
      if constexpr (!PART) copy16(r_q + t * DP + c, gq + g);
      copy16(r_f + t * DP + c, gf + g);
    }
    for (int i = tid; i < n * vv; i += blockDim.x) {
      const int t = i / vv, c = (i - t * vv) * 8;
      copy16(s_v + (buf * TOK + t) * VPITCH + c, gv + static_cast<size_t>(t0 + t) * p.ld + c);
    }
    copies_commit();
  };
  const int g = lane >> 2, tq = lane & 3;                // row and column pair of a lane in an accumulator
  const size_t head_state = static_cast<size_t>(p.dim) * p.vdim;
  const int v_lo = warp * 16 + g, v_hi = v_lo + 8;       // this lane's columns of the head (rows of Sᵀ), relative to col0
  float S[NT][4];
  {
    const float* init = (!PART && seg > 0) ? p.part + ((static_cast<size_t>(seq) * (p.segments - 1) + seg - 1) * p.H + head) * head_state + col0 : nullptr;
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = n * 8 + tq * 2 + (e & 1), c = e < 2 ? v_lo : v_hi;
        S[n][e] = init != nullptr && r < p.dim && c < ncol ? init[static_cast<size_t>(r) * p.vdim + c] : 0.f;
      }
  }
  float keep[(DP + 31) / 32];
  if constexpr (PART) {
#pragma unroll
    for (int i = 0; i < (DP + 31) / 32; ++i) keep[i] = 1.f;
  }
  fetch(a, 0);
  int buf = 0;
  for (int t0 = a; t0 < b; t0 += TOK, buf ^= 1) {
    const int n = min(TOK, b - t0);
    copies_wait();
    __syncthreads();
    // what enters the recurrence, in fp32; tokens past the end write nothing and decay nothing
    for (int i = tid; i < TOK * DP / 2; i += blockDim.x) {
      const int t = i / (DP / 2), c = (i - t * (DP / 2)) * 2;
      float2 q = make_float2(0.f, 0.f), k = q;
      if (t < n) {
        if constexpr (!PART) {
          q = unpack_bf16(reinterpret_cast<const uint32_t*>(r_q)[i]);
          q.x = silu(q.x); q.y = silu(q.y);
        }
        const float2 f = unpack_bf16(reinterpret_cast<const uint32_t*>(r_f)[i]);
        k.x = let_in(f.x + s_bias[c], s_low[c]); k.y = let_in(f.y + s_bias[c + 1], s_low[c + 1]);
      }
      if constexpr (!PART) reinterpret_cast<float2*>(s_q)[i] = q;
      reinterpret_cast<float2*>(s_k)[i] = k;
    }
    if (n < TOK)
      for (int i = tid; i < (TOK - n) * VP; i += blockDim.x) s_v[(buf * TOK + n + i / VP) * VPITCH + i % VP] = __float2bfloat16(0.f);
    __syncthreads();
    if (t0 + TOK < b) fetch(t0 + TOK, buf ^ 1);
    // q P, k R and D: a thread follows one channel through one step
    for (int i = tid; i < 2 * DP; i += blockDim.x) {
      const int step = i / DP, c = i - step * DP, at = step * 16;
      float w = 1.f;
#pragma unroll
      for (int t = 15; t >= 0; --t) {
        const float k = s_k[(at + t) * DP + c];
        split(k * w, s_kh + (at + t) * PITCH + c, s_kl + (at + t) * PITCH + c);
        w *= 1.f - k;
      }
      s_d[i] = w;
      if constexpr (!PART) {
        w = 1.f;
#pragma unroll
        for (int t = 0; t < 16; ++t) {
          w *= 1.f - s_k[(at + t) * DP + c];
          split(s_q[(at + t) * DP + c] * w, s_qh + (at + t) * PITCH + c, s_ql + (at + t) * PITCH + c);
        }
      }
    }
    // A: DS lanes share token j's row of products and follow what j wrote through the tokens behind it
    if constexpr (!PART) {
      constexpr int JW = 32 / DS, ITEMS = 16 / JW;       // tokens j a warp follows at once, such groups in a step
      const int sub = lane % DS;
      for (int i = warp; i < 2 * ITEMS; i += warps) {
        // the second step's groups in reverse: a warp that followed the longest rows follows the shortest next
        const int step = i / ITEMS, first = (step ? 2 * ITEMS - 1 - i : i) * JW, j = first + lane / DS;
        const float *qr = s_q + (step * 16 + first) * DP + sub * 4, *kr = s_k + (step * 16 + first) * DP + sub * 4;
        float w[8], acc[16];                             // acc[r]: token first + r
#pragma unroll
        for (int t = 0; t < 16; ++t) acc[t] = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) w[e] = 0.f;
#pragma unroll
        for (int r = 0; r < 16; ++r) {
          if (first + r < 16) {
#pragma unroll
            for (int u = 0; u < 2; ++u) {
              const float4 q4 = *reinterpret_cast<const float4*>(qr + r * DP + u * (DP / 2)), k4 = *reinterpret_cast<const float4*>(kr + r * DP + u * (DP / 2));
              const float q[4] = {q4.x, q4.y, q4.z, q4.w}, k[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                float& x = w[4 * u + e];
                x = fmaf(-x, k[e], x);
                if (r < JW && first + r == j) x = k[e];
                acc[r] = fmaf(q[e], x, acc[r]);
              }
            }
          }
        }
        // sum over the DS lanes; lane `sub` is left with 16 / DS of the sixteen
        int left = 16, base = 0;
#pragma unroll
        for (int o = DS / 2; o > 0; o >>= 1) {
          const bool upper = sub & o;
          left >>= 1;
#pragma unroll
          for (int x = 0; x < 8; ++x) {
            if (x < left) {
              const float send = upper ? acc[x] : acc[x + left], kept = upper ? acc[x + left] : acc[x];
              acc[x] = kept + __shfl_xor_sync(0xffffffffu, send, o);
            }
          }
          base += upper ? left : 0;
        }
        bf16* ah = s_a + step * 2 * 16 * 24;
#pragma unroll
        for (int x = 0; x < 16 / DS; ++x) {
          const int t = first + base + x;                // tokens in front of the group's first see nothing of it
          if (t < 16) split(acc[x], ah + t * 24 + j, ah + 16 * 24 + t * 24 + j);
          else ah[(t - 16) * 24 + j] = ah[16 * 24 + (t - 16) * 24 + j] = __float2bfloat16(0.f);
        }
      }
    }
    __syncthreads();
#pragma unroll 1
    for (int step = 0; step < 2; ++step) {
      if (step * 16 >= n) break;
      const int at = step * 16;
      uint32_t va[4];                                    // Vᵀ of the step: [16 columns, 16 tokens]
      ldsm4t(va, s_v + (buf * TOK + at + (lane >> 4) * 8 + (lane & 7)) * VPITCH + warp * 16 + (lane >> 3 & 1) * 8);
      if constexpr (!PART) {
        float o[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
        const int tok = at + (lane >> 4) * 8 + (lane & 7), kc = (lane >> 3 & 1) * 8;
#pragma unroll
        for (int s = 0; s < DP / 16; ++s) {
          uint32_t sh[4], sl[4], qh[4], ql[4];
          ldsm4(qh, s_qh + tok * PITCH + s * 16 + kc);
          ldsm4(ql, s_ql + tok * PITCH + s * 16 + kc);
          split2(S[2 * s][0], S[2 * s][1], sh[0], sl[0]);
          split2(S[2 * s][2], S[2 * s][3], sh[1], sl[1]);
          split2(S[2 * s + 1][0], S[2 * s + 1][1], sh[2], sl[2]);
          split2(S[2 * s + 1][2], S[2 * s + 1][3], sh[3], sl[3]);
          mma(o[0], sh, qh[0], qh[1]); mma(o[1], sh, qh[2], qh[3]);
          mma(o[0], sl, qh[0], qh[1]); mma(o[1], sl, qh[2], qh[3]);
          mma(o[0], sh, ql[0], ql[1]); mma(o[1], sh, ql[2], ql[3]);
        }
        uint32_t ah[4], al[4];
        const bf16* ar = s_a + step * 2 * 16 * 24 + (tok - at) * 24 + kc;
        ldsm4(ah, ar);
        ldsm4(al, ar + 16 * 24);
        mma(o[0], va, ah[0], ah[1]); mma(o[1], va, ah[2], ah[3]);
        mma(o[0], va, al[0], al[1]); mma(o[1], va, al[2], al[3]);
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int e = 0; e < 2; ++e) {                  // token 8 h + 2 tq + e: columns v_lo and v_hi
            const int t = at + h * 8 + tq * 2 + e;
            s_o[t * L.po + v_lo] = o[h][e];
            s_o[t * L.po + v_hi] = o[h][e + 2];
            float ss = o[h][e] * o[h][e] + o[h][e + 2] * o[h][e + 2];       // columns past the head's are zero
            ss += __shfl_xor_sync(0xffffffffu, ss, 4);
            ss += __shfl_xor_sync(0xffffffffu, ss, 8);
            ss += __shfl_xor_sync(0xffffffffu, ss, 16);
            if (g == 0) s_ss[warp * TOK + t] = ss;
          }
      }
      const int ktok = at + (lane >> 3 & 1) * 8 + (lane & 7), kd = (lane >> 4) * 8;
#pragma unroll
      for (int s = 0; s < DP / 16; ++s) {
        uint32_t kh[4], kl[4];
        ldsm4t(kh, s_kh + ktok * PITCH + s * 16 + kd);
        ldsm4t(kl, s_kl + ktok * PITCH + s * 16 + kd);
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const float2 d = *reinterpret_cast<const float2*>(s_d + step * DP + s * 16 + h * 8 + tq * 2);
          float (&x)[4] = S[2 * s + h];
          x[0] *= d.x; x[1] *= d.y; x[2] *= d.x; x[3] *= d.y;
          mma(x, va, kh[2 * h], kh[2 * h + 1]);
          mma(x, va, kl[2 * h], kl[2 * h + 1]);
        }
      }
    }
    if constexpr (PART) {
#pragma unroll
      for (int i = 0; i < (DP + 31) / 32; ++i) {
        const int r = i * blockDim.x + tid;
        if (r < DP) keep[i] *= s_d[r] * s_d[DP + r];
      }
    } else {
      __syncthreads();
      for (int t = warp; t < n; t += warps) {
        const size_t out = static_cast<size_t>(s0 + t0 + t) * p.H * p.vdim + static_cast<size_t>(head) * p.vdim + col0;
        if (p.raw != nullptr) {
          for (int c = lane; c < ncol; c += 32) p.raw[out + c] = s_o[t * L.po + c];
          continue;
        }
        float ss = 0.f;
        for (int w = 0; w < warps; ++w) ss += s_ss[w * TOK + t];
        const float r = rsqrtf(ss / p.vdim + p.eps);
        for (int c = lane * 2; c < ncol; c += 64) {
          const float2 x = *reinterpret_cast<const float2*>(s_o + t * L.po + c), w = unpack_bf16(*reinterpret_cast<const uint32_t*>(p.weight + c));
          *reinterpret_cast<uint32_t*>(p.o + out + c) = pack_bf16(x.x * r * w.x, x.y * r * w.y);
        }
      }
    }
  }
  float* out = nullptr;
  if constexpr (PART) {
    out = p.part + ((static_cast<size_t>(seq) * (p.segments - 1) + seg) * p.H + head) * head_state + col0;
    if (slice == 0) {
      float* d = p.decay + ((static_cast<size_t>(seq) * (p.segments - 1) + seg) * p.H + head) * p.dim;
#pragma unroll
      for (int i = 0; i < (DP + 31) / 32; ++i) {
        const int r = i * blockDim.x + tid;
        if (r < p.dim) d[r] = keep[i];
      }
    }
  } else if (p.pool != nullptr && b == len) {
    const int sl = p.slot[s0];
    if (sl > 0) out = p.pool + (static_cast<size_t>(sl) * p.H + head) * head_state + col0;
  }
  if (out != nullptr) {
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = n * 8 + tq * 2 + (e & 1), c = e < 2 ? v_lo : v_hi;
        if (r < p.dim && c < ncol) out[static_cast<size_t>(r) * p.vdim + c] = S[n][e];
      }
  }
}

// part[s] becomes the state behind segment s: a scan over the segments of every sequence, one thread per state element.
__global__ void __launch_bounds__(256) hgrn2_scan_kernel(float* part, const float* __restrict__ decay, const int* __restrict__ cu, int H, int dim, int vdim,
                                                         int seg_len, int segments) {
  const int seq = blockIdx.y, len = cu[seq + 1] - cu[seq];
  const long per = static_cast<long>(H) * dim * vdim, i = blockIdx.x * 256L + threadIdx.x;
  if (i >= per) return;
  float S = 0.f;
  for (int s = 0; s < segments - 1 && (s + 1) * seg_len < len; ++s) {
    const size_t at = (static_cast<size_t>(seq) * (segments - 1) + s) * per + i;
    S = fmaf(decay[(static_cast<size_t>(seq) * (segments - 1) + s) * H * dim + i / vdim], S, part[at]);
    part[at] = S;
  }
}

// Norm of heads whose columns were split over blocks: one warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(256) hgrn2_norm_kernel(const float* __restrict__ raw, const T* __restrict__ weight, T* __restrict__ o, long heads, int vdim, float eps) {
  const long i = blockIdx.x * 8L + (threadIdx.x >> 5);
  if (i >= heads) return;
  const int lane = threadIdx.x & 31;
  float ss = 0.f;
  for (int c = lane; c < vdim; c += 32) ss += raw[i * vdim + c] * raw[i * vdim + c];
  const float r = rsqrtf(warp_sum(ss) / vdim + eps);
  for (int c = lane; c < vdim; c += 32) hg::st(o + i * vdim + c, raw[i * vdim + c] * r * hg::ld(weight + c));
}

// One token per sequence: block = (head, sequence), V consecutive columns per access.  Slot 0: a row that fills up a batch.
template <typename T, int V>
__global__ void __launch_bounds__(256) hgrn2_step_kernel(const Hgrn2<T> p) {
  using namespace hg;
  extern __shared__ __align__(16) float sm_step[];
  __shared__ float s_part[8];
  const int head = blockIdx.x, row = blockIdx.y, tid = threadIdx.x, dim = p.dim, vdim = p.vdim;
  T* o = p.o + static_cast<size_t>(row) * p.H * vdim + static_cast<size_t>(head) * vdim;
  const int slot = p.slot[row];
  if (slot <= 0) {
    for (int c = tid; c < vdim; c += 256) st(o + c, 0.f);
    return;
  }
  float *s_q = sm_step, *s_k = s_q + dim, *s_v = s_k + dim, *s_o = s_v + (vdim + 3) / 4 * 4;
  const size_t g = static_cast<size_t>(row) * p.ld, hd = static_cast<size_t>(head) * dim;
  for (int c = tid; c < dim; c += 256) {
    s_q[c] = silu(ld(p.q + g + hd + c));
    s_k[c] = let_in(ld(p.f + g + hd + c) + ld(p.bias + hd + c), ld(p.lower + hd + c));
  }
  for (int c = tid; c < vdim; c += 256) s_v[c] = ld(p.v + g + static_cast<size_t>(head) * vdim + c);
  const int cg = vdim / V, rg = 256 / cg, c = tid % cg * V, r0 = tid / cg;
  float* S = p.pool + (static_cast<size_t>(slot) * p.H + head) * dim * vdim + c;
  float acc[V];
#pragma unroll
  for (int i = 0; i < V; ++i) acc[i] = 0.f;
  __syncthreads();
  if (r0 < rg) {
    constexpr int U = 8;
    for (int rb = r0; rb < dim; rb += rg * U) {
      float x[U][V];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int r = rb + u * rg;
        if (r < dim) {
          if constexpr (V == 4) {
            const float4 w = *reinterpret_cast<const float4*>(S + static_cast<size_t>(r) * vdim);
            x[u][0] = w.x; x[u][1] = w.y; x[u][2] = w.z; x[u][3] = w.w;
          } else {
            x[u][0] = S[static_cast<size_t>(r) * vdim];
          }
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int r = rb + u * rg;
        if (r < dim) {
          const float k = s_k[r], q = s_q[r];
#pragma unroll
          for (int i = 0; i < V; ++i) {
            x[u][i] = fmaf(k, s_v[c + i] - x[u][i], x[u][i]);
            acc[i] = fmaf(q, x[u][i], acc[i]);
          }
          if constexpr (V == 4) *reinterpret_cast<float4*>(S + static_cast<size_t>(r) * vdim) = make_float4(x[u][0], x[u][1], x[u][2], x[u][3]);
          else S[static_cast<size_t>(r) * vdim] = x[u][0];
        }
      }
    }
#pragma unroll
    for (int i = 0; i < V; ++i) s_o[r0 * vdim + c + i] = acc[i];
  }
  __syncthreads();
  float y = 0.f;                                  // vdim ≤ 256: a thread finishes one column
  if (tid < vdim)
    for (int r = 0; r < rg; ++r) y += s_o[r * vdim + tid];
  const float part = warp_sum(y * y);
  if ((tid & 31) == 0) s_part[tid >> 5] = part;
  __syncthreads();
  float ss = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) ss += s_part[w];
  if (tid < vdim) st(o + tid, y * rsqrtf(ss / vdim + p.eps) * ld(p.weight + tid));
}

namespace {

template <typename T>
Hgrn2<T> hgrn2_args(const torch::Tensor& proj, int64_t q0, int64_t f0, int64_t v0, int64_t H, int64_t dim, int64_t vdim, const torch::Tensor& bias,
                    const torch::Tensor& lower, const torch::Tensor& weight, double eps, torch::Tensor& o, const OptT& pool, const OptT& slot) {
  Hgrn2<T> p{};
  const T* base = reinterpret_cast<const T*>(proj.data_ptr());
  p.q = base + q0; p.f = base + f0; p.v = base + v0; p.ld = proj.stride(0);
  p.bias = reinterpret_cast<const T*>(bias.data_ptr()); p.lower = reinterpret_cast<const T*>(lower.data_ptr());
  p.weight = reinterpret_cast<const T*>(weight.data_ptr()); p.o = reinterpret_cast<T*>(o.data_ptr());
  if (pool.has_value() && pool->defined()) { p.pool = pool->data_ptr<float>(); p.slot = slot->data_ptr<int>(); }
  p.H = H; p.dim = dim; p.vdim = vdim; p.eps = eps;
  return p;
}

void hgrn2_check(const torch::Tensor& proj, int64_t q0, int64_t f0, int64_t v0, int64_t H, int64_t dim, int64_t vdim, const torch::Tensor& bias,
                 const torch::Tensor& lower, const torch::Tensor& weight, const OptT& pool, const OptT& slot) {
  const auto st = proj.scalar_type();
  TORCH_CHECK(proj.is_cuda() && proj.dim() == 2 && proj.stride(1) == 1 && (st == torch::kBFloat16 || st == torch::kFloat32), "projection [rows, N] bf16 or fp32");
  TORCH_CHECK(H > 0 && dim > 0 && vdim > 0 && dim <= 256 && vdim <= 256, "hgrn2: head widths up to 256");
  TORCH_CHECK(q0 >= 0 && f0 >= 0 && v0 >= 0 && q0 + H * dim <= proj.size(1) && f0 + H * dim <= proj.size(1) && v0 + H * vdim <= proj.size(1), "columns outside the projection");
  for (const auto* t : {&bias, &lower}) TORCH_CHECK(t->scalar_type() == st && t->is_contiguous() && t->numel() == H * dim, "gate bias and lower bound [heads·dim]");
  TORCH_CHECK(weight.scalar_type() == st && weight.is_contiguous() && weight.numel() == vdim, "norm weight [vdim]");
  if (pool.has_value() && pool->defined()) {
    TORCH_CHECK(pool->scalar_type() == torch::kFloat32 && pool->is_contiguous() && pool->dim() == 4 && pool->size(1) == H && pool->size(2) == dim && pool->size(3) == vdim,
                "state pool [slots, heads, dim, vdim] fp32");
    TORCH_CHECK(slot.has_value() && slot->defined() && slot->scalar_type() == torch::kInt32 && slot->is_contiguous() && slot->numel() == proj.size(0), "slot int32 [rows]");
  }
}

bool on16(const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; }

}  // namespace

torch::Tensor hgrn2_prefill(const torch::Tensor& proj, int64_t q0, int64_t f0, int64_t v0, int64_t H, int64_t dim, int64_t vdim, const torch::Tensor& bias,
                            const torch::Tensor& lower, const torch::Tensor& weight, double eps, const torch::Tensor& cu, int64_t max_seqlen, const OptT& pool,
                            const OptT& slot) {
  hgrn2_check(proj, q0, f0, v0, H, dim, vdim, bias, lower, weight, pool, slot);
  TORCH_CHECK(cu.is_cuda() && cu.scalar_type() == torch::kInt32 && cu.is_contiguous(), "cu_seqlens int32 on device");
  c10::cuda::CUDAGuard guard(proj.device());
  const int rows = proj.size(0), n = cu.numel() - 1;
  auto o = torch::empty({rows, H * vdim}, proj.options());
  if (rows == 0 || n <= 0 || max_seqlen <= 0) return o;
  auto f32 = proj.options().dtype(torch::kFloat32);
  auto stream = at::cuda::getCurrentCUDAStream();
  auto run = [&](auto tag) {
    using T = decltype(tag);
    auto p = hgrn2_args<T>(proj, q0, f0, v0, H, dim, vdim, bias, lower, weight, eps, o, pool, slot);
    p.cu = cu.data_ptr<int>();
    constexpr int E = 16 / sizeof(T);
    const bool whole = dim % E == 0 && vdim % E == 0 && p.ld % E == 0 && on16(p.q) && on16(p.f) && on16(p.v);      // 16-byte vectors everywhere
    const bool chunks = sizeof(T) == 2 && whole && dim <= 128 && reinterpret_cast<uintptr_t>(p.weight) % 4 == 0;
    const int rpt = dim <= 64 ? 32 : 64, rs = dim <= 32 ? 1 : (dim <= 128 ? 2 : 4);
    const int most = chunks ? 128 : 256 / rs * 2;                // columns a block can hold
    p.slices = (vdim + most - 1) / most;
    p.cols = p.slices == 1 ? (vdim + 1) / 2 * 2 : most;
    torch::Tensor raw, part, decay;
    if (p.slices > 1) { raw = torch::empty({rows, H * vdim}, f32); p.raw = raw.data_ptr<float>(); }
    // time segments: at most two blocks per SM (one wave), none shorter than 128 tokens (a segment costs a second pass over its state)
    const long blocks = static_cast<long>(H) * p.slices * n;
    long segs = blocks >= num_sms() ? 1 : std::min<long>(2L * num_sms() / blocks, max_seqlen / 128);
    segs = std::max<long>(segs, 1);
    p.seg_len = static_cast<int>(((max_seqlen + segs - 1) / segs + hg::CH - 1) / hg::CH * hg::CH);
    p.segments = static_cast<int>((max_seqlen + p.seg_len - 1) / p.seg_len);
    if (p.segments > 1) {
      part = torch::empty({n, p.segments - 1, H, dim, vdim}, f32);
      decay = torch::empty({n, p.segments - 1, H, dim}, f32);
      p.part = part.data_ptr<float>(); p.decay = decay.data_ptr<float>();
    }
    TORCH_CHECK(n <= 65535, "too many sequences in one call");
    const bool vec = whole && p.cols % E == 0;
    const int warps = (p.cols + 15) / 16, dp = chunks ? (dim <= 32 ? 32 : (dim <= 64 ? 64 : 128)) : rpt * rs;
    const int threads = chunks ? 32 * warps : (((std::min<int>(p.cols, vdim) + 1) / 2) * rs + 31) / 32 * 32;
    const size_t smem = chunks ? hg::Layout(dp, warps * 16).total
                               : sizeof(float) * (2 * hg::CH * dp + hg::CH * p.cols + 2 * dp) + (vec ? sizeof(T) * hg::CH * (2 * dim + p.cols) : 0);
    auto go = [&](auto kern, int segments) {
      TK_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
      kern<<<dim3(H * p.slices, segments, n), threads, smem, stream>>>(p);
      count_launch();
      TK_CUDA_CHECK(cudaGetLastError());
    };
#define TK_HGRN2(PART, SEGS)                                                                                             \
  do {                                                                                                                   \
    if constexpr (sizeof(T) == 2) {                                                                                      \
      if (chunks) {                                                                                                      \
        if (dp == 32) go(hgrn2_chunk_kernel<32, PART>, SEGS);                                                            \
        else if (dp == 64) go(hgrn2_chunk_kernel<64, PART>, SEGS);                                                       \
        else go(hgrn2_chunk_kernel<128, PART>, SEGS);                                                                    \
        break;                                                                                                           \
      }                                                                                                                  \
    }                                                                                                                    \
    if (vec) {                                                                                                           \
      if (rpt == 32 && rs == 1) go(hgrn2_prefill_kernel<T, 32, 1, true, PART>, SEGS);                                    \
      else if (rpt == 32) go(hgrn2_prefill_kernel<T, 32, 2, true, PART>, SEGS);                                          \
      else if (rs == 2) go(hgrn2_prefill_kernel<T, 64, 2, true, PART>, SEGS);                                            \
      else go(hgrn2_prefill_kernel<T, 64, 4, true, PART>, SEGS);                                                         \
    } else {                                                                                                             \
      if (rpt == 32 && rs == 1) go(hgrn2_prefill_kernel<T, 32, 1, false, PART>, SEGS);                                   \
      else if (rpt == 32) go(hgrn2_prefill_kernel<T, 32, 2, false, PART>, SEGS);                                         \
      else if (rs == 2) go(hgrn2_prefill_kernel<T, 64, 2, false, PART>, SEGS);                                           \
      else go(hgrn2_prefill_kernel<T, 64, 4, false, PART>, SEGS);                                                        \
    }                                                                                                                    \
  } while (0)
    if (p.segments > 1) {
      TK_HGRN2(true, p.segments - 1);
      hgrn2_scan_kernel<<<dim3(static_cast<unsigned>((H * dim * vdim + 255) / 256), n), 256, 0, stream>>>(p.part, p.decay, cu.data_ptr<int>(), H, dim, vdim, p.seg_len,
                                                                                                          p.segments);
      count_launch();
    }
    TK_HGRN2(false, p.segments);
#undef TK_HGRN2
    if (p.raw != nullptr) {
      const long heads = static_cast<long>(rows) * H;
      hgrn2_norm_kernel<T><<<static_cast<unsigned>((heads + 7) / 8), 256, 0, stream>>>(p.raw, p.weight, p.o, heads, vdim, p.eps);
      count_launch();
    }
    TK_CUDA_CHECK(cudaGetLastError());
  };
  if (proj.scalar_type() == torch::kBFloat16) run(bf16{}); else run(float{});
  return o;
}

torch::Tensor hgrn2_step(const torch::Tensor& proj, int64_t q0, int64_t f0, int64_t v0, int64_t H, int64_t dim, int64_t vdim, const torch::Tensor& bias,
                         const torch::Tensor& lower, const torch::Tensor& weight, double eps, const torch::Tensor& pool, const torch::Tensor& slot) {
  hgrn2_check(proj, q0, f0, v0, H, dim, vdim, bias, lower, weight, pool, slot);
  c10::cuda::CUDAGuard guard(proj.device());
  const int rows = proj.size(0);
  auto o = torch::empty({rows, H * vdim}, proj.options());
  if (rows == 0) return o;
  TORCH_CHECK(rows <= 65535, "too many sequences in one step");
  auto stream = at::cuda::getCurrentCUDAStream();
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const auto p = hgrn2_args<T>(proj, q0, f0, v0, H, dim, vdim, bias, lower, weight, eps, o, pool, slot);
    const int v = vdim % 4 == 0 ? 4 : 1, rg = 256 / static_cast<int>(vdim / v);
    const size_t smem = sizeof(float) * (2 * dim + (vdim + 3) / 4 * 4 + static_cast<size_t>(rg) * vdim);
    if (v == 4) hgrn2_step_kernel<T, 4><<<dim3(H, rows), 256, smem, stream>>>(p);
    else hgrn2_step_kernel<T, 1><<<dim3(H, rows), 256, smem, stream>>>(p);
  };
  if (proj.scalar_type() == torch::kBFloat16) run(bf16{}); else run(float{});
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return o;
}

}  // namespace tk
