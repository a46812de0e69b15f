// Matrix memory (mLSTM) between its projections.  Per head, with S ∈ R^{dim × vdim}, n ∈ R^dim and m in fp32, all zero at the start:
//
//   i = cap tanh((i_raw + b) / cap),  f = log σ(cap tanh((f_raw + b) / cap)),  m' = max(f + m, i)
//   S ← e^{f + m − m'} S + e^{i − m'} k vᵀ,   n ← likewise with k,   o = Sᵀ q / (max(|n·q|, e^{−m'}) + 10⁻⁶),   q = q_raw / √dim
//   output = o / rms(o) · weight · σ(gate)                              (rms over the head's vdim)
//
//   mlstm_prefill  packed prompts; a block owns one head of one sequence (or columns of it), the state is in registers.
//     bf16: 64 tokens per step on the tensor cores (``mlstm_chunk_kernel``).  With F the running sum of f over the step, g = i − F, m the maximum in front
//           of the step and M_t = max(m, max_{s ≤ t} g_s), the running maximum is F_t + M_t, F cancels from every weight, and none exceeds one:
//               num_t = e^{m − M_t} Sᵀ q_t + Σ_{s ≤ t} e^{g_s − M_t} (q_t · k_s) v_s,   den_t likewise with n and without v
//               S ← e^{m − M} S + Σ_s k_s (e^{g_s − M} v_s)ᵀ,   n ← likewise,   m ← F + M                      (at the step's end)
//           Operands that are not bf16 already (state, weighted scores, weighted values) go in as a bf16 value plus the bf16 of what it left over:
//           products keep 16 bits and more, sums are fp32, and the state itself is never rounded.  When sequences × heads do not fill the device,
//           sequences are cut into time segments: a first pass forms what each builds up from nothing, and the second starts every
//           segment from those before it.
//     else: token by token in fp32 (``mlstm_prefill_kernel``), sixteen at a time in shared memory.  The normaliser rides along as one more
//           column whose values are one.
//   mlstm_step     one token of every sequence: the state passes once through the block, 16 bytes per access.
// A state is a row of the pool: the matrix by rows, n and m, each from a 16-byte boundary on.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/types.h>

#include "common.cuh"
#include "host.h"
#include "mma16.cuh"
#include "scores.cuh"
#include "vec.cuh"

namespace tk {

template <typename T>
struct Mlstm {
  const T *q, *k, *v, *g, *i, *f; long ld;       // column ranges of the projection
  const T *i_bias, *f_bias, *weight;             // [H], [H], [H · vdim]
  T* o;                                          // [rows, H · vdim]
  float* raw;                                    // the same before norm, weight and gate, when a block does not hold a whole head
  const int* cu;
  float* pool; long pool_ld; const int* slot;    // [slots, H, pool_ld]
  float* part;                                   // [n, segments − 1, H, pool_ld]: like the pool, the sum of f behind the maximum
  int H, dim, vdim, n0, m0, cols, slices, rows, seg_len, segments, stages;
  float cap, inv_cap, eps, scale;
};

namespace ml {
constexpr int CH = 16;          // tokens per round of the fp32 kernel
__device__ __forceinline__ float log_sigmoid(float x) { return x < -15.f ? x : -log1pf(__expf(-x)); }
}  // namespace ml

// log gates of one token and head
template <typename T>
__device__ __forceinline__ void mlstm_gates(const Mlstm<T>& p, size_t row, int head, float& i, float& f) {
  i = p.cap * tanh_any((to_f(p.i[row * p.ld + head]) + to_f(p.i_bias[head])) * p.inv_cap);
  f = ml::log_sigmoid(p.cap * tanh_any((to_f(p.f[row * p.ld + head]) + to_f(p.f_bias[head])) * p.inv_cap));
}

// RS neighbouring lanes share a column, RPT rows each.
template <typename T, int RPT, int RS>
__global__ void __launch_bounds__(256) mlstm_prefill_kernel(const Mlstm<T> p) {
  using namespace ml;
  constexpr int DP = RPT * RS, SLOTS = 256 / RS;      // columns of a block, the last of them for the normaliser
  extern __shared__ __align__(16) float sm_ml[];
  float *s_q = sm_ml, *s_k = s_q + CH * DP, *s_v = s_k + CH * DP;       // [CH][DP], [CH][DP], [CH][SLOTS]: values, then outputs
  __shared__ float s_keep[CH], s_add[CH], s_floor[CH], s_i[CH], s_f[CH], s_m;
  const int head = blockIdx.x / p.slices, slice = blockIdx.x - head * p.slices, seq = blockIdx.z;
  const int s0 = p.cu[seq], len = p.cu[seq + 1] - s0;
  if (len <= 0) return;
  const int col0 = slice * p.cols, ncol = min(p.cols, p.vdim - col0), tid = threadIdx.x, rs = tid % RS, col = tid / RS;
  const bool norm = col == SLOTS - 1, mine = col < ncol || norm;
  if (tid == 0) s_m = 0.f;
  for (int x = tid; x < 2 * CH * DP; x += 256) s_q[x] = 0.f;            // rows that fill up the head's width stay zero
  float S[RPT];
#pragma unroll
  for (int x = 0; x < RPT; ++x) S[x] = 0.f;
  auto row_of = [&](int x) { return ((x >> 2) * RS + rs) * 4 + (x & 3); };
  for (int t0 = 0; t0 < len; t0 += CH) {
    const int n = min(CH, len - t0);
    __syncthreads();
    for (int x = tid; x < n * p.dim; x += 256) {
      const int t = x / p.dim, c = x - t * p.dim;
      const size_t at = static_cast<size_t>(s0 + t0 + t) * p.ld + static_cast<size_t>(head) * p.dim + c;
      s_q[t * DP + c] = to_f(p.q[at]) * p.scale;
      s_k[t * DP + c] = to_f(p.k[at]);
    }
    for (int x = tid; x < n * ncol; x += 256) {
      const int t = x / ncol, c = x - t * ncol;
      s_v[t * SLOTS + c] = to_f(p.v[static_cast<size_t>(s0 + t0 + t) * p.ld + static_cast<size_t>(head) * p.vdim + col0 + c]);
    }
    if (tid < n) mlstm_gates(p, static_cast<size_t>(s0 + t0 + tid), head, s_i[tid], s_f[tid]);
    __syncthreads();
    if (tid == 0) {
      float m = s_m;
      for (int t = 0; t < n; ++t) {
        const float top = fmaxf(s_f[t] + m, s_i[t]);
        s_keep[t] = __expf(s_f[t] + m - top);
        s_add[t] = __expf(s_i[t] - top);
        s_floor[t] = __expf(-top);
        m = top;
      }
      s_m = m;
    }
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float keep = s_keep[t], av = mine ? s_add[t] * (norm ? 1.f : s_v[t * SLOTS + col]) : 0.f;
      float o = 0.f, u = 0.f;
#pragma unroll
      for (int x = 0; x < RPT; x += 4) {
        const int at = t * DP + ((x >> 2) * RS + rs) * 4;
        const float4 kk = *reinterpret_cast<const float4*>(s_k + at), qq = *reinterpret_cast<const float4*>(s_q + at);
        S[x] = fmaf(kk.x, av, keep * S[x]); S[x + 1] = fmaf(kk.y, av, keep * S[x + 1]);
        S[x + 2] = fmaf(kk.z, av, keep * S[x + 2]); S[x + 3] = fmaf(kk.w, av, keep * S[x + 3]);
        o = fmaf(qq.x, S[x], o); u = fmaf(qq.y, S[x + 1], u);
        o = fmaf(qq.z, S[x + 2], o); u = fmaf(qq.w, S[x + 3], u);
      }
      o += u;
#pragma unroll
      for (int x = 1; x < RS; x <<= 1) o += __shfl_xor_sync(0xffffffffu, o, x);
      if (rs == 0 && mine) s_v[t * SLOTS + col] = o;      // every lane of the column has read its value by now
    }
    __syncthreads();
    for (int x = tid; x < n * ncol; x += 256) {
      const int t = x / ncol, c = x - t * ncol;
      const float den = fmaxf(fabsf(s_v[t * SLOTS + SLOTS - 1]), s_floor[t]) + 1e-6f;
      p.raw[static_cast<size_t>(s0 + t0 + t) * p.H * p.vdim + static_cast<size_t>(head) * p.vdim + col0 + c] = s_v[t * SLOTS + c] / den;
    }
  }
  if (p.pool == nullptr) return;
  const int sl = p.slot[s0];
  if (sl <= 0) return;
  float* out = p.pool + (static_cast<size_t>(sl) * p.H + head) * p.pool_ld;
#pragma unroll
  for (int x = 0; x < RPT; ++x) {
    const int r = row_of(x);
    if (r < p.dim) {
      if (norm) { if (slice == 0) out[p.n0 + r] = S[x]; }
      else if (mine) out[static_cast<size_t>(r) * p.vdim + col0 + col] = S[x];
    }
  }
  if (slice == 0 && tid == 0) out[p.m0] = s_m;
}

// ------------------------------------------------------------------ 64 tokens per step on the tensor cores
namespace ml {
constexpr int L = 64, PP = L + 8;      // tokens of a step, row pitch of the weighted scores
// shared memory of a block, in bytes from its start
struct Layout {
  int pitch, vpitch, opitch, qk, stage, k, v, g, p, n, rows, ss, total;
  __host__ __device__ Layout(int DP, int VP, int stages) {
    pitch = DP + 8; vpitch = VP + 8; opitch = VP + 4;
    k = L * pitch * 2;
    qk = 2 * k > L * opitch * 4 ? 2 * k : L * opitch * 4;              // outputs take the place of q and k
    v = qk; g = v + L * vpitch * 2; stage = g + L * vpitch * 2;
    p = stages * stage;                                                 // [hi, lo][L][PP]
    n = p + 2 * L * PP * 2;                                             // [DP]
    rows = n + DP * 4;                                                  // [2][5][L]: g, M, start, end weight, floor; [4][L]: row sums; [L]: q·n; [L]: 1 / den; [2]: keep
    ss = rows + (10 + 4 + 1 + 1) * L * 4 + 16;                          // [8 warps][L]
    total = ss + 8 * L * 4;
  }
};
}  // namespace ml

// A warp owns 16 columns of the head's values: Sᵀ [16, DP] lies in its registers as accumulators of (weighted V)ᵀ K and, packed, as the left
// operand of Sᵀ Qᵀ.  PART: only the state a segment builds up from nothing.
template <int DP, bool PART>
__global__ void __launch_bounds__(256, 1) mlstm_chunk_kernel(const Mlstm<bf16> p) {
  using namespace ml;
  extern __shared__ __align__(16) uint8_t sm_chunk[];
  constexpr int PITCH = DP + 8, NT = DP / 8;
  const int head = blockIdx.x / p.slices, slice = blockIdx.x - head * p.slices, seg = blockIdx.y, seq = blockIdx.z;
  const int s0 = p.cu[seq], len = p.cu[seq + 1] - s0, a = seg * p.seg_len, b = min(len, a + p.seg_len);
  if (a >= len || (PART && b >= len)) return;         // the last segment of a sequence is nobody's past
  const int col0 = slice * p.cols, ncol = min(p.cols, p.vdim - col0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, warps = blockDim.x >> 5, VP = warps * 16;
  const Layout lay(DP, VP, p.stages);
  const int VPITCH = lay.vpitch, OP = lay.opitch;
  bf16 *s_ph = reinterpret_cast<bf16*>(sm_chunk + lay.p), *s_pl = s_ph + L * PP;
  float *s_n = reinterpret_cast<float*>(sm_chunk + lay.n), *s_row = reinterpret_cast<float*>(sm_chunk + lay.rows), *s_rs = s_row + 10 * L, *s_qn = s_rs + 4 * L, *s_inv = s_qn + L,
        *s_keep = s_inv + L, *s_ss = reinterpret_cast<float*>(sm_chunk + lay.ss);
  // what copies never write stays zero: columns past the head's, and (until a step's tokens lie there) rows past the end
  for (int i = tid; i < p.stages * lay.stage / 16; i += blockDim.x) reinterpret_cast<uint4*>(sm_chunk)[i] = make_uint4(0u, 0u, 0u, 0u);
  for (int i = tid; i < 2 * L * PP / 8; i += blockDim.x) reinterpret_cast<uint4*>(s_ph)[i] = make_uint4(0u, 0u, 0u, 0u);
  const int g = lane >> 2, tq = lane & 3;             // row and column pair of a lane in an accumulator
  const int v_lo = warp * 16 + g, v_hi = v_lo + 8;    // this lane's columns of the head (rows of Sᵀ), relative to col0
  float S[NT][4], n_mine = 0.f, m_run = PART ? -INFINITY : 0.f, f_total = 0.f;
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) S[n][e] = 0.f;
  if constexpr (!PART) {
    // what the segments before this one leave behind
    for (int k = 0; k < seg; ++k) {
      const float* from = p.part + ((static_cast<size_t>(seq) * (p.segments - 1) + k) * p.H + head) * p.pool_ld;
      const float mk = from[p.m0], fk = from[p.m0 + 1], top = fmaxf(fk + m_run, mk), keep = __expf(fk + m_run - top), add = __expf(mk - top);
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = n * 8 + tq * 2 + (e & 1), c = e < 2 ? v_lo : v_hi;
          if (r < p.dim && c < ncol) S[n][e] = fmaf(keep, S[n][e], add * from[static_cast<size_t>(r) * p.vdim + col0 + c]);
        }
      if (tid < p.dim) n_mine = fmaf(keep, n_mine, add * from[p.n0 + tid]);
      m_run = top;
    }
  }
  // (dim ≤ threads or not: rows beyond the threads are re-read below)
  __syncthreads();
  for (int d = tid; d < DP; d += blockDim.x) s_n[d] = d == tid ? n_mine : 0.f;
  if constexpr (!PART) {
    for (int d = tid + blockDim.x; d < p.dim; d += blockDim.x) {
      float m = 0.f, n = 0.f;
      for (int k = 0; k < seg; ++k) {
        const float* from = p.part + ((static_cast<size_t>(seq) * (p.segments - 1) + k) * p.H + head) * p.pool_ld;
        const float mk = from[p.m0], fk = from[p.m0 + 1], top = fmaxf(fk + m, mk);
        n = __expf(fk + m - top) * n + __expf(mk - top) * from[p.n0 + d];
        m = top;
      }
      s_n[d] = n;
    }
  }
  const bf16* gq = p.q + static_cast<size_t>(s0) * p.ld + static_cast<size_t>(head) * p.dim;
  const bf16* gk = p.k + static_cast<size_t>(s0) * p.ld + static_cast<size_t>(head) * p.dim;
  const bf16* gv = p.v + static_cast<size_t>(s0) * p.ld + static_cast<size_t>(head) * p.vdim + col0;
  const bf16* gg = p.g + static_cast<size_t>(s0) * p.ld + static_cast<size_t>(head) * p.vdim + col0;
  auto fetch = [&](int t0, int st) {
    uint8_t* base = sm_chunk + st * lay.stage;
    bf16 *q = reinterpret_cast<bf16*>(base), *k = reinterpret_cast<bf16*>(base + lay.k), *v = reinterpret_cast<bf16*>(base + lay.v), *gt = reinterpret_cast<bf16*>(base + lay.g);
    const int n = min(L, b - t0), dv = p.dim >> 3, vv = ncol >> 3;
    for (int i = tid; i < n * dv; i += blockDim.x) {
      const int t = i / dv, c = (i - t * dv) * 8;
      const size_t at = static_cast<size_t>(t0 + t) * p.ld + c;
      if constexpr (!PART) copy16(q + t * PITCH + c, gq + at);
      copy16(k + t * PITCH + c, gk + at);
    }
    for (int i = tid; i < n * vv; i += blockDim.x) {
      const int t = i / vv, c = (i - t * vv) * 8;
      const size_t at = static_cast<size_t>(t0 + t) * p.ld + c;
      copy16(v + t * VPITCH + c, gv + at);
      if constexpr (!PART) { if (p.raw == nullptr) copy16(gt + t * VPITCH + c, gg + at); }
    }
    // outputs may lie in rows past the end
    for (int i = tid + n * PITCH / 8; i < L * PITCH / 8; i += blockDim.x) reinterpret_cast<uint4*>(q)[i] = reinterpret_cast<uint4*>(k)[i] = make_uint4(0u, 0u, 0u, 0u);
    copies_commit();
  };
  // The last warp forms the gates of a step while the others work on the one before: a lane has two neighbouring tokens.
  const bool keeper = warp == warps - 1;
  bf16 raw_i[2], raw_f[2];
  auto fetch_gates = [&](int t0) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = t0 + 2 * lane + e;
      if (t < b) {
        raw_i[e] = p.i[static_cast<size_t>(s0 + t) * p.ld + head];
        raw_f[e] = p.f[static_cast<size_t>(s0 + t) * p.ld + head];
      }
    }
  };
  const float i_bias = to_f(p.i_bias[head]), f_bias = to_f(p.f_bias[head]);
  auto form_gates = [&](int t0, int par) {
    float fi[2], ii[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const bool in = t0 + 2 * lane + e < b;           // tokens past the end write nothing and decay nothing
      ii[e] = in ? p.cap * tanh_any((to_f(raw_i[e]) + i_bias) * p.inv_cap) : -INFINITY;
      fi[e] = in ? ml::log_sigmoid(p.cap * tanh_any((to_f(raw_f[e]) + f_bias) * p.inv_cap)) : 0.f;
    }
    float sum = fi[0] + fi[1], incl = sum;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, incl, o);
      if (lane >= o) incl += x;
    }
    const float F0 = incl - sum + fi[0], F1 = F0 + fi[1], g0 = ii[0] - F0, g1 = ii[1] - F1;
    float top = fmaxf(g0, g1);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, top, o);
      if (lane >= o) top = fmaxf(top, x);
    }
    float before = __shfl_up_sync(0xffffffffu, top, 1);
    if (lane == 0) before = -INFINITY;
    const float M0 = fmaxf(m_run, fmaxf(before, g0)), M1 = fmaxf(m_run, top);
    const float Mend = __shfl_sync(0xffffffffu, M1, 31), Fend = __shfl_sync(0xffffffffu, F1, 31);
    float* row = s_row + par * 5 * L + 2 * lane;
    row[0] = g0; row[1] = g1;
    row[L] = M0; row[L + 1] = M1;
    row[2 * L] = __expf(m_run - M0); row[2 * L + 1] = __expf(m_run - M1);
    row[3 * L] = __expf(g0 - Mend); row[3 * L + 1] = __expf(g1 - Mend);
    row[4 * L] = __expf(-F0 - M0); row[4 * L + 1] = __expf(-F1 - M1);
    if (lane == 0) s_keep[par] = __expf(m_run - Mend);
    m_run = Fend + Mend;
    f_total += Fend;
  };
  fetch(a, 0);
  if (keeper) {
    fetch_gates(a);
    form_gates(a, 0);
    if (a + L < b) fetch_gates(a + L);
  }
  int st = 0, par = 0;
  for (int t0 = a; t0 < b; t0 += L, par ^= 1) {
    copies_wait();
    __syncthreads();                                  // this step's tokens and gates are there; nobody reads the other stage any more
    const int next = p.stages == 2 ? st ^ 1 : 0;
    if (p.stages == 2 && t0 + L < b) fetch(t0 + L, next);
    uint8_t* base = sm_chunk + st * lay.stage;
    const bf16 *s_q = reinterpret_cast<bf16*>(base), *s_k = reinterpret_cast<bf16*>(base + lay.k), *s_v = reinterpret_cast<bf16*>(base + lay.v),
               *s_g = reinterpret_cast<bf16*>(base + lay.g);
    const float *r_g = s_row + par * 5 * L, *r_M = r_g + L, *r_start = r_M + L, *r_end = r_start + L, *r_floor = r_end + L;
    const int tok = (lane >> 4) * 8 + (lane & 7), kc = (lane >> 3 & 1) * 8;
    float o[8][4];
    if constexpr (!PART) {
      // weighted scores: the ten 16 × 16 tiles on and below the diagonal
      for (int i = warp; i < 10; i += warps) {
        const int tr = i < 1 ? 0 : (i < 3 ? 1 : (i < 6 ? 2 : 3)), sc = i - tr * (tr + 1) / 2;
        float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
        for (int s = 0; s < DP / 16; ++s) {
          uint32_t qa[4], kb[4];
          ldsm4(qa, s_q + (tr * 16 + (lane & 15)) * PITCH + s * 16 + (lane >> 4) * 8);
          ldsm4(kb, s_k + (sc * 16 + tok) * PITCH + s * 16 + kc);
          mma(acc[0], qa, kb[0], kb[1]);
          mma(acc[1], qa, kb[2], kb[3]);
        }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int t = tr * 16 + g + r * 8;
          const float M = r_M[t];
          float sum = 0.f;
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            float w[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              const int s = sc * 16 + h * 8 + tq * 2 + e;
              w[e] = s <= t ? acc[h][r * 2 + e] * p.scale * __expf(r_g[s] - M) : 0.f;
              sum += w[e];
            }
            uint32_t hi, lo;
            split2(w[0], w[1], hi, lo);
            const int at = t * PP + sc * 16 + h * 8 + tq * 2;
            *reinterpret_cast<uint32_t*>(s_ph + at) = hi;
            *reinterpret_cast<uint32_t*>(s_pl + at) = lo;
          }
          sum += __shfl_xor_sync(0xffffffffu, sum, 1);
          sum += __shfl_xor_sync(0xffffffffu, sum, 2);
          if (tq == 0) s_rs[sc * L + t] = sum;
        }
      }
      // q · n: four lanes per token
      for (int i = tid; i < 4 * L; i += blockDim.x) {
        const int t = i >> 2, sub = i & 3;
        float dot = 0.f;
        for (int d = sub * 2; d < DP; d += 8) {
          const float2 q = unpack_bf16(*reinterpret_cast<const uint32_t*>(s_q + t * PITCH + d)), n = *reinterpret_cast<const float2*>(s_n + d);
          dot = fmaf(q.x, n.x, fmaf(q.y, n.y, dot));
        }
        dot += __shfl_xor_sync(0xffffffffu, dot, 1);
        dot += __shfl_xor_sync(0xffffffffu, dot, 2);
        if (sub == 0) s_qn[t] = dot;
      }
    }
    if (keeper && t0 + L < b) {
      form_gates(t0 + L, par ^ 1);
      if (t0 + 2 * L < b) fetch_gates(t0 + 2 * L);
    }
    if constexpr (!PART) {
      // Sᵀ Qᵀ: [16 columns, 64 tokens]
#pragma unroll
      for (int x = 0; x < 8; ++x)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[x][e] = 0.f;
#pragma unroll
      for (int s = 0; s < DP / 16; ++s) {
        uint32_t sh[4], sl[4];
        split2(S[2 * s][0], S[2 * s][1], sh[0], sl[0]);
        split2(S[2 * s][2], S[2 * s][3], sh[1], sl[1]);
        split2(S[2 * s + 1][0], S[2 * s + 1][1], sh[2], sl[2]);
        split2(S[2 * s + 1][2], S[2 * s + 1][3], sh[3], sl[3]);
#pragma unroll
        for (int tg = 0; tg < 4; ++tg) {
          uint32_t qb[4];
          ldsm4(qb, s_q + (tg * 16 + tok) * PITCH + s * 16 + kc);
          mma(o[2 * tg], sh, qb[0], qb[1]);
          mma(o[2 * tg + 1], sh, qb[2], qb[3]);
          mma(o[2 * tg], sl, qb[0], qb[1]);
          mma(o[2 * tg + 1], sl, qb[2], qb[3]);
        }
      }
#pragma unroll
      for (int x = 0; x < 8; ++x) {
        const float2 w = *reinterpret_cast<const float2*>(r_start + x * 8 + tq * 2);
        o[x][0] *= w.x * p.scale; o[x][1] *= w.y * p.scale; o[x][2] *= w.x * p.scale; o[x][3] *= w.y * p.scale;
      }
      __syncthreads();                                // weighted scores, their row sums and q · n are there
      for (int t = tid; t < L; t += blockDim.x) {
        float den = r_start[t] * p.scale * s_qn[t];
        for (int c = 0; c <= t >> 4; ++c) den += s_rs[c * L + t];
        s_inv[t] = 1.f / (fmaxf(fabsf(den), r_floor[t]) + 1e-6f);
      }
    }
    // the state decays; then, sixteen tokens at a time, Vᵀ meets the weighted scores and, weighted itself, K
    const float keep = s_keep[par];
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[n][e] *= keep;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t va[4];                                 // Vᵀ: [16 columns, 16 tokens]
      ldsm4t(va, s_v + (ks * 16 + tok) * VPITCH + warp * 16 + kc);
      if constexpr (!PART) {
#pragma unroll
        for (int tg = ks; tg < 4; ++tg) {
          uint32_t ph[4], pl[4];
          ldsm4(ph, s_ph + (tg * 16 + tok) * PP + ks * 16 + kc);
          ldsm4(pl, s_pl + (tg * 16 + tok) * PP + ks * 16 + kc);
          mma(o[2 * tg], va, ph[0], ph[1]);
          mma(o[2 * tg + 1], va, ph[2], ph[3]);
          mma(o[2 * tg], va, pl[0], pl[1]);
          mma(o[2 * tg + 1], va, pl[2], pl[3]);
        }
      }
      uint32_t vh[4], vl[4];
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const float2 v = unpack_bf16(va[x]), w = *reinterpret_cast<const float2*>(r_end + ks * 16 + (x >> 1) * 8 + tq * 2);
        split2(v.x * w.x, v.y * w.y, vh[x], vl[x]);
      }
#pragma unroll
      for (int s = 0; s < DP / 16; ++s) {
        uint32_t kb[4];
        ldsm4t(kb, s_k + (ks * 16 + kc + (lane & 7)) * PITCH + s * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          mma(S[2 * s + h], vh, kb[2 * h], kb[2 * h + 1]);
          mma(S[2 * s + h], vl, kb[2 * h], kb[2 * h + 1]);
        }
      }
    }
    for (int d = tid; d < DP; d += blockDim.x) {
      float n = keep * s_n[d];
#pragma unroll 8
      for (int s = 0; s < L; ++s) n = fmaf(r_end[s], to_f(s_k[s * PITCH + d]), n);
      s_n[d] = n;
    }
    if constexpr (!PART) {
      if (p.raw == nullptr) {
#pragma unroll
        for (int x = 0; x < 8; ++x)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            float ss = o[x][e] * o[x][e] + o[x][e + 2] * o[x][e + 2];       // columns past the head's are zero
            ss += __shfl_xor_sync(0xffffffffu, ss, 4);
            ss += __shfl_xor_sync(0xffffffffu, ss, 8);
            ss += __shfl_xor_sync(0xffffffffu, ss, 16);
            if (g == 0) s_ss[warp * L + x * 8 + tq * 2 + e] = ss;
          }
      }
      __syncthreads();                                // q and k have been read; denominators and sums of squares are there
      float* s_o = reinterpret_cast<float*>(base);
#pragma unroll
      for (int x = 0; x < 8; ++x)
#pragma unroll
        for (int e = 0; e < 4; ++e) s_o[(x * 8 + tq * 2 + (e & 1)) * OP + (e < 2 ? v_lo : v_hi)] = o[x][e];
      __syncthreads();
      const int n = min(L, b - t0);
      for (int t = warp; t < n; t += warps) {
        const size_t row = static_cast<size_t>(s0 + t0 + t) * p.H * p.vdim + static_cast<size_t>(head) * p.vdim + col0;
        float f = s_inv[t];
        if (p.raw != nullptr) {
          for (int c = lane; c < ncol; c += 32) p.raw[row + c] = s_o[t * OP + c] * f;
          continue;
        }
        float ss = 0.f;
        for (int w = 0; w < warps; ++w) ss += s_ss[w * L + t];
        f *= rsqrtf(ss * f * f / p.vdim + p.eps);
        for (int c = lane * 2; c < ncol; c += 64) {
          const float2 x = *reinterpret_cast<const float2*>(s_o + t * OP + c), z = unpack_bf16(*reinterpret_cast<const uint32_t*>(s_g + t * VPITCH + c)),
                       w = unpack_bf16(*reinterpret_cast<const uint32_t*>(p.weight + static_cast<size_t>(head) * p.vdim + col0 + c));
          *reinterpret_cast<uint32_t*>(p.o + row + c) = pack_bf16(x.x * f * w.x * sigmoid_of(z.x), x.y * f * w.y * sigmoid_of(z.y));
        }
      }
      // outputs lay where columns past the head's width must be zero
      if (t0 + L < b && p.dim < DP) {
        __syncthreads();
        for (int i = tid; i < lay.qk / 16; i += blockDim.x) reinterpret_cast<uint4*>(base)[i] = make_uint4(0u, 0u, 0u, 0u);
      }
    }
    if (p.stages != 2 && t0 + L < b) {
      __syncthreads();
      fetch(t0 + L, 0);
    }
    st = next;
  }
  __syncthreads();
  float* out = nullptr;
  if constexpr (PART) {
    out = p.part + ((static_cast<size_t>(seq) * (p.segments - 1) + seg) * p.H + head) * p.pool_ld;
  } else if (p.pool != nullptr && b == len) {
    const int sl = p.slot[s0];
    if (sl > 0) out = p.pool + (static_cast<size_t>(sl) * p.H + head) * p.pool_ld;
  }
  if (out == nullptr) return;
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = n * 8 + tq * 2 + (e & 1), c = e < 2 ? v_lo : v_hi;
      if (r < p.dim && c < ncol) out[static_cast<size_t>(r) * p.vdim + col0 + c] = S[n][e];
    }
  if (slice != 0) return;
  for (int d = tid; d < p.dim; d += blockDim.x) out[p.n0 + d] = s_n[d];
  if (keeper && lane == 0) {
    out[p.m0] = m_run;
    if constexpr (PART) out[p.m0 + 1] = f_total;
  }
}

// Norm, weight and gate of raw outputs: one warp per token and head.
template <typename T>
__global__ void __launch_bounds__(256) mlstm_finish_kernel(const Mlstm<T> p) {
  const long i = blockIdx.x * 8L + (threadIdx.x >> 5);
  if (i >= static_cast<long>(p.rows) * p.H) return;
  const int lane = threadIdx.x & 31;
  const size_t row = i / p.H;
  const int head = static_cast<int>(i - row * p.H);
  const size_t at = row * p.H * p.vdim + static_cast<size_t>(head) * p.vdim;
  float ss = 0.f;
  for (int c = lane; c < p.vdim; c += 32) ss += p.raw[at + c] * p.raw[at + c];
  const float r = rsqrtf(warp_sum(ss) / p.vdim + p.eps);
  for (int c = lane; c < p.vdim; c += 32)
    p.o[at + c] = from_f<T>(p.raw[at + c] * r * to_f(p.weight[head * p.vdim + c]) * sigmoid_of(to_f(p.g[row * p.ld + static_cast<size_t>(head) * p.vdim + c])));
}

// One block per (head, sequence).  V columns per access.
template <typename T, int V>
__global__ void __launch_bounds__(256) mlstm_step_kernel(const Mlstm<T> p) {
  extern __shared__ __align__(16) float sm_step[];
  __shared__ float sh[32], sh2[32];
  float *s_q = sm_step, *s_k = s_q + p.dim, *s_red = s_k + p.dim;        // [dim], [dim], [row groups][vdim]
  const int head = blockIdx.x, row = blockIdx.y, tid = threadIdx.x, slot = p.slot[row];
  const size_t base = static_cast<size_t>(row) * p.ld;
  float* S = p.pool + (static_cast<size_t>(slot) * p.H + head) * p.pool_ld;
  float i, f;
  mlstm_gates(p, static_cast<size_t>(row), head, i, f);
  const float m = S[p.m0], top = fmaxf(f + m, i), keep = __expf(f + m - top), add = __expf(i - top);
  float dot = 0.f;
  for (int r = tid; r < p.dim; r += 256) {
    const float q = to_f(p.q[base + static_cast<size_t>(head) * p.dim + r]) * p.scale, k = to_f(p.k[base + static_cast<size_t>(head) * p.dim + r]);
    s_q[r] = q;
    s_k[r] = k;
    const float n = fmaf(add, k, keep * S[p.n0 + r]);
    if (slot > 0) S[p.n0 + r] = n;
    dot = fmaf(n, q, dot);
  }
  dot = block_sum(dot, sh);                                             // (with barriers: s_q and s_k are there, m has been read)
  if (tid == 0 && slot > 0) S[p.m0] = top;
  const int per_row = p.vdim / V, groups = max(1, min(256 / per_row, p.dim));
  for (int x0 = 0; x0 < per_row; x0 += 256) {                            // heads wider than the block take several rounds
    const int x = x0 + tid % min(per_row, 256), group = tid / min(per_row, 256);
    if (x < per_row && group < groups) {
      const T* vp = p.v + base + static_cast<size_t>(head) * p.vdim + x * V;
      float av[V], o[V];
#pragma unroll
      for (int j = 0; j < V; ++j) {
        av[j] = add * to_f(vp[j]);
        o[j] = 0.f;
      }
      constexpr int U = 8;                                                // rows on their way at a time
      for (int rb = group; rb < p.dim; rb += groups * U) {
        float s[U][V];
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int r = rb + u * groups;
          if (r >= p.dim) continue;
          const float* at = S + static_cast<size_t>(r) * p.vdim + x * V;
          if constexpr (V == 4) {
            const float4 w = *reinterpret_cast<const float4*>(at);
            s[u][0] = w.x; s[u][1] = w.y; s[u][2] = w.z; s[u][3] = w.w;
          } else {
            s[u][0] = *at;
          }
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int r = rb + u * groups;
          if (r >= p.dim) continue;
          float* at = S + static_cast<size_t>(r) * p.vdim + x * V;
          const float q = s_q[r], k = s_k[r];
#pragma unroll
          for (int j = 0; j < V; ++j) {
            s[u][j] = fmaf(k, av[j], keep * s[u][j]);
            o[j] = fmaf(q, s[u][j], o[j]);
          }
          if (slot > 0) {
            if constexpr (V == 4) *reinterpret_cast<float4*>(at) = make_float4(s[u][0], s[u][1], s[u][2], s[u][3]);
            else *at = s[u][0];
          }
        }
      }
#pragma unroll
      for (int j = 0; j < V; ++j) s_red[group * p.vdim + x * V + j] = o[j];
    }
  }
  __syncthreads();
  const float inv = 1.f / (fmaxf(fabsf(dot), __expf(-top)) + 1e-6f);
  float ss = 0.f;
  for (int c = tid; c < p.vdim; c += 256) {
    float o = 0.f;
    for (int gr = 0; gr < groups; ++gr) o += s_red[gr * p.vdim + c];
    o *= inv;
    s_red[c] = o;                                                       // (this thread alone reads column c)
    ss += o * o;
  }
  const float r = rsqrtf(block_sum(ss, sh2) / p.vdim + p.eps);
  for (int c = tid; c < p.vdim; c += 256)
    p.o[static_cast<size_t>(row) * p.H * p.vdim + static_cast<size_t>(head) * p.vdim + c] =
        from_f<T>(s_red[c] * r * to_f(p.weight[head * p.vdim + c]) * sigmoid_of(to_f(p.g[base + static_cast<size_t>(head) * p.vdim + c])));
}

template <typename T>
static Mlstm<T> mlstm_params(const torch::Tensor& proj, int64_t first, int64_t H, int64_t dim, int64_t vdim, const torch::Tensor& i_bias, const torch::Tensor& f_bias, double cap,
                             const torch::Tensor& weight, double eps, torch::Tensor& o) {
  Mlstm<T> p{};
  const T* base = reinterpret_cast<const T*>(proj.data_ptr()) + first;
  p.q = base; p.k = p.q + H * dim; p.v = p.k + H * dim; p.g = p.v + H * vdim; p.i = p.g + H * vdim; p.f = p.i + H; p.ld = proj.stride(0);
  p.i_bias = reinterpret_cast<const T*>(i_bias.data_ptr()); p.f_bias = reinterpret_cast<const T*>(f_bias.data_ptr()); p.weight = reinterpret_cast<const T*>(weight.data_ptr());
  p.o = reinterpret_cast<T*>(o.data_ptr());
  p.H = H; p.dim = dim; p.vdim = vdim; p.n0 = (dim * vdim + 3) / 4 * 4; p.m0 = p.n0 + (dim + 3) / 4 * 4; p.pool_ld = p.m0 + 4; p.rows = proj.size(0);
  p.cap = cap; p.inv_cap = static_cast<float>(1.0 / cap); p.eps = eps; p.scale = static_cast<float>(1.0 / std::sqrt(static_cast<double>(dim)));
  return p;
}

static void mlstm_check(const torch::Tensor& proj, int64_t first, int64_t H, int64_t dim, int64_t vdim, const torch::Tensor& i_bias, const torch::Tensor& f_bias, double cap,
                        const torch::Tensor& weight) {
  const auto st = proj.scalar_type();
  TORCH_CHECK(proj.is_cuda() && proj.dim() == 2 && proj.stride(1) == 1 && (st == torch::kBFloat16 || st == torch::kFloat32), "proj [rows, N] bf16 or fp32");
  TORCH_CHECK(H > 0 && dim > 0 && vdim > 0 && dim <= 256 && vdim <= 4096 && cap > 0, "heads up to 256 × 4096, a positive cap");
  TORCH_CHECK(first >= 0 && first + 2 * H * (dim + vdim + 1) <= proj.size(1), "columns outside the projection");
  for (const auto* t : {&i_bias, &f_bias}) TORCH_CHECK(t->scalar_type() == st && t->is_contiguous() && t->numel() == H, "gate biases [heads]");
  TORCH_CHECK(weight.scalar_type() == st && weight.is_contiguous() && weight.numel() == H * vdim, "norm weight [heads * vdim]");
}

static void mlstm_check_pool(const torch::Tensor& pool, int64_t H, int64_t dim, int64_t vdim, const torch::Tensor& slot, int64_t rows) {
  TORCH_CHECK(pool.is_cuda() && pool.scalar_type() == torch::kFloat32 && pool.is_contiguous() && pool.dim() == 3 && pool.size(1) == H &&
                  pool.size(2) == (dim * vdim + 3) / 4 * 4 + (dim + 3) / 4 * 4 + 4, "states [slots, heads, matrix | normaliser | maximum] fp32");
  TORCH_CHECK(slot.scalar_type() == torch::kInt32 && slot.is_contiguous() && slot.numel() == rows, "slots int32 [rows]");
}

torch::Tensor mlstm_prefill(const torch::Tensor& proj, int64_t first, int64_t H, int64_t dim, int64_t vdim, const torch::Tensor& i_bias, const torch::Tensor& f_bias, double cap,
                            const torch::Tensor& weight, double eps, const torch::Tensor& cu, int64_t max_seqlen, const OptT& pool, const OptT& slot) {
  mlstm_check(proj, first, H, dim, vdim, i_bias, f_bias, cap, weight);
  TORCH_CHECK(cu.is_cuda() && cu.scalar_type() == torch::kInt32 && cu.is_contiguous() && cu.numel() >= 1, "cu_seqlens int32 on device");
  const int64_t rows = proj.size(0), n = cu.numel() - 1;
  if (has(pool)) {
    TORCH_CHECK(has(slot), "states come with slots");
    mlstm_check_pool(*pool, H, dim, vdim, *slot, rows);
  }
  c10::cuda::CUDAGuard guard(proj.device());
  auto o = torch::empty({rows, H * vdim}, proj.options());
  if (rows == 0 || n == 0 || max_seqlen <= 0) return o;
  auto stream = at::cuda::getCurrentCUDAStream();
  auto run = [&](auto tag) {
    using T = decltype(tag);
    auto p = mlstm_params<T>(proj, first, H, dim, vdim, i_bias, f_bias, cap, weight, eps, o);
    p.cu = cu.data_ptr<int>();
    if (has(pool)) { p.pool = pool->data_ptr<float>(); p.slot = slot->data_ptr<int>(); }
    torch::Tensor raw, part;
    auto f32 = proj.options().dtype(torch::kFloat32);
    if constexpr (sizeof(T) == 2) {
      const bool whole = dim % 8 == 0 && vdim % 8 == 0 && p.ld % 8 == 0 && aligned16(p.q) && aligned16(p.k) && aligned16(p.v) && aligned16(p.g) &&
                         reinterpret_cast<uintptr_t>(p.weight) % 4 == 0;
      if (whole && n <= 65535) {
        p.slices = static_cast<int>((vdim + 127) / 128);
        p.cols = p.slices == 1 ? vdim : static_cast<int>((vdim / 8 + p.slices - 1) / p.slices * 8);
        if (p.slices > 1) { raw = torch::empty({rows, H * vdim}, f32); p.raw = raw.data_ptr<float>(); }
        const int DP = dim <= 32 ? 32 : (dim <= 64 ? 64 : (dim <= 128 ? 128 : 256)), warps = (p.cols + 15) / 16;
        // time segments: as many as fill the device, none shorter than 256 tokens (a segment costs a second pass over its state)
        const int64_t blocks = H * p.slices * n;
        const int64_t segs = std::max<int64_t>(1, std::min<int64_t>(num_sms() / blocks, max_seqlen / 256));
        p.seg_len = static_cast<int>(((max_seqlen + segs - 1) / segs + ml::L - 1) / ml::L * ml::L);
        p.segments = static_cast<int>((max_seqlen + p.seg_len - 1) / p.seg_len);
        if (p.segments > 1) { part = torch::empty({n * (p.segments - 1) * H * p.pool_ld}, f32); p.part = part.data_ptr<float>(); }
        p.stages = 2;
        if (ml::Layout(DP, warps * 16, 2).total > 227 * 1024) p.stages = 1;
        const int smem = ml::Layout(DP, warps * 16, p.stages).total;
        auto go = [&](auto kern, int segments) {
          TK_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
          kern<<<dim3(H * p.slices, segments, n), 32 * warps, smem, stream>>>(p);
          count_launch();
        };
        if (p.segments > 1) {
          if (DP == 32) go(mlstm_chunk_kernel<32, true>, p.segments - 1);
          else if (DP == 64) go(mlstm_chunk_kernel<64, true>, p.segments - 1);
          else if (DP == 128) go(mlstm_chunk_kernel<128, true>, p.segments - 1);
          else go(mlstm_chunk_kernel<256, true>, p.segments - 1);
        }
        if (DP == 32) go(mlstm_chunk_kernel<32, false>, p.segments);
        else if (DP == 64) go(mlstm_chunk_kernel<64, false>, p.segments);
        else if (DP == 128) go(mlstm_chunk_kernel<128, false>, p.segments);
        else go(mlstm_chunk_kernel<256, false>, p.segments);
        if (p.raw != nullptr) {
          mlstm_finish_kernel<T><<<static_cast<unsigned>((rows * H + 7) / 8), 256, 0, stream>>>(p);
          count_launch();
        }
        return;
      }
    }
    raw = torch::empty({rows, H * vdim}, f32);
    p.raw = raw.data_ptr<float>();
    auto go = [&](auto kern, int RPT, int RS) {
      const int slots = 256 / RS;
      p.slices = static_cast<int>((vdim + slots - 2) / (slots - 1));
      p.cols = (vdim + p.slices - 1) / p.slices;
      const int smem = static_cast<int>(sizeof(float)) * ml::CH * (2 * RPT * RS + slots);
      TK_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
      kern<<<dim3(H * p.slices, 1, n), 256, smem, stream>>>(p);
    };
    if (dim <= 32) go(mlstm_prefill_kernel<T, 32, 1>, 32, 1);
    else if (dim <= 64) go(mlstm_prefill_kernel<T, 32, 2>, 32, 2);
    else if (dim <= 128) go(mlstm_prefill_kernel<T, 32, 4>, 32, 4);
    else go(mlstm_prefill_kernel<T, 32, 8>, 32, 8);
    count_launch();
    mlstm_finish_kernel<T><<<static_cast<unsigned>((rows * H + 7) / 8), 256, 0, stream>>>(p);
    count_launch();
  };
  if (proj.scalar_type() == torch::kBFloat16) run(bf16{}); else run(float{});
  TK_CUDA_CHECK(cudaGetLastError());
  return o;
}

torch::Tensor mlstm_step(const torch::Tensor& proj, int64_t first, int64_t H, int64_t dim, int64_t vdim, const torch::Tensor& i_bias, const torch::Tensor& f_bias, double cap,
                         const torch::Tensor& weight, double eps, const torch::Tensor& pool, const torch::Tensor& slot) {
  mlstm_check(proj, first, H, dim, vdim, i_bias, f_bias, cap, weight);
  const int64_t rows = proj.size(0);
  mlstm_check_pool(pool, H, dim, vdim, slot, rows);
  TORCH_CHECK(rows <= 65535, "too many rows in one call");
  c10::cuda::CUDAGuard guard(proj.device());
  auto o = torch::empty({rows, H * vdim}, proj.options());
  if (rows == 0) return o;
  auto stream = at::cuda::getCurrentCUDAStream();
  auto run = [&](auto tag) {
    using T = decltype(tag);
    auto p = mlstm_params<T>(proj, first, H, dim, vdim, i_bias, f_bias, cap, weight, eps, o);
    p.pool = pool.data_ptr<float>(); p.slot = slot.data_ptr<int>();
    auto go = [&](auto kern, int V) {
      const int per_row = static_cast<int>(vdim) / V, groups = std::max(1, std::min<int>(256 / per_row, dim));
      const int smem = static_cast<int>(sizeof(float)) * static_cast<int>(2 * dim + groups * vdim);
      TK_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
      kern<<<dim3(H, rows), 256, smem, stream>>>(p);
    };
    if (vdim % 4 == 0) go(mlstm_step_kernel<T, 4>, 4); else go(mlstm_step_kernel<T, 1>, 1);
  };
  if (proj.scalar_type() == torch::kBFloat16) run(bf16{}); else run(float{});
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return o;
}

}  // namespace tk
