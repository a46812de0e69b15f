// Selective scan (Mamba) between its projections.
//   conv_silu          causal depth-wise convolution, bias and silu on columns of a projection; the last inputs of a sequence stay in a ring
//                      over positions, from which single steps take their past
//   selective_prefill  packed prompts.  Per channel c and state n, in fp32:
//                          δ = softplus(dt + b),  S ← e^{−δ e^{A}} S + δ u B,  y = (Σ_n S C + D u) silu(z)
//                      LN neighbouring lanes share a channel, NS states each in registers; tokens pass through shared memory sixteen (with many states, eight) at a
//                      time, the next ones on their way while these are worked on.  When sequences × channels do not fill the device,
//                      sequences are cut into time segments: a first pass forms what each segment builds up from nothing and its sum of
//                      steps (decays multiply, so the steps add up), and the second starts every segment from those before it.
//   selective_step     one token of every sequence: the state passes once through the block, 16 bytes per access.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/types.h>

#include "common.cuh"
#include "host.h"
#include "vec.cuh"

namespace tk {

// ------------------------------------------------------------------- conv_silu
template <typename T>
struct ConvSilu {
  const T* x; long ld;
  const T *w, *bias;                   // [C, taps], [C]
  T* out;                              // [rows, C]
  const int64_t* pos;
  T* hist; const int *slot, *left;     // [slots, taps − 1, C] (null: not kept)
  int C, taps, rows, tile;
  bool step;
};

__device__ __forceinline__ float silu_of(float z) { return __fdividef(z, 1.f + __expf(-z)); }

// A thread owns eight channels of `tile` consecutive rows and keeps the last TAPS − 1 inputs in registers; four rows are on their way at a time.
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) conv_silu_kernel(const ConvSilu<T> p) {
  constexpr int N = TAPS > 1 ? TAPS - 1 : 1, U = 4;      // rows of the ring, rows fetched together
  const int c = (blockIdx.x * 128 + threadIdx.x) * 8;
  if (c >= p.C) return;
  const int t0 = blockIdx.y * p.tile, t1 = min(p.rows, t0 + p.tile);
  float w[TAPS][8], b[8], past[N][8];
  Raw8<T> r;
  r.load(p.bias + c);
  r.get(b);
#pragma unroll
  for (int v = 0; v < TAPS; ++v) {                       // the filters of eight channels are TAPS whole vectors
    float f[8];
    r.load(p.w + static_cast<size_t>(c) * TAPS + v * 8);
    r.get(f);
#pragma unroll
    for (int i = 0; i < 8; ++i) w[(v * 8 + i) % TAPS][(v * 8 + i) / TAPS] = f[i];
  }
  auto load = [&](const T* src, float (&y)[8]) {
    Raw8<T> q;
    q.load(src);
    q.get(y);
  };
  const int first = static_cast<int>(min(p.pos[t0], static_cast<int64_t>(TAPS)));      // inputs of the same sequence before the tile's first row
#pragma unroll
  for (int j = 1; j < TAPS; ++j) {
#pragma unroll
    for (int i = 0; i < 8; ++i) past[j - 1][i] = 0.f;
    if (!p.step && j <= first) load(p.x + static_cast<size_t>(t0 - j) * p.ld + c, past[j - 1]);
  }
  const bool keeps = TAPS > 1 && p.hist != nullptr;
  for (int tb = t0; tb < t1; tb += U) {
    Raw8<T> raw[U];
    int64_t pos[U];
    int left[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (tb + u >= t1) continue;
      raw[u].load(p.x + static_cast<size_t>(tb + u) * p.ld + c);
      pos[u] = p.pos[tb + u];
      left[u] = keeps ? p.left[tb + u] : TAPS;
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int t = tb + u;
      if (t >= t1) continue;
      const bool store = keeps && left[u] < TAPS - 1;
      T* ring = nullptr;
      int slot = 0;
      if (keeps && (store || p.step)) {
        slot = p.slot[t];
        ring = p.hist + static_cast<size_t>(slot) * N * p.C + c;
      }
      float x[8], y[8];
      raw[u].get(x);
#pragma unroll
      for (int i = 0; i < 8; ++i) y[i] = fmaf(w[TAPS - 1][i], x[i], b[i]);
#pragma unroll
      for (int j = 1; j < TAPS; ++j) {
        if (pos[u] < j) continue;
        if (p.step) load(ring + static_cast<size_t>((pos[u] - j) % N) * p.C, past[j - 1]);
#pragma unroll
        for (int i = 0; i < 8; ++i) y[i] = fmaf(w[TAPS - 1 - j][i], past[j - 1][i], y[i]);
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) y[i] = silu_of(y[i]);
      r.set(y);
      r.store(p.out + static_cast<size_t>(t) * p.C + c);
      if constexpr (TAPS > 1) {
        if (store && slot > 0) raw[u].store(ring + static_cast<size_t>(pos[u] % N) * p.C);
#pragma unroll
        for (int j = TAPS - 2; j > 0; --j)
#pragma unroll
          for (int i = 0; i < 8; ++i) past[j][i] = past[j - 1][i];
#pragma unroll
        for (int i = 0; i < 8; ++i) past[0][i] = x[i];
      }
    }
  }
}

// Any sizes: one thread per element.
template <typename T>
__global__ void __launch_bounds__(256) conv_silu_any_kernel(const ConvSilu<T> p) {
  const long i = blockIdx.x * 256L + threadIdx.x;
  if (i >= static_cast<long>(p.rows) * p.C) return;
  const int t = static_cast<int>(i / p.C), c = static_cast<int>(i - static_cast<long>(t) * p.C), n = p.taps - 1;
  const int64_t pos = p.pos[t];
  const int slot = p.hist != nullptr ? p.slot[t] : 0;
  T* ring = p.hist != nullptr ? p.hist + static_cast<size_t>(slot) * n * p.C + c : nullptr;
  const T own = p.x[static_cast<size_t>(t) * p.ld + c];
  float y = to_f(p.bias[c]) + to_f(p.w[static_cast<size_t>(c) * p.taps + n]) * to_f(own);
  for (int j = 1; j <= n && j <= pos; ++j)
    y += to_f(p.w[static_cast<size_t>(c) * p.taps + n - j]) * to_f(p.step ? ring[static_cast<size_t>((pos - j) % n) * p.C] : p.x[static_cast<size_t>(t - j) * p.ld + c]);
  p.out[i] = from_f<T>(silu_of(y));
  if (ring != nullptr && slot > 0 && p.left[t] < n) ring[static_cast<size_t>(pos % n) * p.C] = own;
}

// Columns first … first + C of proj [rows, N]; pos [rows] counts from each sequence's start.  hist [slots, taps − 1, C]: kept inputs.
torch::Tensor conv_silu(const torch::Tensor& proj, int64_t first, const torch::Tensor& w, const torch::Tensor& bias, const torch::Tensor& pos, bool step, const OptT& hist,
                        const OptT& slot, const OptT& left) {
  const auto st = proj.scalar_type();
  TORCH_CHECK(proj.is_cuda() && proj.dim() == 2 && proj.stride(1) == 1 && (st == torch::kBFloat16 || st == torch::kFloat32), "proj [rows, N] bf16 or fp32");
  TORCH_CHECK(w.dim() == 2 && w.scalar_type() == st && w.is_contiguous() && bias.scalar_type() == st && bias.is_contiguous() && bias.numel() == w.size(0), "filters [C, taps], bias [C]");
  const int64_t rows = proj.size(0), C = w.size(0), taps = w.size(1);
  TORCH_CHECK(taps >= 1 && taps <= 1024 && first >= 0 && first + C <= proj.size(1), "columns outside the projection, or no taps");
  TORCH_CHECK(pos.is_cuda() && pos.scalar_type() == torch::kInt64 && pos.is_contiguous() && pos.numel() == rows, "positions int64 [rows]");
  if (has(hist)) {
    TORCH_CHECK(hist->is_cuda() && hist->scalar_type() == st && hist->is_contiguous() && hist->dim() == 3 && hist->size(1) == taps - 1 && hist->size(2) == C, "history [slots, taps - 1, C]");
    TORCH_CHECK(has(slot) && has(left) && slot->scalar_type() == torch::kInt32 && left->scalar_type() == torch::kInt32 && slot->is_contiguous() && left->is_contiguous() &&
                    slot->numel() == rows && left->numel() == rows, "slots and rows left int32 [rows]");
  }
  TORCH_CHECK(!step || taps == 1 || has(hist), "single steps take their past from the history");
  c10::cuda::CUDAGuard guard(proj.device());
  auto out = torch::empty({rows, C}, proj.options());
  if (rows == 0) return out;
  auto stream = at::cuda::getCurrentCUDAStream();
  auto run = [&](auto tag) {
    using T = decltype(tag);
    ConvSilu<T> p{};
    p.x = reinterpret_cast<const T*>(proj.data_ptr()) + first; p.ld = proj.stride(0);
    p.w = reinterpret_cast<const T*>(w.data_ptr()); p.bias = reinterpret_cast<const T*>(bias.data_ptr()); p.out = reinterpret_cast<T*>(out.data_ptr());
    p.pos = pos.data_ptr<int64_t>();
    if (has(hist)) { p.hist = reinterpret_cast<T*>(hist->data_ptr()); p.slot = slot->data_ptr<int>(); p.left = left->data_ptr<int>(); }
    p.C = C; p.taps = taps; p.rows = rows; p.step = step;
    const bool vec = C % 8 == 0 && p.ld % 8 == 0 && aligned16(p.x) && aligned16(p.bias) && aligned16(p.w) && aligned16(p.out) && aligned16(p.hist) && taps <= 5;
    if (!vec) {
      conv_silu_any_kernel<T><<<static_cast<unsigned>((rows * C + 255) / 256), 256, 0, stream>>>(p);
      return;
    }
    const int across = static_cast<int>((C / 8 + 127) / 128);
    // sixteen rows per thread once that leaves blocks enough; single steps have nothing to share between rows
    p.tile = step ? 1 : static_cast<int>(std::min<int64_t>(16, std::max<int64_t>(1, rows * across / (num_sms() * 8))));
    const dim3 grid(across, static_cast<unsigned>((rows + p.tile - 1) / p.tile));
    TORCH_CHECK(grid.y <= 65535, "too many rows in one call");
    if (taps == 1) conv_silu_kernel<T, 1><<<grid, 128, 0, stream>>>(p);
    else if (taps == 2) conv_silu_kernel<T, 2><<<grid, 128, 0, stream>>>(p);
    else if (taps == 3) conv_silu_kernel<T, 3><<<grid, 128, 0, stream>>>(p);
    else if (taps == 4) conv_silu_kernel<T, 4><<<grid, 128, 0, stream>>>(p);
    else conv_silu_kernel<T, 5><<<grid, 128, 0, stream>>>(p);
  };
  if (st == torch::kBFloat16) run(bf16{}); else run(float{});
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return out;
}

// -------------------------------------------------------------- selective scan
template <typename T>
struct Selective {
  const T *u, *dt, *z; long ldd, ldz;            // [rows, C] with row strides C, ldd, ldz
  const T *B, *Cm; long ldb;                     // [rows, N]
  const T *dt_bias, *A_log, *D;                  // [C], [C, N], [C]
  T* y;                                          // [rows, C]
  const int* cu;
  float* pool; const int* slot;                  // [slots, C, N] (null: last states are not kept)
  float *part, *steps;                           // [n, segments − 1, C, N], [n, segments − 1, C]
  int C, N, seg_len, segments;
};

// ln(1 + e^x) = max(x, 0) + 2 artanh(e / (2 + e)) with e = e^−|x| ≤ 1: odd series of artanh up to the 13th power, relative error 1e-7
__device__ __forceinline__ float softplus_of(float x) {
  const float e = __expf(-fabsf(x)), s = __fdividef(e, 2.f + e), v = s * s;
  float r = fmaf(v, 2.f / 13.f, 2.f / 11.f);
  r = fmaf(v, r, 2.f / 9.f);
  r = fmaf(v, r, 2.f / 7.f);
  r = fmaf(v, r, 2.f / 5.f);
  r = fmaf(v, r, 2.f / 3.f);
  r = fmaf(v, r, 2.f);
  return fmaf(s, r, fmaxf(x, 0.f));
}

// two fp32 operations per instruction
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
  float2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(reinterpret_cast<uint64_t&>(d)) : "l"(reinterpret_cast<uint64_t&>(a)), "l"(reinterpret_cast<uint64_t&>(b)));
  return d;
}
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  float2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(reinterpret_cast<uint64_t&>(d)) : "l"(reinterpret_cast<uint64_t&>(a)), "l"(reinterpret_cast<uint64_t&>(b)), "l"(reinterpret_cast<uint64_t&>(c)));
  return d;
}
__device__ __forceinline__ float2 both(float x) { return make_float2(x, x); }

namespace sel {
constexpr int THREADS = 128;
constexpr int tokens(int states) { return states > 128 ? 8 : 16; }      // per round
}

// V neighbouring elements as they lie in memory
template <typename T, int V> struct Few { T v[V]; };
template <> struct alignas(4) Few<bf16, 2> { bf16 v[2]; };
template <> struct alignas(8) Few<float, 2> { float v[2]; };
template <> struct alignas(8) Few<bf16, 4> { bf16 v[4]; };
template <> struct alignas(16) Few<float, 4> { float v[4]; };

// NS states per lane, LN lanes per channel, V channels per access.  PART: only the state a segment builds up from nothing and its sum of steps.
template <typename T, int NS, int LN, int V, bool PART>
__global__ void __launch_bounds__(sel::THREADS, NS == 4 ? 6 : 5) selective_prefill_kernel(const Selective<T> p) {
  using namespace sel;
  constexpr int CH = THREADS / LN, NP = NS * LN, TOK = tokens(NP);       // channels of a block, states filled up, tokens of a round
  constexpr int COLS = CH / V, ROWS = THREADS / COLS, PER = TOK > ROWS ? TOK / ROWS : 1;      // staging: a thread has V channels of every ROWS-th row
  __shared__ __align__(16) float2 s_du[2][TOK][CH];                      // step, step times input
  __shared__ __align__(16) float s_y[TOK][CH + 4], s_b[2][TOK][NP], s_c[2][TOK][NP];
  const int seg = blockIdx.y, seq = blockIdx.z, c0 = blockIdx.x * CH;
  const int s0 = p.cu[seq], len = p.cu[seq + 1] - s0, a = seg * p.seg_len, b = min(len, a + p.seg_len);
  if (a >= len || (PART && b >= len)) return;         // the last segment of a sequence is nobody's past
  const int tid = threadIdx.x, sub = tid % LN, ch = tid / LN, c = c0 + ch;
  const bool mine = c < p.C;
  // A in log2 units; states that fill up the lanes neither decay nor take anything in
  float2 A2[NS / 2], S2[NS / 2];
  float *A = reinterpret_cast<float*>(A2), *S = reinterpret_cast<float*>(S2);
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const int n = sub * NS + i;
    A[i] = mine && n < p.N ? -__expf(to_f(p.A_log[static_cast<size_t>(c) * p.N + n])) * 1.4426950408889634f : 0.f;
    S[i] = 0.f;
  }
  if constexpr (!PART) {
    // what the segments before this one leave behind
    for (int k = 0; k < seg; ++k) {
      const size_t at = (static_cast<size_t>(seq) * (p.segments - 1) + k) * p.C + c;
      if (mine) {
        const float d = p.steps[at];
#pragma unroll
        for (int i = 0; i < NS; ++i) {
          const int n = sub * NS + i;
          if (n < p.N) S[i] = fmaf(fast_exp2(d * A[i]), S[i], p.part[at * p.N + n]);
        }
      }
    }
  }
  // staging
  const int sc = tid % COLS * V, sr = tid / COLS, gc = c0 + sc;
  const bool column = gc < p.C && sr < TOK;           // (V divides the number of channels)
  float dt_bias[V], skip[V];
#pragma unroll
  for (int v = 0; v < V; ++v) {
    dt_bias[v] = column ? to_f(p.dt_bias[gc + v]) : 0.f;
    skip[v] = !PART && column ? to_f(p.D[gc + v]) : 0.f;
  }
  using F = Few<T, V>;
  F zero;
#pragma unroll
  for (int v = 0; v < V; ++v) zero.v[v] = from_f<T>(0.f);
  const size_t at0 = static_cast<size_t>(s0 + a + sr);
  const T *pu = p.u + at0 * p.C + gc, *pd = p.dt + at0 * p.ldd + gc, *pz = p.z + at0 * p.ldz + gc;
  const long su = static_cast<long>(ROWS) * p.C, sd = ROWS * p.ldd, sz = ROWS * p.ldz;
  T* py = p.y + at0 * p.C + gc;
  // B and C: a thread has the same state of every BROWS-th row
  constexpr int BROWS = 2 * NP >= THREADS ? 1 : THREADS / (2 * NP), BCOLS = 2 * NP > THREADS ? 2 * NP / THREADS : 1, BPER = TOK > BROWS ? TOK / BROWS : 1;
  const int bn = tid % (2 * NP), br = tid / (2 * NP);
  const T* pb = p.B + static_cast<size_t>(s0 + a + br) * p.ldb;
  const T* pc = p.Cm + static_cast<size_t>(s0 + a + br) * p.ldb;
  F r_u[PER], r_d[PER], r_z[PER];
  T r_b[BPER][BCOLS];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const bool in = column && t0 + sr + i * ROWS < b;
      r_u[i] = in ? *reinterpret_cast<const F*>(pu + i * su) : zero;
      r_d[i] = in ? *reinterpret_cast<const F*>(pd + i * sd) : zero;
      if constexpr (!PART) r_z[i] = in ? *reinterpret_cast<const F*>(pz + i * sz) : zero;
    }
    pu += static_cast<long>(TOK) * p.C; pd += TOK * p.ldd; pz += TOK * p.ldz;
#pragma unroll
    for (int i = 0; i < BPER; ++i) {
      const bool in = br + i * BROWS < TOK && t0 + br + i * BROWS < b;
#pragma unroll
      for (int k = 0; k < BCOLS; ++k) {
        const int n = bn + k * THREADS, m = n >= NP ? n - NP : n;
        r_b[i][k] = in && m < p.N ? (n >= NP ? pc : pb)[i * BROWS * p.ldb + m] : from_f<T>(0.f);
      }
    }
    pb += TOK * p.ldb; pc += TOK * p.ldb;
  };
  float total = 0.f;
  F u_now[PER], z_now[PER];
  auto stage = [&](int buf, int t0) {
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int r = sr + i * ROWS;
      u_now[i] = r_u[i];
      z_now[i] = r_z[i];
      if (r < TOK) {
#pragma unroll
        for (int v = 0; v < V; ++v) {
          const float d = t0 + r < b ? softplus_of(to_f(r_d[i].v[v]) + dt_bias[v]) : 0.f;      // rows past the end change nothing
          s_du[buf][r][sc + v] = make_float2(d, d * to_f(r_u[i].v[v]));
        }
      }
    }
#pragma unroll
    for (int i = 0; i < BPER; ++i) {
      const int r = br + i * BROWS;
      if (r < TOK) {
#pragma unroll
        for (int k = 0; k < BCOLS; ++k) {
          const int n = bn + k * THREADS;
          (n >= NP ? s_c[buf][r] - NP : s_b[buf][r])[n] = to_f(r_b[i][k]);
        }
      }
    }
  };
  fetch(a);
  int buf = 0;
  for (int t0 = a; t0 < b; t0 += TOK, buf ^= 1) {
    stage(buf, t0);
    __syncthreads();
    if (t0 + TOK < b) fetch(t0 + TOK);
#pragma unroll 1
    for (int t = 0; t < TOK; t += 4) {
      float y[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float2 du = s_du[buf][t + k][ch];
        if constexpr (PART) total += du.x;
        const float2 d2 = both(du.x), u2 = both(du.y);
        float2 y2 = make_float2(0.f, 0.f);
#pragma unroll
        for (int i = 0; i < NS / 2; i += 2) {
          const float4 b4 = *reinterpret_cast<const float4*>(&s_b[buf][t + k][sub * NS + 2 * i]);
          float2 e0 = mul2(d2, A2[i]), e1 = mul2(d2, A2[i + 1]);
          e0 = make_float2(fast_exp2(e0.x), fast_exp2(e0.y));
          e1 = make_float2(fast_exp2(e1.x), fast_exp2(e1.y));
          S2[i] = fma2(e0, S2[i], mul2(u2, make_float2(b4.x, b4.y)));
          S2[i + 1] = fma2(e1, S2[i + 1], mul2(u2, make_float2(b4.z, b4.w)));
          if constexpr (!PART) {
            const float4 c4 = *reinterpret_cast<const float4*>(&s_c[buf][t + k][sub * NS + 2 * i]);
            y2 = fma2(S2[i], make_float2(c4.x, c4.y), y2);
            y2 = fma2(S2[i + 1], make_float2(c4.z, c4.w), y2);
          }
        }
        y[k] = y2.x + y2.y;
      }
      if constexpr (!PART) {
        // sums over the lanes of a channel: the first two steps leave a lane one of the four tokens
        if constexpr (LN >= 4) {
          const bool o1 = sub & 1, o2 = sub & 2;
          const float v0 = (o1 ? y[1] : y[0]) + __shfl_xor_sync(0xffffffffu, o1 ? y[0] : y[1], 1);
          const float v1 = (o1 ? y[3] : y[2]) + __shfl_xor_sync(0xffffffffu, o1 ? y[2] : y[3], 1);
          float v = (o2 ? v1 : v0) + __shfl_xor_sync(0xffffffffu, o2 ? v0 : v1, 2);
#pragma unroll
          for (int o = 4; o < LN; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
          if (sub < 4) s_y[t + sub][ch] = v;          // lane's token: bit 0 from the first step, bit 1 from the second
        } else if constexpr (LN == 2) {
          const float v0 = (sub ? y[1] : y[0]) + __shfl_xor_sync(0xffffffffu, sub ? y[0] : y[1], 1);
          const float v1 = (sub ? y[3] : y[2]) + __shfl_xor_sync(0xffffffffu, sub ? y[2] : y[3], 1);
          s_y[t + sub][ch] = v0;
          s_y[t + 2 + sub][ch] = v1;
        } else {
#pragma unroll
          for (int k = 0; k < 4; ++k) s_y[t + k][ch] = y[k];
        }
      }
    }
    if constexpr (!PART) {
      __syncthreads();
#pragma unroll
      for (int i = 0; i < PER; ++i) {
        const int r = sr + i * ROWS;
        if (column && r < TOK && t0 + r < b) {
          F o;
#pragma unroll
          for (int v = 0; v < V; ++v) o.v[v] = from_f<T>(fmaf(skip[v], to_f(u_now[i].v[v]), s_y[r][sc + v]) * silu_of(to_f(z_now[i].v[v])));
          *reinterpret_cast<F*>(py + i * su) = o;
        }
      }
      py += static_cast<long>(TOK) * p.C;
    }
  }
  float* out = nullptr;
  if constexpr (PART) {
    const size_t at = (static_cast<size_t>(seq) * (p.segments - 1) + seg) * p.C + c;
    out = p.part + at * p.N;
    if (mine && sub == 0) p.steps[at] = total;
  } else if (p.pool != nullptr && b == len) {
    const int sl = p.slot[s0];
    if (sl > 0) out = p.pool + (static_cast<size_t>(sl) * p.C + c) * p.N;
  }
  if (out != nullptr && mine) {
#pragma unroll
    for (int i = 0; i < NS; ++i) {
      const int n = sub * NS + i;
      if (n < p.N) out[n] = S[i];
    }
  }
}

// One token of RB sequences.  NS states per lane, LN lanes per channel; VEC: states in 16-byte accesses.  All states of a thread are on their way
// before the first is worked on; the decays' exponents are formed once for all sequences.
template <typename T, int NS, int LN, int RB, bool VEC>
__global__ void __launch_bounds__(128, RB == 4 && NS == 4 ? 7 : 4) selective_step_kernel(const Selective<T> p, int rows) {
  constexpr int CH = 128 / LN, NV = VEC ? 4 : 1;
  const int row0 = blockIdx.y * RB, sub = threadIdx.x % LN, c = blockIdx.x * CH + threadIdx.x / LN;
  const bool mine = c < p.C;
  // neighbouring lanes take neighbouring vectors
  auto place = [&](int i) { return (i / NV * LN + sub) * NV + i % NV; };
  using Raw = Few<T, NV>;                                // kept as they lie in memory until they are used
  float s[RB][NS], A[NS];
  Raw bn[RB][NS / NV], cn[RB][NS / NV];
  T u[RB], d[RB], z[RB];
  int slot[RB];
#pragma unroll
  for (int r = 0; r < RB; ++r) {
    const int row = min(row0 + r, rows - 1);
    slot[r] = p.slot[row];
    const float* S = p.pool + (static_cast<size_t>(slot[r]) * p.C + (mine ? c : 0)) * p.N;
    const T *B = p.B + static_cast<size_t>(row) * p.ldb, *Cm = p.Cm + static_cast<size_t>(row) * p.ldb;
#pragma unroll
    for (int i = 0; i < NS; i += NV) {
      const int n = min(place(i), p.N - NV);          // places past the last state repeat it: their A is not used
      if constexpr (VEC) {
        const float4 w = *reinterpret_cast<const float4*>(S + n);
        s[r][i] = w.x; s[r][i + 1] = w.y; s[r][i + 2] = w.z; s[r][i + 3] = w.w;
      } else {
        s[r][i] = S[n];
      }
      bn[r][i / NV] = *reinterpret_cast<const Raw*>(B + n);
      cn[r][i / NV] = *reinterpret_cast<const Raw*>(Cm + n);
    }
    const int own = mine ? c : 0;
    z[r] = p.z[static_cast<size_t>(row) * p.ldz + own];
    u[r] = p.u[static_cast<size_t>(row) * p.C + own];
    d[r] = p.dt[static_cast<size_t>(row) * p.ldd + own];
  }
  const float bias = mine ? to_f(p.dt_bias[c]) : 0.f, skip = mine ? to_f(p.D[c]) : 0.f;
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const int n = place(i);
    A[i] = mine && n < p.N ? -1.4426950408889634f * __expf(to_f(p.A_log[static_cast<size_t>(c) * p.N + n])) : 0.f;
  }
#pragma unroll
  for (int r = 0; r < RB; ++r) {
    const int row = row0 + r;
    if (row >= rows) break;                            // the same for the whole block
    const float step = softplus_of(to_f(d[r]) + bias), du = step * to_f(u[r]);
    float y = 0.f;
#pragma unroll
    for (int i = 0; i < NS; ++i) {
      const int n = place(i);
      if (n < p.N) {
        s[r][i] = fmaf(fast_exp2(step * A[i]), s[r][i], du * to_f(bn[r][i / NV].v[i % NV]));
        y = fmaf(s[r][i], to_f(cn[r][i / NV].v[i % NV]), y);
      }
    }
    if (mine && slot[r] > 0) {
      float* S = p.pool + (static_cast<size_t>(slot[r]) * p.C + c) * p.N;
#pragma unroll
      for (int i = 0; i < NS; i += NV) {
        const int n = place(i);
        if (n < p.N) {
          if constexpr (VEC) *reinterpret_cast<float4*>(S + n) = make_float4(s[r][i], s[r][i + 1], s[r][i + 2], s[r][i + 3]);
          else S[n] = s[r][i];
        }
      }
    }
#pragma unroll
    for (int o = 1; o < LN; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (mine && sub == 0)
      p.y[static_cast<size_t>(row) * p.C + c] = from_f<T>(fmaf(skip, to_f(u[r]), y) * silu_of(to_f(z[r])));
  }
}

template <typename T>
static Selective<T> selective_params(const torch::Tensor& u, const torch::Tensor& dt, const torch::Tensor& dt_bias, const torch::Tensor& A_log, const torch::Tensor& proj,
                                     int64_t b0, int64_t c0, const torch::Tensor& D, const torch::Tensor& gate, int64_t z0, torch::Tensor& y) {
  Selective<T> p{};
  p.u = reinterpret_cast<const T*>(u.data_ptr());
  p.dt = reinterpret_cast<const T*>(dt.data_ptr()); p.ldd = dt.stride(0);
  p.z = reinterpret_cast<const T*>(gate.data_ptr()) + z0; p.ldz = gate.stride(0);
  p.B = reinterpret_cast<const T*>(proj.data_ptr()) + b0; p.Cm = reinterpret_cast<const T*>(proj.data_ptr()) + c0; p.ldb = proj.stride(0);
  p.dt_bias = reinterpret_cast<const T*>(dt_bias.data_ptr()); p.A_log = reinterpret_cast<const T*>(A_log.data_ptr()); p.D = reinterpret_cast<const T*>(D.data_ptr());
  p.y = reinterpret_cast<T*>(y.data_ptr());
  p.C = A_log.size(0); p.N = A_log.size(1);
  return p;
}

static void selective_check(const torch::Tensor& u, const torch::Tensor& dt, const torch::Tensor& dt_bias, const torch::Tensor& A_log, const torch::Tensor& proj, int64_t b0,
                            int64_t c0, const torch::Tensor& D, const torch::Tensor& gate, int64_t z0) {
  const auto st = u.scalar_type();
  TORCH_CHECK(u.is_cuda() && u.dim() == 2 && u.is_contiguous() && (st == torch::kBFloat16 || st == torch::kFloat32), "inputs [rows, channels] bf16 or fp32");
  const int64_t rows = u.size(0), C = u.size(1);
  TORCH_CHECK(A_log.scalar_type() == st && A_log.is_contiguous() && A_log.dim() == 2 && A_log.size(0) == C && A_log.size(1) >= 1 && A_log.size(1) <= 256, "A_log [channels, up to 256 states]");
  const int64_t N = A_log.size(1);
  for (const auto* t : {&dt_bias, &D}) TORCH_CHECK(t->scalar_type() == st && t->is_contiguous() && t->numel() == C, "step bias and skip [channels]");
  for (const auto* t : {&dt, &proj, &gate}) TORCH_CHECK(t->scalar_type() == st && t->dim() == 2 && t->stride(1) == 1 && t->size(0) == rows, "projections [rows, .]");
  TORCH_CHECK(dt.size(1) == C && b0 >= 0 && c0 >= 0 && z0 >= 0 && b0 + N <= proj.size(1) && c0 + N <= proj.size(1) && z0 + C <= gate.size(1), "columns outside the projections");
}

// Calls f(NS, LN) as integral constants for a number of states.
template <typename F>
static void selective_lanes(int64_t N, F f) {
  auto go = [&](auto ns, auto ln) { f(ns, ln); };
  using std::integral_constant;
  if (N <= 4) go(integral_constant<int, 4>{}, integral_constant<int, 1>{});
  else if (N <= 8) go(integral_constant<int, 4>{}, integral_constant<int, 2>{});
  else if (N <= 16) go(integral_constant<int, 4>{}, integral_constant<int, 4>{});
  else if (N <= 32) go(integral_constant<int, 8>{}, integral_constant<int, 4>{});
  else if (N <= 64) go(integral_constant<int, 8>{}, integral_constant<int, 8>{});
  else if (N <= 128) go(integral_constant<int, 8>{}, integral_constant<int, 16>{});
  else go(integral_constant<int, 8>{}, integral_constant<int, 32>{});
}

torch::Tensor selective_prefill(const torch::Tensor& u, const torch::Tensor& dt, const torch::Tensor& dt_bias, const torch::Tensor& A_log, const torch::Tensor& proj, int64_t b0,
                                int64_t c0, const torch::Tensor& D, const torch::Tensor& gate, int64_t z0, const torch::Tensor& cu, int64_t max_seqlen, const OptT& pool,
                                const OptT& slot) {
  selective_check(u, dt, dt_bias, A_log, proj, b0, c0, D, gate, z0);
  TORCH_CHECK(cu.is_cuda() && cu.scalar_type() == torch::kInt32 && cu.is_contiguous() && cu.numel() >= 1, "cu_seqlens int32 on device");
  const int64_t rows = u.size(0), C = u.size(1), N = A_log.size(1), n = cu.numel() - 1;
  if (has(pool)) {
    TORCH_CHECK(pool->is_cuda() && pool->scalar_type() == torch::kFloat32 && pool->is_contiguous() && pool->dim() == 3 && pool->size(1) == C && pool->size(2) == N, "states [slots, channels, N] fp32");
    TORCH_CHECK(has(slot) && slot->scalar_type() == torch::kInt32 && slot->is_contiguous() && slot->numel() == rows, "slots int32 [rows]");
  }
  c10::cuda::CUDAGuard guard(u.device());
  auto y = torch::empty_like(u);
  if (rows == 0 || n == 0 || max_seqlen <= 0) return y;
  auto stream = at::cuda::getCurrentCUDAStream();
  auto run = [&](auto tag) {
    using T = decltype(tag);
    auto p = selective_params<T>(u, dt, dt_bias, A_log, proj, b0, c0, D, gate, z0, y);
    p.cu = cu.data_ptr<int>();
    if (has(pool)) { p.pool = pool->data_ptr<float>(); p.slot = slot->data_ptr<int>(); }
    auto pair = [](const T* q, int64_t ld) { return reinterpret_cast<uintptr_t>(q) % (2 * sizeof(T)) == 0 && ld % 2 == 0; };
    auto go = [&](auto ns, auto ln, auto v) {
      constexpr int NS = decltype(ns)::value, LN = decltype(ln)::value, V = decltype(v)::value, CH = sel::THREADS / LN, TOK = sel::tokens(NS * LN);
      const int64_t across = (C + CH - 1) / CH, blocks = across * n, fill = num_sms() * 6L;
      // segments of at least 64 tokens, as many as fill the device (the work of all but the last is done twice)
      int64_t segments = blocks * 2 > fill ? 1 : std::min<int64_t>({fill / blocks, (max_seqlen + 63) / 64, 32});
      const int64_t seg_len = ((max_seqlen + segments - 1) / segments + TOK - 1) / TOK * TOK;
      segments = (max_seqlen + seg_len - 1) / seg_len;
      p.segments = static_cast<int>(segments);
      p.seg_len = static_cast<int>(seg_len);
      torch::Tensor part, steps;
      if (segments > 1) {
        part = torch::empty({n * (segments - 1) * C * N}, u.options().dtype(torch::kFloat32));
        steps = torch::empty({n * (segments - 1) * C}, part.options());
        p.part = part.data_ptr<float>();
        p.steps = steps.data_ptr<float>();
        selective_prefill_kernel<T, NS, LN, V, true><<<dim3(across, segments - 1, n), sel::THREADS, 0, stream>>>(p);
        count_launch();
      }
      selective_prefill_kernel<T, NS, LN, V, false><<<dim3(across, segments, n), sel::THREADS, 0, stream>>>(p);
      count_launch();
    };
    using std::integral_constant;
    // odd numbers of channels: one instance for any number of states
    if (pair(p.u, C) && pair(p.dt, p.ldd) && pair(p.z, p.ldz)) selective_lanes(N, [&](auto ns, auto ln) { go(ns, ln, integral_constant<int, 2>{}); });
    else go(integral_constant<int, 8>{}, integral_constant<int, 32>{}, integral_constant<int, 1>{});
  };
  if (u.scalar_type() == torch::kBFloat16) run(bf16{}); else run(float{});
  TK_CUDA_CHECK(cudaGetLastError());
  return y;
}

torch::Tensor selective_step(const torch::Tensor& u, const torch::Tensor& dt, const torch::Tensor& dt_bias, const torch::Tensor& A_log, const torch::Tensor& proj, int64_t b0,
                             int64_t c0, const torch::Tensor& D, const torch::Tensor& gate, int64_t z0, const torch::Tensor& pool, const torch::Tensor& slot) {
  selective_check(u, dt, dt_bias, A_log, proj, b0, c0, D, gate, z0);
  const int64_t rows = u.size(0), C = u.size(1), N = A_log.size(1);
  TORCH_CHECK(pool.is_cuda() && pool.scalar_type() == torch::kFloat32 && pool.is_contiguous() && pool.dim() == 3 && pool.size(1) == C && pool.size(2) == N, "states [slots, channels, N] fp32");
  TORCH_CHECK(slot.scalar_type() == torch::kInt32 && slot.is_contiguous() && slot.numel() == rows && rows <= 65535, "slots int32 [rows]");
  c10::cuda::CUDAGuard guard(u.device());
  auto y = torch::empty_like(u);
  if (rows == 0) return y;
  auto stream = at::cuda::getCurrentCUDAStream();
  auto run = [&](auto tag) {
    using T = decltype(tag);
    auto p = selective_params<T>(u, dt, dt_bias, A_log, proj, b0, c0, D, gate, z0, y);
    p.pool = pool.data_ptr<float>(); p.slot = slot.data_ptr<int>();
    selective_lanes(N, [&](auto ns, auto ln) {
      constexpr int NS = decltype(ns)::value, LN = decltype(ln)::value, CH = 128 / LN;
      const int64_t across = (C + CH - 1) / CH;
      auto go = [&](auto kern, int rb) { kern<<<dim3(static_cast<unsigned>(across), static_cast<unsigned>((rows + rb - 1) / rb)), 128, 0, stream>>>(p, static_cast<int>(rows)); };
      // four sequences per block once that leaves blocks enough
      const bool vec = N % 4 == 0 && p.ldb % 4 == 0 && reinterpret_cast<uintptr_t>(p.B) % (4 * sizeof(T)) == 0 && reinterpret_cast<uintptr_t>(p.Cm) % (4 * sizeof(T)) == 0;
      const bool four = across * rows >= 4L * 8 * num_sms();
      if (!vec) go(selective_step_kernel<T, NS, LN, 1, false>, 1);
      else if (four) go(selective_step_kernel<T, NS, LN, 4, true>, 4);
      else go(selective_step_kernel<T, NS, LN, 1, true>, 1);
    });
  };
  if (u.scalar_type() == torch::kBFloat16) run(bf16{}); else run(float{});
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return y;
}

}  // namespace tk
