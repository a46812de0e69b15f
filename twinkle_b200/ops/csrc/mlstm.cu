// Matrix memory (mLSTM) between its projections.  Per head, with S ∈ R^{dim × vdim}, n ∈ R^dim and m in fp32, all zero at the start:
//
//   i = cap tanh((i_raw + b) / cap),  f = log σ(cap tanh((f_raw + b) / cap)),  m' = max(f + m, i)
//   S ← e^{f + m − m'} S + e^{i − m'} k vᵀ,   n ← likewise with k,   o = Sᵀ q / (max(|n·q|, e^{−m'}) + 10⁻⁶),   q = q_raw / √dim
//   output = o / rms(o) · weight · σ(gate)                              (rms over the head's vdim)
//
//   mlstm_prefill  packed prompts; a block owns one head of one sequence (or columns of it), the state is in registers, tokens pass
//                  through shared memory sixteen at a time.  The normaliser rides along as one more column whose values are one.
//   mlstm_step     one token of every sequence: the state passes once through the block, 16 bytes per access.
// A state is a row of the pool: the matrix by rows, n and m, each from a 16-byte boundary on.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/types.h>

#include "common.cuh"
#include "host.h"
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
  int H, dim, vdim, n0, m0, cols, slices, rows;
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
#pragma unroll 8
      for (int r = group; r < p.dim; r += groups) {
        float* at = S + static_cast<size_t>(r) * p.vdim + x * V;
        const float q = s_q[r], k = s_k[r];
        if constexpr (V == 4) {
          float4 s = *reinterpret_cast<const float4*>(at);
          s.x = fmaf(k, av[0], keep * s.x); s.y = fmaf(k, av[1], keep * s.y); s.z = fmaf(k, av[2], keep * s.z); s.w = fmaf(k, av[3], keep * s.w);
          if (slot > 0) *reinterpret_cast<float4*>(at) = s;
          o[0] = fmaf(q, s.x, o[0]); o[1] = fmaf(q, s.y, o[1]); o[2] = fmaf(q, s.z, o[2]); o[3] = fmaf(q, s.w, o[3]);
        } else {
          const float s = fmaf(k, av[0], keep * *at);
          if (slot > 0) *at = s;
          o[0] = fmaf(q, s, o[0]);
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
    auto raw = torch::empty({rows, H * vdim}, proj.options().dtype(torch::kFloat32));
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
