// Latent attention (keys and values expanded from one cached vector per token, which serves as both in latent space):
//   latent_norms   RMS norms of the query bottleneck and of the new latents, and the write into the paged cache — one pass
//   latent_decode  one token per sequence, all heads against the same cached rows, optionally the last `window` of them, a sink logit in
//                  the denominator and a sigmoid gate on the result.  A cached row may be wider than its value (rotated key
//                  dimensions).  This file holds the fp32-arithmetic form for any rank up to 1024 (32-bit models, odd sizes, small
//                  pages); latent_decode.cu the tensor-core form for bf16.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/types.h>

#include "common.cuh"
#include "host.h"

namespace tk {

using bf16 = __nv_bfloat16;
using OptT = c10::optional<torch::Tensor>;

namespace lt {
__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(bf16* p, float v) { *p = __float2bfloat16(v); }
// two consecutive elements
__device__ __forceinline__ float2 ld2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 ld2(const bf16* p) { return unpack_bf16(*reinterpret_cast<const uint32_t*>(p)); }
__device__ __forceinline__ void st2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void st2(bf16* p, float a, float b) { *reinterpret_cast<uint32_t*>(p) = pack_bf16(a, b); }
bool has(const OptT& t) { return t.has_value() && t->defined(); }
}  // namespace lt

// One warp per (row, range): range 0 the query bottleneck, range 1 the latent.
template <typename T, bool PAIRS>
__global__ void __launch_bounds__(256) latent_norms_kernel(const T* __restrict__ proj, long ld, int q0, int nq, const T* __restrict__ wq, T* __restrict__ q, int c0, int nc,
                                                           int ncp, const T* __restrict__ wc, T* __restrict__ c, T* __restrict__ pool, const int64_t* __restrict__ pool_row,
                                                           int rows, float eps) {
  const int per = nc > 0 ? 2 : 1;
  const long i = blockIdx.x * 8L + (threadIdx.x >> 5);
  if (i >= static_cast<long>(rows) * per) return;
  const int lane = threadIdx.x & 31, t = static_cast<int>(i / per);
  const bool is_c = per == 2 && (i & 1);
  const T* x = proj + t * ld + (is_c ? c0 : q0);
  const T* w = is_c ? wc : wq;
  const int n = is_c ? nc : nq;
  float ss = 0.f;
  if constexpr (PAIRS) {
    for (int j = lane * 2; j < n; j += 64) { const float2 a = lt::ld2(x + j); ss += a.x * a.x + a.y * a.y; }
  } else {
    for (int j = lane; j < n; j += 32) { const float a = lt::ld(x + j); ss += a * a; }
  }
  const float r = rsqrtf(warp_sum(ss) / n + eps);
  T* out = is_c ? c + static_cast<size_t>(t) * ncp : q + static_cast<size_t>(t) * nq;
  const int64_t row = is_c && pool != nullptr ? pool_row[t] : -1;
  T* kept = row >= 0 ? pool + static_cast<size_t>(row) * ncp : nullptr;
  const int wide = is_c ? ncp : n;
  if constexpr (PAIRS) {
    for (int j = lane * 2; j < wide; j += 64) {
      float2 a = make_float2(0.f, 0.f);
      if (j < n) {
        a = lt::ld2(x + j);
        const float2 g = lt::ld2(w + j);
        a.x *= r * g.x; a.y *= r * g.y;
      }
      lt::st2(out + j, a.x, a.y);
      if (kept != nullptr) lt::st2(kept + j, a.x, a.y);
    }
  } else {
    for (int j = lane; j < wide; j += 32) {
      const float a = j < n ? lt::ld(x + j) * r * lt::ld(w + j) : 0.f;
      lt::st(out + j, a);
      if (kept != nullptr) lt::st(kept + j, a);
    }
  }
}

std::vector<torch::Tensor> latent_norms(const torch::Tensor& proj, int64_t q0, int64_t nq, const torch::Tensor& wq, int64_t c0, int64_t nc, const OptT& wc, double eps,
                                        const OptT& pool, const OptT& pool_row) {
  const auto st = proj.scalar_type();
  TORCH_CHECK(proj.is_cuda() && proj.dim() == 2 && proj.stride(1) == 1 && (st == torch::kBFloat16 || st == torch::kFloat32), "projection [rows, N] bf16 or fp32");
  TORCH_CHECK(nq > 0 && nc >= 0 && q0 >= 0 && c0 >= 0 && q0 + nq <= proj.size(1) && c0 + nc <= proj.size(1), "columns outside the projection");
  TORCH_CHECK(wq.scalar_type() == st && wq.is_contiguous() && wq.numel() == nq, "query norm weight");
  const int64_t rows = proj.size(0), ncp = (nc + 7) / 8 * 8;
  if (nc > 0) TORCH_CHECK(lt::has(wc) && wc->scalar_type() == st && wc->is_contiguous() && wc->numel() == nc, "latent norm weight");
  if (lt::has(pool)) {
    TORCH_CHECK(nc > 0 && pool->scalar_type() == st && pool->is_contiguous() && pool->size(-1) == ncp, "latent pool [..., rank rounded up to 8]");
    TORCH_CHECK(lt::has(pool_row) && pool_row->scalar_type() == torch::kInt64 && pool_row->is_contiguous() && pool_row->numel() == rows, "pool rows int64 [rows]");
  }
  c10::cuda::CUDAGuard guard(proj.device());
  auto q = torch::empty({rows, nq}, proj.options());
  auto c = torch::empty({rows, ncp}, proj.options());
  if (rows == 0) return {q, c};
  const long warps = rows * (nc > 0 ? 2 : 1);
  const bool pairs = ((proj.stride(0) | q0 | c0 | nq | nc) % 2) == 0 && reinterpret_cast<uintptr_t>(proj.data_ptr()) % 8 == 0;
  auto stream = at::cuda::getCurrentCUDAStream();
  auto run = [&](auto tag) {
    using T = decltype(tag);
    auto go = [&](auto kern) {
      kern<<<static_cast<unsigned>((warps + 7) / 8), 256, 0, stream>>>(
          reinterpret_cast<const T*>(proj.data_ptr()), proj.stride(0), q0, nq, reinterpret_cast<const T*>(wq.data_ptr()), reinterpret_cast<T*>(q.data_ptr()), c0, nc, ncp,
          nc > 0 ? reinterpret_cast<const T*>(wc->data_ptr()) : nullptr, reinterpret_cast<T*>(c.data_ptr()),
          lt::has(pool) ? reinterpret_cast<T*>(pool->data_ptr()) : nullptr, lt::has(pool) ? pool_row->data_ptr<int64_t>() : nullptr, rows, static_cast<float>(eps));
    };
    if (pairs) go(latent_norms_kernel<T, true>); else go(latent_norms_kernel<T, false>);
  };
  if (st == torch::kBFloat16) run(bf16{}); else run(float{});
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return {q, c};
}

// ---------------------------------------------------------------- latent decode, fp32 arithmetic
// Block = (GH heads, sequence), 256 threads.  Sixteen cached rows at a time in shared memory; four threads form a score over the K
// columns of a row, a thread owns RI of the R ≤ K value columns of every head.
template <typename T, int RI>
__global__ void __launch_bounds__(256) latent_decode_plain_kernel(const T* __restrict__ q, const T* __restrict__ pool, const int* __restrict__ tables,
                                                                  const int* __restrict__ lens, const T* __restrict__ sinks, const T* __restrict__ gate, long ldg,
                                                                  T* __restrict__ out, int H, int K, int R, int RP, int block_size, int max_blocks, int window, float scale) {
  constexpr int GH = 4, TK = 16;
  extern __shared__ float sm_latent[];
  __shared__ float s_s[GH][TK];
  const int h0 = blockIdx.x * GH, b = blockIdx.y, tid = threadIdx.x, n = lens[b];
  const int pitch = K + 1;
  float *s_q = sm_latent, *s_c = s_q + GH * pitch;
  for (int i = tid; i < GH * K; i += 256) {
    const int g = i / K, c = i - g * K;
    s_q[g * pitch + c] = h0 + g < H ? lt::ld(q + (static_cast<size_t>(b) * H + h0 + g) * K + c) * scale : 0.f;
  }
  float acc[GH][RI], m[GH], l[GH];
#pragma unroll
  for (int g = 0; g < GH; ++g) {
    // the sink is a key without a value that every step already sees
    m[g] = sinks == nullptr ? -1e30f : (h0 + g < H ? lt::ld(sinks + h0 + g) : 0.f);
    l[g] = sinks == nullptr ? 0.f : 1.f;
#pragma unroll
    for (int i = 0; i < RI; ++i) acc[g][i] = 0.f;
  }
  const int* table = tables + static_cast<size_t>(b) * max_blocks;
  for (int t0 = window > 0 ? max(0, n - window) : 0; t0 < n; t0 += TK) {
    __syncthreads();
    for (int i = tid; i < TK * K; i += 256) {
      const int t = i / K, c = i - t * K, p = t0 + t;
      s_c[t * pitch + c] = p < n ? lt::ld(pool + (static_cast<size_t>(table[p / block_size]) * block_size + p % block_size) * RP + c) : 0.f;
    }
    __syncthreads();
    {
      const int pair = tid >> 2, sub = tid & 3, g = pair / TK, t = pair % TK;
      float s = 0.f;
      for (int c = sub; c < K; c += 4) s += s_q[g * pitch + c] * s_c[t * pitch + c];
      s += __shfl_xor_sync(0xffffffffu, s, 1);
      s += __shfl_xor_sync(0xffffffffu, s, 2);
      if (sub == 0) s_s[g][t] = t0 + t < n ? s : -INFINITY;
    }
    __syncthreads();
#pragma unroll
    for (int g = 0; g < GH; ++g) {
      float mx = m[g];
#pragma unroll
      for (int t = 0; t < TK; ++t) mx = fmaxf(mx, s_s[g][t]);
      const float corr = __expf(m[g] - mx);
      m[g] = mx;
      l[g] *= corr;
#pragma unroll
      for (int i = 0; i < RI; ++i) acc[g][i] *= corr;
#pragma unroll
      for (int t = 0; t < TK; ++t) {
        const float w = __expf(s_s[g][t] - mx);
        l[g] += w;
#pragma unroll
        for (int i = 0; i < RI; ++i)
          if (tid + i * 256 < R) acc[g][i] += w * s_c[t * pitch + tid + i * 256];
      }
    }
  }
#pragma unroll
  for (int g = 0; g < GH; ++g) {
    if (h0 + g >= H) break;
    float f = l[g] > 0.f ? 1.f / l[g] : 0.f;
    if (gate != nullptr) f /= 1.f + __expf(-lt::ld(gate + b * ldg + h0 + g));
#pragma unroll
    for (int i = 0; i < RI; ++i)
      if (tid + i * 256 < R) lt::st(out + (static_cast<size_t>(b) * H + h0 + g) * R + tid + i * 256, acc[g][i] * f);
  }
}

bool latent_decode_tc(const torch::Tensor& q, const torch::Tensor& pool, const torch::Tensor& tables, const torch::Tensor& lens, double scale, const OptT& sinks,
                      const OptT& gate, int window, torch::Tensor& out);

// q [B, H, K], pool [blocks, bs, 1, K rounded up to 8], tables int32 [B, ·], lens int32 [B] → [B, H, R] (values: the first R ≤ K columns)
torch::Tensor latent_decode(const torch::Tensor& q, const torch::Tensor& pool, const torch::Tensor& tables, const torch::Tensor& lens, double scale,
                            const OptT& sinks, const OptT& gate, int64_t rank, int64_t window) {
  const auto st = q.scalar_type();
  TORCH_CHECK(q.is_cuda() && q.dim() == 3 && q.is_contiguous() && (st == torch::kBFloat16 || st == torch::kFloat32), "q [B, H, K] bf16 or fp32");
  const int B = q.size(0), H = q.size(1), K = q.size(2), R = rank;
  TORCH_CHECK(R >= 1 && R <= K && window >= 0 && window < (int64_t(1) << 30), "value columns within the key's, window 0 (none) or positive");
  TORCH_CHECK(pool.scalar_type() == st && pool.is_contiguous() && pool.dim() == 4 && pool.size(2) == 1 && pool.size(3) >= K, "latent pool [blocks, bs, 1, >= K]");
  TORCH_CHECK(tables.scalar_type() == torch::kInt32 && tables.is_contiguous() && tables.dim() == 2 && tables.size(0) == B && lens.scalar_type() == torch::kInt32 &&
                  lens.is_contiguous() && lens.numel() == B, "int32 tables / lens");
  if (lt::has(sinks)) TORCH_CHECK(sinks->scalar_type() == st && sinks->is_contiguous() && sinks->numel() == H, "sinks [H]");
  if (lt::has(gate)) TORCH_CHECK(gate->scalar_type() == st && gate->dim() == 2 && gate->size(0) == B && gate->size(1) == H && gate->stride(1) == 1, "gate [B, H]");
  TORCH_CHECK(R <= 1024 && K <= 2048, "latent rank up to 1024, rows up to 2048 wide");
  c10::cuda::CUDAGuard guard(q.device());
  auto out = torch::empty({B, H, R}, q.options());
  if (B == 0) return out;
  if (latent_decode_tc(q, pool, tables, lens, scale, sinks, gate, static_cast<int>(window), out)) return out;
  auto stream = at::cuda::getCurrentCUDAStream();
  const size_t smem = sizeof(float) * 20 * (K + 1);
  auto run = [&](auto tag) {
    using T = decltype(tag);
    auto go = [&](auto kern) {
      TK_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
      kern<<<dim3((H + 3) / 4, B), 256, smem, stream>>>(
          reinterpret_cast<const T*>(q.data_ptr()), reinterpret_cast<const T*>(pool.data_ptr()), tables.data_ptr<int>(), lens.data_ptr<int>(),
          lt::has(sinks) ? reinterpret_cast<const T*>(sinks->data_ptr()) : nullptr, lt::has(gate) ? reinterpret_cast<const T*>(gate->data_ptr()) : nullptr, lt::has(gate) ? gate->stride(0) : 0L,
          reinterpret_cast<T*>(out.data_ptr()), H, K, R, static_cast<int>(pool.size(3)), static_cast<int>(pool.size(1)), static_cast<int>(tables.size(1)),
          static_cast<int>(window), static_cast<float>(scale));
    };
    if (R <= 256) go(latent_decode_plain_kernel<T, 1>);
    else if (R <= 512) go(latent_decode_plain_kernel<T, 2>);
    else go(latent_decode_plain_kernel<T, 4>);
  };
  if (st == torch::kBFloat16) run(bf16{}); else run(float{});
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return out;
}

}  // namespace tk
