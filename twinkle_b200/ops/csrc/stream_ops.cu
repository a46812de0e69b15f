// Element-wise steps of decoder layers whose residual stream is 32-bit:
//   stream_rmsnorm  x += mult · (y1 ⊙ s1 + y2 ⊙ s2) in fp32 and the RMS norm of the sum in the compute dtype — one pass
//   stream_joined_rmsnorm  x += y + open · beside in fp32 and the RMS norm of the sum — one pass; y is a row of its own or the
//                   weighted sum of a token's expert rows, beside a shared expert's row with a weight per token
//   stream_gated_rmsnorm  x += norm(σ(gate + bias) ⊙ y) in fp32 and the RMS norm of the sum — one pass; y is a row of its own or
//                   the weighted sum of a token's expert rows
//   stream_normed_add  x += norm(y + bias) in fp32, or the norm of half the sum of two normed results, and the sum or its RMS norm in the
//                   compute dtype — one pass
//   embed_positions an embedding's row plus sines and cosines of the position, fp32
//   glu_columns     silu(gate) · up, gelu(gate) · up (tanh form) or the clamped form, on two column ranges of a projection
// All are templated on the compute dtype (bf16 or fp32) and work for any width: vector kernels where rows are made of
// whole vectors, plain ones otherwise.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/types.h>

#include "common.cuh"
#include "host.h"
#include "vec.cuh"

namespace tk {

// -------------------------------------------------------------- stream_rmsnorm
// One block per row.  VPT > 0: a thread keeps its VPT groups of four sums in registers between the two passes; VPT = 0:
// rows of any width, element-wise, the second pass re-reads what the thread wrote.
template <typename T, int VPT>
__global__ void stream_rmsnorm_kernel(float* __restrict__ x, const T* __restrict__ y1, const T* __restrict__ s1, const T* __restrict__ y2,
                                      const T* __restrict__ s2, float mult, const T* __restrict__ w, T* __restrict__ h, int W, float eps, float offset) {
  __shared__ float sh[32];
  const size_t base = static_cast<size_t>(blockIdx.x) * W;
  float ss = 0.f;
  if constexpr (VPT > 0) {
    float4 v[VPT];
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * 4;
      v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < W) {
        v[i] = load4(x + base + c);
        if (y1 != nullptr) {
          const float4 a = load4(y1 + base + c), b = load4(s1 + c);
          float4 s = make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w);
          if (y2 != nullptr) {
            const float4 e = load4(y2 + base + c), f = load4(s2 + c);
            s.x += e.x * f.x; s.y += e.y * f.y; s.z += e.z * f.z; s.w += e.w * f.w;
          }
          v[i].x += mult * s.x; v[i].y += mult * s.y; v[i].z += mult * s.z; v[i].w += mult * s.w;
          store4(x + base + c, v[i]);
        }
      }
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    const float r = rsqrtf(block_sum(ss, sh) / W + eps);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * 4;
      if (c < W) {
        const float4 g = load4(w + c);
        store4(h + base + c, make_float4(v[i].x * r * (offset + g.x), v[i].y * r * (offset + g.y), v[i].z * r * (offset + g.z), v[i].w * r * (offset + g.w)));
      }
    }
  } else {
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
      float v = x[base + c];
      if (y1 != nullptr) {
        float s = to_f(y1[base + c]) * to_f(s1[c]);
        if (y2 != nullptr) s += to_f(y2[base + c]) * to_f(s2[c]);
        v += mult * s;
        x[base + c] = v;
      }
      ss += v * v;
    }
    const float r = rsqrtf(block_sum(ss, sh) / W + eps);
    for (int c = threadIdx.x; c < W; c += blockDim.x) h[base + c] = from_f<T>(x[base + c] * r * (offset + to_f(w[c])));
  }
}

// x [rows, W] fp32 is updated in place when y1 is given; returns the norm (weights offset + w) in w's dtype.
torch::Tensor stream_rmsnorm(torch::Tensor x, const torch::Tensor& w, double eps, const OptT& y1, const OptT& s1, const OptT& y2, const OptT& s2, double mult,
                             double offset) {
  const auto st = w.scalar_type();
  TORCH_CHECK(x.is_cuda() && x.scalar_type() == torch::kFloat32 && x.is_contiguous() && x.dim() == 2, "stream [rows, W] fp32 contiguous");
  TORCH_CHECK((st == torch::kBFloat16 || st == torch::kFloat32) && w.is_contiguous() && w.numel() == x.size(1), "norm weight [W] bf16 or fp32");
  const int rows = x.size(0), W = x.size(1);
  bool vec = W % 4 == 0 && W <= 8192 && aligned16(w.data_ptr());
  auto check = [&](const OptT& y, const OptT& s) {
    if (!has(y)) return;
    TORCH_CHECK(y->scalar_type() == st && y->is_contiguous() && y->numel() == x.numel(), "sub-layer result [rows, W] in the norm weight's dtype");
    TORCH_CHECK(has(s) && s->scalar_type() == st && s->is_contiguous() && s->numel() == W, "channel scale [W]");
    vec = vec && aligned16(y->data_ptr()) && aligned16(s->data_ptr());
  };
  TORCH_CHECK(has(y1) || !has(y2), "the second result comes with a first");
  check(y1, s1);
  check(y2, s2);
  c10::cuda::CUDAGuard guard(x.device());
  auto h = torch::empty(x.sizes(), w.options());
  if (rows == 0) return h;
  auto stream = at::cuda::getCurrentCUDAStream();
  auto run = [&](auto tag) {
    using T = decltype(tag);
    auto ptr = [](const OptT& t) { return has(t) ? reinterpret_cast<const T*>(t->data_ptr()) : static_cast<const T*>(nullptr); };
    auto go = [&](auto kern, int threads) {
      kern<<<rows, threads, 0, stream>>>(x.data_ptr<float>(), ptr(y1), ptr(s1), ptr(y2), ptr(s2), static_cast<float>(mult),
                                         reinterpret_cast<const T*>(w.data_ptr()), reinterpret_cast<T*>(h.data_ptr()), W, static_cast<float>(eps),
                                         static_cast<float>(offset));
    };
    const int nvec = (W + 3) / 4;
    const int vpt = nvec <= 512 ? 1 : (nvec <= 1024 ? 2 : 4);
    const int threads = std::min(512, ((nvec + vpt - 1) / vpt + 31) / 32 * 32);
    if (!vec) go(stream_rmsnorm_kernel<T, 0>, std::min(512, (W + 31) / 32 * 32));
    else if (vpt == 1) go(stream_rmsnorm_kernel<T, 1>, threads);
    else if (vpt == 2) go(stream_rmsnorm_kernel<T, 2>, threads);
    else go(stream_rmsnorm_kernel<T, 4>, threads);
  };
  if (st == torch::kBFloat16) run(bf16{}); else run(float{});
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return h;
}

// -------------------------------------------------------- stream_gated_rmsnorm
// One block per row, as above: gated result in registers, its mean square, the sum, the sum's mean square.  With k > 0 the result is
// the weighted sum of the token's k ≤ 32 expert rows; their places and weights are read once per block.
struct GatedNorm {
  float* x;
  const void *y, *gate, *bias, *post, *next;
  void* h;
  const int* row_of; const float* share;     // [rows, k] (k = 0: y has one row per token)
  long ldg;                                  // row stride of the gate
  int k, W;
  float eps, offset;
};

template <typename T, int VPT>
__global__ void stream_gated_rmsnorm_kernel(const GatedNorm p) {
  __shared__ float sh[32];
  __shared__ int s_row[32];
  __shared__ float s_share[32];
  const int W = p.W, t = blockIdx.x;
  const T *y = reinterpret_cast<const T*>(p.y), *gate = reinterpret_cast<const T*>(p.gate) + t * p.ldg, *bias = reinterpret_cast<const T*>(p.bias);
  const T *post = reinterpret_cast<const T*>(p.post), *next = reinterpret_cast<const T*>(p.next);
  float* x = p.x + static_cast<size_t>(t) * W;
  T* h = reinterpret_cast<T*>(p.h) + static_cast<size_t>(t) * W;
  const int k = p.k;
  if (k > 0) {
    if (threadIdx.x < k) {
      s_row[threadIdx.x] = p.row_of[static_cast<size_t>(t) * k + threadIdx.x];
      s_share[threadIdx.x] = p.share[static_cast<size_t>(t) * k + threadIdx.x];
    }
    __syncthreads();
  }
  if constexpr (VPT > 0) {
    float4 z[VPT], v[VPT];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * 4;
      z[i] = v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < W) {
        v[i] = load4(x + c);
        const float4 g = load4(gate + c), b = load4(bias + c);
        float4 a;
        if (k == 0) {
          a = load4(y + static_cast<size_t>(t) * W + c);
        } else {
          a = make_float4(0.f, 0.f, 0.f, 0.f);
          for (int j = 0; j < k; ++j) {
            const float4 e = load4(y + static_cast<size_t>(s_row[j]) * W + c);
            const float w = s_share[j];
            a.x += w * e.x; a.y += w * e.y; a.z += w * e.z; a.w += w * e.w;
          }
        }
        z[i].x = a.x / (1.f + __expf(-(g.x + b.x))); z[i].y = a.y / (1.f + __expf(-(g.y + b.y)));
        z[i].z = a.z / (1.f + __expf(-(g.z + b.z))); z[i].w = a.w / (1.f + __expf(-(g.w + b.w)));
      }
      ss += z[i].x * z[i].x + z[i].y * z[i].y + z[i].z * z[i].z + z[i].w * z[i].w;
    }
    const float r1 = rsqrtf(block_sum(ss, sh) / W + p.eps);
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * 4;
      if (c < W) {
        const float4 w = load4(post + c);
        v[i].x += z[i].x * r1 * (p.offset + w.x); v[i].y += z[i].y * r1 * (p.offset + w.y);
        v[i].z += z[i].z * r1 * (p.offset + w.z); v[i].w += z[i].w * r1 * (p.offset + w.w);
        store4(x + c, v[i]);
      }
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    const float r2 = rsqrtf(block_sum(ss, sh) / W + p.eps);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * 4;
      if (c < W) {
        const float4 w = load4(next + c);
        store4(h + c, make_float4(v[i].x * r2 * (p.offset + w.x), v[i].y * r2 * (p.offset + w.y), v[i].z * r2 * (p.offset + w.z), v[i].w * r2 * (p.offset + w.w)));
      }
    }
  } else {                                   // any width: the gated result is formed twice
    auto gated = [&](int c) {
      float a = 0.f;
      if (k == 0) a = to_f(y[static_cast<size_t>(t) * W + c]);
      for (int j = 0; j < k; ++j) a += s_share[j] * to_f(y[static_cast<size_t>(s_row[j]) * W + c]);
      return a / (1.f + __expf(-(to_f(gate[c]) + to_f(bias[c]))));
    };
    float ss = 0.f;
    for (int c = threadIdx.x; c < W; c += blockDim.x) { const float z = gated(c); ss += z * z; }
    const float r1 = rsqrtf(block_sum(ss, sh) / W + p.eps);
    ss = 0.f;
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
      const float v = x[c] + gated(c) * r1 * (p.offset + to_f(post[c]));
      x[c] = v;
      ss += v * v;
    }
    const float r2 = rsqrtf(block_sum(ss, sh) / W + p.eps);
    for (int c = threadIdx.x; c < W; c += blockDim.x) h[c] = from_f<T>(x[c] * r2 * (p.offset + to_f(next[c])));
  }
}

// x [rows, W] fp32 is updated in place; returns the norm in w's dtype.  gate: [rows, ≥ W] with any row stride.
torch::Tensor stream_gated_rmsnorm(torch::Tensor x, const torch::Tensor& w, double eps, double offset, const torch::Tensor& y, const torch::Tensor& gate,
                                   const torch::Tensor& bias, const torch::Tensor& post, const OptT& row_of, const OptT& share) {
  const auto st = w.scalar_type();
  TORCH_CHECK(x.is_cuda() && x.scalar_type() == torch::kFloat32 && x.is_contiguous() && x.dim() == 2, "stream [rows, W] fp32 contiguous");
  const int rows = x.size(0), W = x.size(1);
  TORCH_CHECK(st == torch::kBFloat16 || st == torch::kFloat32, "bf16 or fp32");
  for (const auto* t : {&w, &bias, &post}) TORCH_CHECK(t->scalar_type() == st && t->is_contiguous() && t->numel() == W, "norm weights and gate bias [W] in one dtype");
  TORCH_CHECK(gate.scalar_type() == st && gate.dim() == 2 && gate.stride(1) == 1 && gate.size(0) == rows && gate.size(1) >= W, "gate [rows, >= W]");
  TORCH_CHECK(y.scalar_type() == st && y.dim() == 2 && y.is_contiguous() && y.size(1) == W, "result [., W]");
  GatedNorm p{};
  if (has(row_of)) {
    TORCH_CHECK(has(share) && row_of->scalar_type() == torch::kInt32 && share->scalar_type() == torch::kFloat32 && row_of->is_contiguous() && share->is_contiguous() &&
                    row_of->dim() == 2 && row_of->size(0) == rows && share->sizes() == row_of->sizes() && row_of->size(1) >= 1 && row_of->size(1) <= 32, "row_of / share [rows, k], k <= 32");
    p.k = row_of->size(1); p.row_of = row_of->data_ptr<int>(); p.share = share->data_ptr<float>();
  } else {
    TORCH_CHECK(y.size(0) == rows, "one result row per token");
  }
  c10::cuda::CUDAGuard guard(x.device());
  auto h = torch::empty(x.sizes(), w.options());
  if (rows == 0) return h;
  p.x = x.data_ptr<float>(); p.y = y.data_ptr(); p.gate = gate.data_ptr(); p.bias = bias.data_ptr(); p.post = post.data_ptr(); p.next = w.data_ptr(); p.h = h.data_ptr();
  p.ldg = gate.stride(0); p.W = W; p.eps = eps; p.offset = offset;
  const bool vec = W % 4 == 0 && W <= 8192 && gate.stride(0) % 4 == 0 && aligned16(p.y) && aligned16(p.gate) && aligned16(p.bias) && aligned16(p.post) && aligned16(p.next);
  const int nvec = (W + 3) / 4, vpt = nvec <= 512 ? 1 : (nvec <= 1024 ? 2 : 4);
  auto stream = at::cuda::getCurrentCUDAStream();
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const int threads = std::min(512, ((nvec + vpt - 1) / vpt + 31) / 32 * 32);
    if (!vec) stream_gated_rmsnorm_kernel<T, 0><<<rows, std::min(512, (W + 31) / 32 * 32), 0, stream>>>(p);
    else if (vpt == 1) stream_gated_rmsnorm_kernel<T, 1><<<rows, threads, 0, stream>>>(p);
    else if (vpt == 2) stream_gated_rmsnorm_kernel<T, 2><<<rows, threads, 0, stream>>>(p);
    else stream_gated_rmsnorm_kernel<T, 4><<<rows, threads, 0, stream>>>(p);
  };
  if (st == torch::kBFloat16) run(bf16{}); else run(float{});
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return h;
}

// ------------------------------------------------------- stream_joined_rmsnorm
// One block per row, as above.
struct JoinedNorm {
  float* x;
  const void *y, *beside, *next;
  const float* open;                         // [rows]
  void* h;
  const int* row_of; const float* share;     // [rows, k] (k = 0: y has one row per token)
  int k, W;
  float eps, offset;
};

template <typename T, int VPT>
__global__ void stream_joined_rmsnorm_kernel(const JoinedNorm p) {
  __shared__ float sh[32];
  __shared__ int s_row[32];
  __shared__ float s_share[32];
  const int W = p.W, t = blockIdx.x, k = p.k;
  const T *y = reinterpret_cast<const T*>(p.y), *next = reinterpret_cast<const T*>(p.next);
  const T* beside = p.beside == nullptr ? nullptr : reinterpret_cast<const T*>(p.beside) + static_cast<size_t>(t) * W;
  float* x = p.x + static_cast<size_t>(t) * W;
  T* h = reinterpret_cast<T*>(p.h) + static_cast<size_t>(t) * W;
  const float open = beside != nullptr ? p.open[t] : 0.f;
  if (k > 0) {
    if (threadIdx.x < k) {
      s_row[threadIdx.x] = p.row_of[static_cast<size_t>(t) * k + threadIdx.x];
      s_share[threadIdx.x] = p.share[static_cast<size_t>(t) * k + threadIdx.x];
    }
    __syncthreads();
  }
  float ss = 0.f;
  if constexpr (VPT > 0) {
    float4 v[VPT];
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * 4;
      v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < W) {
        v[i] = load4(x + c);
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
        if (k == 0) {
          a = load4(y + static_cast<size_t>(t) * W + c);
        } else {
          int j = 0;
          for (; j + 4 <= k; j += 4) {       // four rows on their way at a time
            float4 e[4];
#pragma unroll
            for (int u = 0; u < 4; ++u) e[u] = load4(y + static_cast<size_t>(s_row[j + u]) * W + c);
#pragma unroll
            for (int u = 0; u < 4; ++u) {
              const float w = s_share[j + u];
              a.x += w * e[u].x; a.y += w * e[u].y; a.z += w * e[u].z; a.w += w * e[u].w;
            }
          }
          for (; j < k; ++j) {
            const float4 e = load4(y + static_cast<size_t>(s_row[j]) * W + c);
            const float w = s_share[j];
            a.x += w * e.x; a.y += w * e.y; a.z += w * e.z; a.w += w * e.w;
          }
        }
        if (beside != nullptr) {
          const float4 b = load4(beside + c);
          a.x += open * b.x; a.y += open * b.y; a.z += open * b.z; a.w += open * b.w;
        }
        v[i].x += a.x; v[i].y += a.y; v[i].z += a.z; v[i].w += a.w;
        store4(x + c, v[i]);
      }
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    const float r = rsqrtf(block_sum(ss, sh) / W + p.eps);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * 4;
      if (c < W) {
        const float4 w = load4(next + c);
        store4(h + c, make_float4(v[i].x * r * (p.offset + w.x), v[i].y * r * (p.offset + w.y), v[i].z * r * (p.offset + w.z), v[i].w * r * (p.offset + w.w)));
      }
    }
  } else {                                   // any width: the second pass re-reads what the thread wrote
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
      float a = 0.f;
      if (k == 0) a = to_f(y[static_cast<size_t>(t) * W + c]);
      for (int j = 0; j < k; ++j) a += s_share[j] * to_f(y[static_cast<size_t>(s_row[j]) * W + c]);
      if (beside != nullptr) a += open * to_f(beside[c]);
      const float v = x[c] + a;
      x[c] = v;
      ss += v * v;
    }
    const float r = rsqrtf(block_sum(ss, sh) / W + p.eps);
    for (int c = threadIdx.x; c < W; c += blockDim.x) h[c] = from_f<T>(x[c] * r * (p.offset + to_f(next[c])));
  }
}

// x [rows, W] fp32 is updated in place; returns the norm in w's dtype.
torch::Tensor stream_joined_rmsnorm(torch::Tensor x, const torch::Tensor& w, double eps, double offset, const torch::Tensor& y, const OptT& row_of, const OptT& share,
                                    const OptT& beside, const OptT& open) {
  const auto st = w.scalar_type();
  TORCH_CHECK(x.is_cuda() && x.scalar_type() == torch::kFloat32 && x.is_contiguous() && x.dim() == 2, "stream [rows, W] fp32 contiguous");
  const int rows = x.size(0), W = x.size(1);
  TORCH_CHECK((st == torch::kBFloat16 || st == torch::kFloat32) && w.is_contiguous() && w.numel() == W, "norm weight [W] bf16 or fp32");
  TORCH_CHECK(y.scalar_type() == st && y.dim() == 2 && y.is_contiguous() && y.size(1) == W, "result [., W]");
  JoinedNorm p{};
  if (has(row_of)) {
    TORCH_CHECK(has(share) && row_of->scalar_type() == torch::kInt32 && share->scalar_type() == torch::kFloat32 && row_of->is_contiguous() && share->is_contiguous() &&
                    row_of->dim() == 2 && row_of->size(0) == rows && share->sizes() == row_of->sizes() && row_of->size(1) >= 1 && row_of->size(1) <= 32, "row_of / share [rows, k], k <= 32");
    p.k = row_of->size(1); p.row_of = row_of->data_ptr<int>(); p.share = share->data_ptr<float>();
  } else {
    TORCH_CHECK(y.size(0) == rows, "one result row per token");
  }
  if (has(beside)) {
    TORCH_CHECK(beside->scalar_type() == st && beside->is_contiguous() && beside->dim() == 2 && beside->size(0) == rows && beside->size(1) == W, "second result [rows, W]");
    TORCH_CHECK(has(open) && open->scalar_type() == torch::kFloat32 && open->is_contiguous() && open->numel() == rows, "its weights [rows] fp32");
    p.beside = beside->data_ptr(); p.open = open->data_ptr<float>();
  }
  c10::cuda::CUDAGuard guard(x.device());
  auto h = torch::empty(x.sizes(), w.options());
  if (rows == 0) return h;
  p.x = x.data_ptr<float>(); p.y = y.data_ptr(); p.next = w.data_ptr(); p.h = h.data_ptr();
  p.W = W; p.eps = eps; p.offset = offset;
  const bool vec = W % 4 == 0 && W <= 8192 && aligned16(p.y) && aligned16(p.next) && (p.beside == nullptr || aligned16(p.beside));
  const int nvec = (W + 3) / 4, vpt = nvec <= 512 ? 1 : (nvec <= 1024 ? 2 : 4);
  auto stream = at::cuda::getCurrentCUDAStream();
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const int threads = std::min(512, ((nvec + vpt - 1) / vpt + 31) / 32 * 32);
    if (!vec) stream_joined_rmsnorm_kernel<T, 0><<<rows, std::min(512, (W + 31) / 32 * 32), 0, stream>>>(p);
    else if (vpt == 1) stream_joined_rmsnorm_kernel<T, 1><<<rows, threads, 0, stream>>>(p);
    else if (vpt == 2) stream_joined_rmsnorm_kernel<T, 2><<<rows, threads, 0, stream>>>(p);
    else stream_joined_rmsnorm_kernel<T, 4><<<rows, threads, 0, stream>>>(p);
  };
  if (st == torch::kBFloat16) run(bf16{}); else run(float{});
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return h;
}

// ----------------------------------------------------------- stream_normed_add
// One block per row, as above.
struct NormedAdd {
  float* x;
  const void *y, *bias, *post, *inner, *beside, *beside_inner, *next;     // bias, beside (with the inner norms) and next may be null
  void* h;
  int W;
  float eps;
};

template <typename T, int VPT>
__global__ void stream_normed_add_kernel(const NormedAdd p) {
  __shared__ float sh[32], sh2[32];
  const int W = p.W, t = blockIdx.x;
  const size_t base = static_cast<size_t>(t) * W;
  const T *y = reinterpret_cast<const T*>(p.y) + base, *bias = reinterpret_cast<const T*>(p.bias), *post = reinterpret_cast<const T*>(p.post);
  const T *inner = reinterpret_cast<const T*>(p.inner), *beside = p.beside != nullptr ? reinterpret_cast<const T*>(p.beside) + base : nullptr;
  const T *beside_inner = reinterpret_cast<const T*>(p.beside_inner), *next = reinterpret_cast<const T*>(p.next);
  float* x = p.x + base;
  T* h = reinterpret_cast<T*>(p.h) + base;
  const float inv_w = 1.f / W;
  if constexpr (VPT > 0) {
    float4 z[VPT], v[VPT], b[VPT];
    float ss = 0.f, sb = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * 4;
      z[i] = v[i] = b[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < W) {
        z[i] = load4(y + c);
        v[i] = load4(x + c);
        if (beside != nullptr) b[i] = load4(beside + c);
        if (bias != nullptr) {
          const float4 a = load4(bias + c);
          z[i].x += a.x; z[i].y += a.y; z[i].z += a.z; z[i].w += a.w;
        }
      }
      ss += z[i].x * z[i].x + z[i].y * z[i].y + z[i].z * z[i].z + z[i].w * z[i].w;
      sb += b[i].x * b[i].x + b[i].y * b[i].y + b[i].z * b[i].z + b[i].w * b[i].w;
    }
    float r = rsqrtf(block_sum(ss, sh) * inv_w + p.eps);
    if (beside != nullptr) {
      const float rb = 0.5f * rsqrtf(block_sum(sb, sh2) * inv_w + p.eps);
      r *= 0.5f;
      ss = 0.f;
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int c = (i * blockDim.x + threadIdx.x) * 4;
        if (c < W) {
          const float4 w = load4(inner + c), u = load4(beside_inner + c);
          z[i].x = z[i].x * r * w.x + b[i].x * rb * u.x; z[i].y = z[i].y * r * w.y + b[i].y * rb * u.y;
          z[i].z = z[i].z * r * w.z + b[i].z * rb * u.z; z[i].w = z[i].w * r * w.w + b[i].w * rb * u.w;
        }
        ss += z[i].x * z[i].x + z[i].y * z[i].y + z[i].z * z[i].z + z[i].w * z[i].w;
      }
      r = rsqrtf(block_sum(ss, sh) * inv_w + p.eps);
    }
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * 4;
      if (c < W) {
        const float4 w = load4(post + c);
        v[i].x += z[i].x * r * w.x; v[i].y += z[i].y * r * w.y; v[i].z += z[i].z * r * w.z; v[i].w += z[i].w * r * w.w;
        store4(x + c, v[i]);
        if (next == nullptr) store4(h + c, v[i]);
      }
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    if (next == nullptr) return;
    r = rsqrtf(block_sum(ss, sh2) * inv_w + p.eps);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * 4;
      if (c < W) {
        const float4 w = load4(next + c);
        store4(h + c, make_float4(v[i].x * r * w.x, v[i].y * r * w.y, v[i].z * r * w.z, v[i].w * r * w.w));
      }
    }
  } else {                                   // any width: results are read once per pass
    auto own = [&](int c) { return to_f(y[c]) + (bias != nullptr ? to_f(bias[c]) : 0.f); };
    float ss = 0.f, sb = 0.f;
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
      const float a = own(c), b = beside != nullptr ? to_f(beside[c]) : 0.f;
      ss += a * a;
      sb += b * b;
    }
    float r = rsqrtf(block_sum(ss, sh) * inv_w + p.eps);
    const float ra = 0.5f * r, rb = 0.5f * rsqrtf(block_sum(sb, sh2) * inv_w + p.eps);
    auto joined = [&](int c) { return beside != nullptr ? own(c) * ra * to_f(inner[c]) + to_f(beside[c]) * rb * to_f(beside_inner[c]) : own(c); };
    if (beside != nullptr) {
      ss = 0.f;
      for (int c = threadIdx.x; c < W; c += blockDim.x) { const float z = joined(c); ss += z * z; }
      r = rsqrtf(block_sum(ss, sh) * inv_w + p.eps);
    }
    ss = 0.f;
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
      const float v = x[c] + joined(c) * r * to_f(post[c]);
      x[c] = v;
      if (next == nullptr) h[c] = from_f<T>(v);
      ss += v * v;
    }
    if (next == nullptr) return;
    r = rsqrtf(block_sum(ss, sh2) * inv_w + p.eps);
    for (int c = threadIdx.x; c < W; c += blockDim.x) h[c] = from_f<T>(x[c] * r * to_f(next[c]));
  }
}

// x [rows, W] fp32 is updated in place; returns the sum (or, with w, its norm) in y's dtype.
torch::Tensor stream_normed(torch::Tensor x, const OptT& w, double eps, const torch::Tensor& y, const OptT& bias, const torch::Tensor& post, const OptT& inner, const OptT& beside,
                            const OptT& beside_inner) {
  const auto st = y.scalar_type();
  TORCH_CHECK(x.is_cuda() && x.scalar_type() == torch::kFloat32 && x.is_contiguous() && x.dim() == 2, "stream [rows, W] fp32 contiguous");
  TORCH_CHECK(st == torch::kBFloat16 || st == torch::kFloat32, "bf16 or fp32");
  const int rows = x.size(0), W = x.size(1);
  bool vec = W % 4 == 0 && W <= 8192;
  auto check = [&](const OptT& t, int64_t n, const char* what) -> const void* {
    if (!has(t)) return nullptr;
    TORCH_CHECK(t->is_cuda() && t->scalar_type() == st && t->is_contiguous() && t->numel() == n, what);
    vec = vec && aligned16(t->data_ptr());
    return t->data_ptr();
  };
  TORCH_CHECK(has(beside) == has(inner) && has(beside) == has(beside_inner), "two results come with a norm each");
  NormedAdd p{};
  p.x = x.data_ptr<float>(); p.W = W; p.eps = eps;
  p.y = check(y, x.numel(), "result [rows, W]"); p.beside = check(beside, x.numel(), "second result [rows, W]");
  p.bias = check(bias, W, "bias [W]"); p.post = check(post, W, "norm weight [W]"); p.next = check(w, W, "norm weight [W]");
  p.inner = check(inner, W, "norm weight [W]"); p.beside_inner = check(beside_inner, W, "norm weight [W]");
  c10::cuda::CUDAGuard guard(x.device());
  auto h = torch::empty(x.sizes(), y.options());
  if (rows == 0) return h;
  p.h = h.data_ptr();
  const int nvec = (W + 3) / 4, vpt = nvec <= 512 ? 1 : (nvec <= 1024 ? 2 : 4);
  auto stream = at::cuda::getCurrentCUDAStream();
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const int threads = std::min(512, ((nvec + vpt - 1) / vpt + 31) / 32 * 32);
    if (!vec) stream_normed_add_kernel<T, 0><<<rows, std::min(512, (W + 31) / 32 * 32), 0, stream>>>(p);
    else if (vpt == 1) stream_normed_add_kernel<T, 1><<<rows, threads, 0, stream>>>(p);
    else if (vpt == 2) stream_normed_add_kernel<T, 2><<<rows, threads, 0, stream>>>(p);
    else stream_normed_add_kernel<T, 4><<<rows, threads, 0, stream>>>(p);
  };
  if (st == torch::kBFloat16) run(bf16{}); else run(float{});
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return h;
}

// ------------------------------------------------------------- embed_positions
// One block per row, a pair per thread at a time.  The angle is reduced to half turns in fp64, so that far positions keep their digits.
template <typename T>
__global__ void __launch_bounds__(256) embed_positions_kernel(const int64_t* __restrict__ ids, const T* __restrict__ weight, const int64_t* __restrict__ pos,
                                                              const double* __restrict__ freq, float* __restrict__ out, int pairs, int W) {
  const int t = blockIdx.x;
  const double at = static_cast<double>(pos[t]) * 0.31830988618379067154;
  const T* w = weight + static_cast<size_t>(ids[t]) * W;
  float* o = out + static_cast<size_t>(t) * W;
  for (int k = threadIdx.x; k < pairs; k += 256) {
    const double half_turns = at * freq[k];
    float s, c;
    sincospif(static_cast<float>(half_turns - 2.0 * rint(0.5 * half_turns)), &s, &c);
    if (W % 2 == 0) {
      *reinterpret_cast<float2*>(o + 2 * k) = make_float2(to_f(w[2 * k]) + s, to_f(w[2 * k + 1]) + c);
    } else {
      o[2 * k] = to_f(w[2 * k]) + s;
      if (2 * k + 1 < W) o[2 * k + 1] = to_f(w[2 * k + 1]) + c;
    }
  }
}

torch::Tensor embed_positions(const torch::Tensor& ids, const torch::Tensor& weight, const torch::Tensor& pos, const torch::Tensor& freq) {
  const auto st = weight.scalar_type();
  TORCH_CHECK(weight.is_cuda() && weight.dim() == 2 && weight.is_contiguous() && (st == torch::kBFloat16 || st == torch::kFloat32), "embedding [vocab, W] bf16 or fp32");
  TORCH_CHECK(ids.is_cuda() && ids.scalar_type() == torch::kInt64 && ids.is_contiguous() && pos.is_cuda() && pos.scalar_type() == torch::kInt64 && pos.is_contiguous() &&
                  ids.dim() == 1 && ids.numel() == pos.numel(), "token ids and positions int64 [rows]");
  const int W = weight.size(1), pairs = (W + 1) / 2;
  TORCH_CHECK(freq.is_cuda() && freq.scalar_type() == torch::kFloat64 && freq.is_contiguous() && freq.numel() == pairs, "frequencies fp64 [pairs]");
  c10::cuda::CUDAGuard guard(weight.device());
  auto out = torch::empty({ids.numel(), W}, weight.options().dtype(torch::kFloat32));
  if (out.numel() == 0) return out;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    embed_positions_kernel<T><<<static_cast<unsigned>(ids.numel()), 256, 0, at::cuda::getCurrentCUDAStream()>>>(
        ids.data_ptr<int64_t>(), reinterpret_cast<const T*>(weight.data_ptr()), pos.data_ptr<int64_t>(), freq.data_ptr<double>(), out.data_ptr<float>(), pairs, W);
  };
  if (st == torch::kBFloat16) run(bf16{}); else run(float{});
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return out;
}

// ----------------------------------------------------------------- glu_columns
// ACT 0: silu(g) · u; 1: g σ(1.702 g) (u + 1) on g ≤ limit, |u| ≤ limit; 2: gelu in its tanh form times u (½ (1 + tanh a) = σ(2a)).
template <int ACT>
__device__ __forceinline__ float glu(float g, float u, float limit) {
  if constexpr (ACT == 2) return g / (1.f + __expf(-1.5957691216057308f * fmaf(0.044715f * g * g, g, g))) * u;
  if constexpr (ACT == 1) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.f + __expf(-1.702f * g)) * (u + 1.f);
  }
  return g / (1.f + __expf(-g)) * u;
}

template <typename T, int V, int ACT>
__global__ void __launch_bounds__(256) glu_columns_kernel(const T* __restrict__ p, long ld, int gate, int up, T* __restrict__ out, long rows, int I, float limit) {
  const int per_row = I / V;
  const long total = rows * per_row;
  for (long i = blockIdx.x * static_cast<long>(blockDim.x) + threadIdx.x; i < total; i += static_cast<long>(gridDim.x) * blockDim.x) {
    const long r = total < (1L << 31) ? static_cast<long>(static_cast<uint32_t>(i) / static_cast<uint32_t>(per_row)) : i / per_row;
    const int c = static_cast<int>(i - r * per_row) * V;
    const T* g = p + r * ld + gate + c;
    const T* u = p + r * ld + up + c;
    T* o = out + r * I + c;
    if constexpr (V == 8) {        // bf16: 16-byte accesses
      const uint4 a = *reinterpret_cast<const uint4*>(g), b = *reinterpret_cast<const uint4*>(u);
      const uint32_t pa[4] = {a.x, a.y, a.z, a.w}, pb[4] = {b.x, b.y, b.z, b.w};
      uint32_t po[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float2 x = unpack_bf16(pa[k]), y = unpack_bf16(pb[k]);
        po[k] = pack_bf16(glu<ACT>(x.x, y.x, limit), glu<ACT>(x.y, y.y, limit));
      }
      *reinterpret_cast<uint4*>(o) = make_uint4(po[0], po[1], po[2], po[3]);
    } else {
#pragma unroll
      for (int k = 0; k < V; ++k) o[k] = from_f<T>(glu<ACT>(to_f(g[k]), to_f(u[k]), limit));
    }
  }
}

torch::Tensor glu_columns(const torch::Tensor& p, int64_t gate, int64_t up, int64_t I, double limit, bool gelu) {
  const auto st = p.scalar_type();
  TORCH_CHECK(p.is_cuda() && p.dim() == 2 && p.stride(1) == 1 && (st == torch::kBFloat16 || st == torch::kFloat32), "projection [rows, N] bf16 or fp32");
  TORCH_CHECK(I > 0 && gate >= 0 && up >= 0 && gate + I <= p.size(1) && up + I <= p.size(1) && limit >= 0, "gate / up columns outside the projection, or a negative limit");
  const long rows = p.size(0), ld = p.stride(0);
  c10::cuda::CUDAGuard guard(p.device());
  auto out = torch::empty({rows, I}, p.options());
  if (rows == 0) return out;
  auto stream = at::cuda::getCurrentCUDAStream();
  const bool vec = st == torch::kBFloat16 && I % 8 == 0 && gate % 8 == 0 && up % 8 == 0 && ld % 8 == 0 && aligned16(p.data_ptr());
  const long total = rows * (vec ? I / 8 : I);
  const int blocks = static_cast<int>(std::min<long>((total + 255) / 256, num_sms() * 16L));
  auto go = [&](auto tag, auto width) {
    using T = decltype(tag);
    constexpr int V = decltype(width)::value;
    const T* in = reinterpret_cast<const T*>(p.data_ptr());
    T* o = reinterpret_cast<T*>(out.data_ptr());
    if (gelu) glu_columns_kernel<T, V, 2><<<blocks, 256, 0, stream>>>(in, ld, gate, up, o, rows, I, 0.f);
    else if (limit > 0) glu_columns_kernel<T, V, 1><<<blocks, 256, 0, stream>>>(in, ld, gate, up, o, rows, I, static_cast<float>(limit));
    else glu_columns_kernel<T, V, 0><<<blocks, 256, 0, stream>>>(in, ld, gate, up, o, rows, I, 0.f);
  };
  if (vec) go(bf16{}, std::integral_constant<int, 8>{});
  else if (st == torch::kBFloat16) go(bf16{}, std::integral_constant<int, 1>{});
  else go(float{}, std::integral_constant<int, 1>{});
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return out;
}

}  // namespace tk
