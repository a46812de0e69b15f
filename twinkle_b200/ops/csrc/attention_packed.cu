// Causal attention over packed sequences in fp32 arithmetic, any key / value widths up to 256, grouped heads, optionally within a
// window or chunk: the prefill kernel for 32-bit models and for heads wider than the tensor-core kernel takes (attention_fwd.cu).
//
// One block per (32 query rows of one sequence, query head), 256 threads: eight threads per row.  Keys and values pass through
// shared memory 32 rows at a time; a thread scores four keys of the tile and owns every eighth output column of its row.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/types.h>

#include "common.cuh"
#include "host.h"
#include "scores.cuh"

namespace tk {

using bf16 = __nv_bfloat16;

namespace pa {
constexpr int BQ = 32, BK = 32;
__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(bf16* p, float v) { *p = __float2bfloat16(v); }
}  // namespace pa

template <typename T, int EI>
__global__ void __launch_bounds__(256) attention_packed_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, T* __restrict__ out,
                                                               const int* __restrict__ cu, int hq, int hkv, int D, int E, float scale_log2,
                                                               const T* __restrict__ sinks, const OutGate gate, int window, int chunk, const ScoreTerms terms) {
  using namespace pa;
  extern __shared__ float sm[];
  const int head = blockIdx.x, seq = blockIdx.z, kvh = head / (hq / hkv);
  const int start = cu[seq], len = cu[seq + 1] - start;
  const int tiles = (len + BQ - 1) / BQ;
  if (static_cast<int>(blockIdx.y) >= tiles) return;
  const int q0 = (tiles - 1 - blockIdx.y) * BQ;    // the longest rows first
  const int ds = D + 1;                             // odd row pitch when D is even: eight rows fall into eight banks
  float* sq = sm;
  float* sk = sq + BQ * ds;
  float* sv = sk + BK * ds;
  float* sp = sv + BK * E;
  const int row = threadIdx.x >> 3, sub = threadIdx.x & 7;
  const DistanceNumber<T> number(terms, head);
  const float q_scale = terms.used ? scale_log2 * 0.6931471805599453f * score_temp<T>(terms, head) : scale_log2;
  for (int i = threadIdx.x; i < BQ * D; i += blockDim.x) {
    const int r = i / D, c = i - r * D;
    sq[r * ds + c] = q0 + r < len ? ld(q + (static_cast<size_t>(start + q0 + r) * hq + head) * D + c) * q_scale : 0.f;
  }
  float acc[EI];
#pragma unroll
  for (int i = 0; i < EI; ++i) acc[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  const int end = min(len, q0 + BQ), first = first_visible(q0 + row, window, chunk);
  for (int k0 = first_visible(q0, window, chunk) / BK * BK; k0 < end; k0 += BK) {
    __syncthreads();
    for (int i = threadIdx.x; i < BK * D; i += blockDim.x) {
      const int r = i / D, c = i - r * D;
      sk[r * ds + c] = k0 + r < len ? ld(k + (static_cast<size_t>(start + k0 + r) * hkv + kvh) * D + c) : 0.f;
    }
    for (int i = threadIdx.x; i < BK * E; i += blockDim.x) {
      const int r = i / E, c = i - r * E;
      sv[i] = k0 + r < len ? ld(v + (static_cast<size_t>(start + k0 + r) * hkv + kvh) * E + c) : 0.f;
    }
    __syncthreads();
    float s[4] = {0.f, 0.f, 0.f, 0.f};
    for (int c = 0; c < D; ++c) {
      const float a = sq[row * ds + c];
#pragma unroll
      for (int i = 0; i < 4; ++i) s[i] += a * sk[(sub + 8 * i) * ds + c];
    }
    if (terms.used) {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        if (terms.cap > 0.f) s[i] = terms.cap * tanh_any(s[i] * terms.inv_cap);
        s[i] = (s[i] + number.at(max(q0 + row - k0 - sub - 8 * i, 0))) * 1.4426950408889634f;
      }
    }
    float mx = m;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      if (k0 + sub + 8 * i > q0 + row || k0 + sub + 8 * i < first || k0 + sub + 8 * i >= len) s[i] = -INFINITY;
      mx = fmaxf(mx, s[i]);
    }
#pragma unroll
    for (int o = 1; o < 8; o <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    // a row may not see any key of its tile's first keys
    const float base = mx == -INFINITY ? 0.f : mx, corr = exp2f(m - base);
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float pr = exp2f(s[i] - base);
      sp[row * (BK + 1) + sub + 8 * i] = pr;
      sum += pr;
    }
#pragma unroll
    for (int o = 1; o < 8; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    l = l * corr + sum;
    m = mx;
    __syncwarp();                                   // the eight threads of a row are in one warp
#pragma unroll
    for (int i = 0; i < EI; ++i) acc[i] *= corr;
    for (int j = 0; j < BK; ++j) {
      const float pr = sp[row * (BK + 1) + j];
#pragma unroll
      for (int i = 0; i < EI; ++i)
        if (sub + 8 * i < E) acc[i] += pr * sv[j * E + sub + 8 * i];
    }
  }
  if (q0 + row < len) {
    T* o = out + (static_cast<size_t>(start + q0 + row) * hq + head) * E;
    if (sinks != nullptr) l += exp2f(ld(sinks + head) * 1.4426950408889634f - m);      // a key without a value that every row sees
    float f = 1.f / l;
    const T* g = gate.p != nullptr ? reinterpret_cast<const T*>(gate.p) + static_cast<size_t>(start + q0 + row) * gate.ld + static_cast<size_t>(head) * max(gate.e, 1) : nullptr;
    if (g != nullptr && gate.e == 0) f *= sigmoid_of(ld(g));
#pragma unroll
    for (int i = 0; i < EI; ++i) {
      const int c = sub + 8 * i;
      if (c < E) st(o + c, acc[i] * f * (g != nullptr && c < gate.e ? sigmoid_of(ld(g + c)) : 1.f));
    }
  }
}

torch::Tensor attention_packed(const torch::Tensor& q, const torch::Tensor& k, const torch::Tensor& v, const torch::Tensor& cu, int64_t max_seqlen, double scale,
                               const c10::optional<torch::Tensor>& sinks, const c10::optional<torch::Tensor>& gate, int64_t window, int64_t chunk,
                               double cap, const c10::optional<torch::Tensor>& temp, const c10::optional<torch::Tensor>& slope, const c10::optional<torch::Tensor>& rate, const c10::optional<torch::Tensor>& table, const c10::optional<torch::Tensor>& bucket) {
  const auto st = q.scalar_type();
  TORCH_CHECK(q.is_cuda() && (st == torch::kBFloat16 || st == torch::kFloat32) && k.scalar_type() == st && v.scalar_type() == st, "q, k, v bf16 or fp32");
  TORCH_CHECK(q.dim() == 3 && k.dim() == 3 && v.dim() == 3 && q.is_contiguous() && k.is_contiguous() && v.is_contiguous(), "[T, H, D] contiguous");
  TORCH_CHECK(q.size(2) == k.size(2) && k.size(0) == q.size(0) && v.size(0) == q.size(0) && k.size(1) == v.size(1) && q.size(1) % k.size(1) == 0, "shapes of q, k, v");
  TORCH_CHECK(q.size(2) <= 256 && v.size(2) <= 256, "head widths up to 256");
  TORCH_CHECK(window >= 0 && chunk >= 0 && window < (int64_t(1) << 30) && chunk < (int64_t(1) << 30), "window and chunk: 0 (none) or positive");
  TORCH_CHECK(cu.is_cuda() && cu.scalar_type() == torch::kInt32 && cu.is_contiguous(), "cu_seqlens int32 on device");
  const bool has_sinks = sinks.has_value() && sinks->defined();
  if (has_sinks) TORCH_CHECK(sinks->is_cuda() && sinks->scalar_type() == st && sinks->is_contiguous() && sinks->numel() == q.size(1), "sinks [Hq]");
  const OutGate g = out_gate(gate, q.size(0), q.size(1), v.size(2), st);
  const ScoreTerms terms = score_terms(cap, temp, slope, rate, table, bucket, q.size(1), st);
  c10::cuda::CUDAGuard guard(q.device());
  const int hq = q.size(1), hkv = k.size(1), D = q.size(2), E = v.size(2), nseq = cu.numel() - 1;
  auto out = torch::empty({q.size(0), hq, E}, q.options());
  if (q.size(0) == 0 || nseq <= 0 || max_seqlen <= 0) return out;
  const size_t smem = sizeof(float) * ((pa::BQ + pa::BK) * static_cast<size_t>(D + 1) + pa::BK * static_cast<size_t>(E) + pa::BQ * (pa::BK + 1));
  const dim3 grid(hq, (static_cast<int>(max_seqlen) + pa::BQ - 1) / pa::BQ, nseq);
  auto stream = at::cuda::getCurrentCUDAStream();
  auto go = [&](auto kern, auto tag) {
    using T = decltype(tag);
    TK_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
    kern<<<grid, 256, smem, stream>>>(reinterpret_cast<const T*>(q.data_ptr()), reinterpret_cast<const T*>(k.data_ptr()), reinterpret_cast<const T*>(v.data_ptr()),
                                      reinterpret_cast<T*>(out.data_ptr()), cu.data_ptr<int>(), hq, hkv, D, E, static_cast<float>(scale * 1.4426950408889634),
                                      has_sinks ? reinterpret_cast<const T*>(sinks->data_ptr()) : nullptr, g, static_cast<int>(window),
                                      static_cast<int>(chunk), terms);
  };
  if (st == torch::kBFloat16) {
    if (E <= 64) go(attention_packed_kernel<bf16, 8>, bf16{});
    else if (E <= 128) go(attention_packed_kernel<bf16, 16>, bf16{});
    else go(attention_packed_kernel<bf16, 32>, bf16{});
  } else {
    if (E <= 64) go(attention_packed_kernel<float, 8>, 0.f);
    else if (E <= 128) go(attention_packed_kernel<float, 16>, 0.f);
    else go(attention_packed_kernel<float, 32>, 0.f);
  }
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return out;
}

}  // namespace tk
