// Mixture-of-experts steps of inference, all without host reads (they are captured into decode graphs):
//   moe_topk          fp32 router logits (+ bias) → the k largest, a softmax over just those, and tokens per expert; or a softmax over
//                     all and a choice among the best groups; the shared expert's sigmoid weight on the way
//   moe_group_rows    token rows copied next to the rows of the same expert, nothing between experts: every expert's range comes
//                     from the histogram, a row's place inside it from an atomic counter (rows do not interact, so their order
//                     inside an expert does not matter)
//   grouped_gemm_f32  per-expert product in true fp32 for 32-bit models (bf16 runs the tcgen05 kernel of gemm.cu)
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/types.h>

#include "common.cuh"
#include "host.h"
#include "vec.cuh"

namespace tk {

namespace ms {
__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const bf16* p) { return __bfloat162float(*p); }
}  // namespace ms

struct Choice {
  int rows, E, k;
  int groups, keep;                      // groups 0: a softmax over the chosen; otherwise over all, and only the `keep` best groups count
  float factor;                          // on the weights of the second form
  const void *x, *shared; long ldx;      // [rows, width], [width]: open[t] = σ(x_t · shared) (nullptr: not wanted)
  float* open; int width;
};

// One warp per token, up to 32·PER experts.
template <typename T, int PER>
__global__ void __launch_bounds__(256) moe_topk_kernel(const float* __restrict__ logits, long ld, const T* __restrict__ bias, const int64_t* __restrict__ forced,
                                                       float* __restrict__ weights, int64_t* __restrict__ indices, int* __restrict__ hist, const Choice p) {
  const int lane = threadIdx.x & 31, rows = p.rows, E = p.E, k = p.k, size = p.groups > 0 ? E / p.groups : E;
  for (int t = blockIdx.x * 8 + (threadIdx.x >> 5); t < rows; t += gridDim.x * 8) {
    if (p.shared != nullptr) {
      const T *x = reinterpret_cast<const T*>(p.x) + t * p.ldx, *w = reinterpret_cast<const T*>(p.shared);
      float s = 0.f;
      if (p.width % 8 == 0 && p.ldx % 8 == 0 && aligned16(p.x) && aligned16(p.shared)) {
        for (int c = lane * 8; c < p.width; c += 256) {
          Raw8<T> a, b;
          a.load(x + c);
          b.load(w + c);
          float u[8], v[8];
          a.get(u);
          b.get(v);
#pragma unroll
          for (int i = 0; i < 8; ++i) s += u[i] * v[i];
        }
      } else {
        for (int c = lane; c < p.width; c += 32) s += ms::ld(x + c) * ms::ld(w + c);
      }
      s = warp_sum(s);
      if (lane == 0) p.open[t] = 1.f / (1.f + __expf(-s));
    }
    float z[PER];
#pragma unroll
    for (int j = 0; j < PER; ++j) {
      const int e = j * 32 + lane;
      z[j] = e < E ? logits[t * ld + e] + (bias != nullptr ? ms::ld(bias + e) : 0.f) : -INFINITY;
    }
    // the largest logit among experts outside `taken`: same result in every lane
    auto largest = [&](uint32_t taken, float& best, int& be) {
      best = -INFINITY;
      be = 1 << 30;
#pragma unroll
      for (int j = 0; j < PER; ++j)
        if (!(taken >> j & 1) && j * 32 + lane < E && (z[j] > best || be == 1 << 30)) { best = z[j]; be = j * 32 + lane; }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ob = __shfl_xor_sync(0xffffffffu, best, o);
        const int oe = __shfl_xor_sync(0xffffffffu, be, o);
        if (ob > best || (ob == best && oe < be)) { best = ob; be = oe; }
      }
    };
    float mine = -INFINITY;
    int my_e = 0;
    const bool given = forced != nullptr && forced[static_cast<size_t>(t) * k] >= 0;
    if (given) {
      if (lane < k) {
        my_e = min(max(static_cast<int>(forced[static_cast<size_t>(t) * k + lane]), 0), E - 1);
        mine = logits[t * ld + my_e] + (bias != nullptr ? ms::ld(bias + my_e) : 0.f);
      }
    } else {
      uint32_t taken = 0;
      if (p.groups > 1 && p.keep < p.groups) {         // a group is as good as its best expert: the next best outside the groups so far names one
        uint32_t inside = 0;
        for (int r = 0; r < p.keep; ++r) {
          float best;
          int be;
          largest(inside, best, be);
#pragma unroll
          for (int j = 0; j < PER; ++j)
            if ((j * 32 + lane) / size == be / size) inside |= 1u << j;
        }
        taken = ~inside;
      }
      for (int r = 0; r < k; ++r) {
        float best;
        int be;
        largest(taken, best, be);
        if ((be & 31) == lane && be < (1 << 30)) taken |= 1u << (be >> 5);
        if (lane == r) { mine = best; my_e = min(be, E - 1); }   // logits that are not numbers still name an expert that exists
      }
    }
    float over = mine;                                  // the softmax runs over the chosen, or over all
    if (p.groups > 0) {
#pragma unroll
      for (int j = 0; j < PER; ++j) over = j == 0 ? z[0] : fmaxf(over, z[j]);
    }
    const float mx = warp_max(over), w = lane < k ? __expf(mine - mx) : 0.f;
    float part = w;
    if (p.groups > 0) {
      part = 0.f;
#pragma unroll
      for (int j = 0; j < PER; ++j) part += j * 32 + lane < E ? __expf(z[j] - mx) : 0.f;
    }
    const float sum = warp_sum(part);
    if (lane < k) {
      weights[static_cast<size_t>(t) * k + lane] = p.groups > 0 ? w / sum * p.factor : w / sum;
      indices[static_cast<size_t>(t) * k + lane] = my_e;
      atomicAdd(hist + my_e, 1);
    }
  }
}

// Returns {weights, experts, tokens per expert} and, with `shared`, its weight per token.
std::vector<torch::Tensor> moe_topk(const torch::Tensor& logits, const OptT& bias, int64_t k, const OptT& forced, int64_t groups, int64_t keep, double factor,
                                    const OptT& x, const OptT& shared) {
  TORCH_CHECK(logits.is_cuda() && logits.dim() == 2 && logits.scalar_type() == torch::kFloat32 && logits.stride(1) == 1, "router logits [T, E] fp32");
  const int rows = logits.size(0), E = logits.size(1);
  TORCH_CHECK(E >= 1 && E <= 256 && k >= 1 && k <= 32 && k <= E, "up to 256 experts and top-32");
  TORCH_CHECK(groups >= 0 && (groups == 0 || (E % groups == 0 && keep >= 1 && keep <= groups && k <= E / groups * keep)), "equal groups that hold enough experts");
  const bool has_bias = has(bias), has_forced = has(forced), has_shared = has(shared);
  auto dt = has_bias ? bias->scalar_type() : torch::kFloat32;
  if (has_shared) {
    TORCH_CHECK(has(x) && x->is_cuda() && x->dim() == 2 && x->size(0) == rows && x->stride(1) == 1 && shared->is_cuda() && shared->is_contiguous() && shared->numel() == x->size(1) &&
                    shared->scalar_type() == x->scalar_type() && (x->scalar_type() == torch::kBFloat16 || x->scalar_type() == torch::kFloat32), "x [T, H] and shared [H] in one dtype");
    TORCH_CHECK(!has_bias || dt == x->scalar_type(), "bias in x's dtype");
    dt = x->scalar_type();
  }
  if (has_bias) TORCH_CHECK(bias->is_cuda() && bias->is_contiguous() && bias->numel() == E && (bias->scalar_type() == torch::kBFloat16 || bias->scalar_type() == torch::kFloat32), "router bias [E]");
  if (has_forced) TORCH_CHECK(forced->is_cuda() && forced->scalar_type() == torch::kInt64 && forced->is_contiguous() && forced->numel() == rows * k, "forced experts int64 [T, k]");
  c10::cuda::CUDAGuard guard(logits.device());
  auto w = torch::empty({rows, k}, logits.options());
  auto idx = torch::empty({rows, k}, logits.options().dtype(torch::kInt64));
  auto hist = torch::zeros({E}, logits.options().dtype(torch::kInt32));
  auto open = torch::empty({has_shared ? rows : 0}, logits.options());
  std::vector<torch::Tensor> out{w, idx, hist};
  if (has_shared) out.push_back(open);
  if (rows == 0) return out;
  Choice p{};
  p.rows = rows; p.E = E; p.k = k; p.groups = groups; p.keep = keep; p.factor = factor;
  if (has_shared) { p.x = x->data_ptr(); p.ldx = x->stride(0); p.shared = shared->data_ptr(); p.open = open.data_ptr<float>(); p.width = x->size(1); }
  const int blocks = std::min((rows + 7) / 8, num_sms() * 8);
  auto stream = at::cuda::getCurrentCUDAStream();
  auto run = [&](auto tag) {
    using T = decltype(tag);
    auto go = [&](auto kern) {
      kern<<<blocks, 256, 0, stream>>>(logits.data_ptr<float>(), logits.stride(0), has_bias ? reinterpret_cast<const T*>(bias->data_ptr()) : nullptr,
                                       has_forced ? forced->data_ptr<int64_t>() : nullptr, w.data_ptr<float>(), idx.data_ptr<int64_t>(), hist.data_ptr<int>(), p);
    };
    if (E <= 32) go(moe_topk_kernel<T, 1>); else if (E <= 64) go(moe_topk_kernel<T, 2>); else if (E <= 128) go(moe_topk_kernel<T, 4>); else go(moe_topk_kernel<T, 8>);
  };
  if (dt == torch::kBFloat16) run(bf16{}); else run(float{});
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return out;
}

// One warp per (token, choice).  Every block forms the expert ranges from the histogram for itself (≤ 256 numbers).
template <int B>   // bytes per access
__global__ void __launch_bounds__(256) moe_group_rows_kernel(const uint8_t* __restrict__ x, const int64_t* __restrict__ idx, const int* __restrict__ hist, int* cursor,
                                                             uint8_t* __restrict__ out, int* __restrict__ row_of, int* __restrict__ offsets, int pairs, int k, int E,
                                                             long row_bytes) {
  __shared__ int s_off[256], s_sum[8];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  int c = tid < E ? hist[tid] : 0, up = c;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) { const int v = __shfl_up_sync(0xffffffffu, up, o); if (lane >= o) up += v; }
  if (lane == 31) s_sum[warp] = up;
  __syncthreads();
  int before = 0;
  for (int w = 0; w < warp; ++w) before += s_sum[w];
  s_off[tid] = before + up - c;
  if (blockIdx.x == 0 && tid < E) {
    offsets[tid] = before + up - c;
    if (tid == E - 1) offsets[E] = before + up;
  }
  __syncthreads();
  for (int i = blockIdx.x * 8 + warp; i < pairs; i += gridDim.x * 8) {
    int row = 0;
    if (lane == 0) {
      const int e = static_cast<int>(idx[i]);
      row = s_off[e] + atomicAdd(cursor + e, 1);
      row_of[i] = row;
    }
    row = __shfl_sync(0xffffffffu, row, 0);
    const uint8_t* src = x + static_cast<size_t>(i / k) * row_bytes;
    uint8_t* dst = out + static_cast<size_t>(row) * row_bytes;
    if constexpr (B == 16) {
      const uint4* s = reinterpret_cast<const uint4*>(src);
      uint4* d = reinterpret_cast<uint4*>(dst);
      const int n = static_cast<int>(row_bytes >> 4);
      int v = lane;
      for (; v + 96 < n; v += 128) {
        const uint4 a = s[v], b = s[v + 32], c4 = s[v + 64], d4 = s[v + 96];
        d[v] = a; d[v + 32] = b; d[v + 64] = c4; d[v + 96] = d4;
      }
      for (; v < n; v += 32) d[v] = s[v];
    } else {
      for (long v = lane; v < row_bytes / 2; v += 32) reinterpret_cast<uint16_t*>(dst)[v] = reinterpret_cast<const uint16_t*>(src)[v];
    }
  }
}

std::vector<torch::Tensor> moe_group_rows(const torch::Tensor& x, const torch::Tensor& idx, const torch::Tensor& hist) {
  TORCH_CHECK(x.is_cuda() && x.dim() == 2 && x.is_contiguous() && (x.scalar_type() == torch::kBFloat16 || x.scalar_type() == torch::kFloat32), "x [T, H] bf16 or fp32");
  TORCH_CHECK(idx.is_cuda() && idx.scalar_type() == torch::kInt64 && idx.dim() == 2 && idx.is_contiguous() && idx.size(0) == x.size(0), "idx int64 [T, k]");
  TORCH_CHECK(hist.is_cuda() && hist.scalar_type() == torch::kInt32 && hist.is_contiguous() && hist.numel() >= 1 && hist.numel() <= 256, "histogram int32 [E <= 256]");
  c10::cuda::CUDAGuard guard(x.device());
  const int T = x.size(0), k = idx.size(1), E = hist.numel(), pairs = T * k;
  auto i32 = hist.options();
  auto out = torch::empty({pairs, x.size(1)}, x.options());
  auto row_of = torch::empty({T, k}, i32);
  auto offsets = torch::empty({E + 1}, i32);
  if (pairs == 0) return {out, row_of, offsets.zero_()};
  auto cursor = torch::zeros({E}, i32);
  const long bytes = x.size(1) * x.element_size();
  const int blocks = std::min((pairs + 7) / 8, num_sms() * 8);
  auto stream = at::cuda::getCurrentCUDAStream();
  auto go = [&](auto kern) {
    kern<<<blocks, 256, 0, stream>>>(reinterpret_cast<const uint8_t*>(x.data_ptr()), idx.data_ptr<int64_t>(), hist.data_ptr<int>(), cursor.data_ptr<int>(),
                                     reinterpret_cast<uint8_t*>(out.data_ptr()), row_of.data_ptr<int>(), offsets.data_ptr<int>(), pairs, k, E, bytes);
  };
  if (bytes % 16 == 0 && reinterpret_cast<uintptr_t>(x.data_ptr()) % 16 == 0) go(moe_group_rows_kernel<16>); else go(moe_group_rows_kernel<2>);
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return {out, row_of, offsets};
}

// 64 × 64 tile of one expert's rows, 256 threads of 4 × 4 sums, 16 columns of the reduction at a time.
template <bool RELU2>
__global__ void __launch_bounds__(256) grouped_gemm_f32_kernel(const float* __restrict__ x, const float* __restrict__ w, const int* __restrict__ offsets,
                                                               float* __restrict__ out, int E, int N, int K) {
  constexpr int TILE = 64, KB = 16;
  __shared__ float s_x[KB][TILE + 4], s_w[KB][TILE + 4];
  int tile = blockIdx.y, e = 0, m0 = 0, m1 = 0;
  for (; e < E; ++e) {
    const int a = offsets[e], b = offsets[e + 1], tiles = (b - a + TILE - 1) / TILE;
    if (tile < tiles) { m0 = a + tile * TILE; m1 = b; break; }
    tile -= tiles;
  }
  if (e == E) return;
  const int n0 = blockIdx.x * TILE, tid = threadIdx.x, ty = tid >> 4, tx = tid & 15;
  const float* we = w + static_cast<size_t>(e) * N * K;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += KB) {
    __syncthreads();
    for (int i = tid; i < TILE * KB; i += 256) {
      const int r = i / KB, c = i % KB;
      s_x[c][r] = m0 + r < m1 && k0 + c < K ? x[static_cast<size_t>(m0 + r) * K + k0 + c] : 0.f;
      s_w[c][r] = n0 + r < N && k0 + c < K ? we[static_cast<size_t>(n0 + r) * K + k0 + c] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < KB; ++c) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = s_x[c][ty * 4 + i]; b[i] = s_w[c][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = m0 + ty * 4 + i, c = n0 + tx * 4 + j;
      if (r >= m1 || c >= N) continue;
      float v = acc[i][j];
      if constexpr (RELU2) { v = fmaxf(v, 0.f); v *= v; }
      out[static_cast<size_t>(r) * N + c] = v;
    }
}

torch::Tensor grouped_gemm_f32(const torch::Tensor& x, const torch::Tensor& w, const torch::Tensor& offsets, bool relu2) {
  TORCH_CHECK(x.is_cuda() && x.scalar_type() == torch::kFloat32 && x.dim() == 2 && x.is_contiguous(), "x [R, K] fp32");
  TORCH_CHECK(w.is_cuda() && w.scalar_type() == torch::kFloat32 && w.dim() == 3 && w.is_contiguous() && w.size(2) == x.size(1), "weight [E, N, K] fp32");
  TORCH_CHECK(offsets.is_cuda() && offsets.scalar_type() == torch::kInt32 && offsets.is_contiguous() && offsets.numel() == w.size(0) + 1, "offsets int32 [E+1]");
  c10::cuda::CUDAGuard guard(x.device());
  const int R = x.size(0), K = x.size(1), E = w.size(0), N = w.size(1);
  auto out = torch::empty({R, N}, x.options());
  if (R == 0 || N == 0) return out;
  const int tiles = std::min(R, (R + 63) / 64 + E);      // every expert wastes at most one partial tile
  TORCH_CHECK(tiles <= 65535, "too many rows");
  auto stream = at::cuda::getCurrentCUDAStream();
  const dim3 grid((N + 63) / 64, tiles);
  if (relu2) grouped_gemm_f32_kernel<true><<<grid, 256, 0, stream>>>(x.data_ptr<float>(), w.data_ptr<float>(), offsets.data_ptr<int>(), out.data_ptr<float>(), E, N, K);
  else grouped_gemm_f32_kernel<false><<<grid, 256, 0, stream>>>(x.data_ptr<float>(), w.data_ptr<float>(), offsets.data_ptr<int>(), out.data_ptr<float>(), E, N, K);
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return out;
}

}  // namespace tk
