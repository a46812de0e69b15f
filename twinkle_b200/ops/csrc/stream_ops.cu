// Element-wise steps of decoder layers whose residual stream is 32-bit and whose mixer and feed-forward block read one
// fused projection [q | k | v | gate | up]:
//   conv_heads      short causal convolution on q, k and v, q / k over their root mean square per head, query temperature,
//                   value mixing, and the writes into the paged K/V pools and the convolution history — one pass
//   stream_rmsnorm  x += mult · (y1 ⊙ s1 + y2 ⊙ s2) in fp32 and the RMS norm of the sum in the compute dtype — one pass
//   stream_gated_rmsnorm  x += norm(σ(gate + bias) ⊙ y) in fp32 and the RMS norm of the sum — one pass; y is a row of its own or
//                   the weighted sum of a token's expert rows
//   glu_columns     silu(gate) · up on two column ranges of the projection
// All are templated on the compute dtype (bf16 or fp32) and work for any width: vector kernels where rows are made of
// whole vectors, plain ones otherwise.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/types.h>

#include "common.cuh"
#include "host.h"

namespace tk {

using bf16 = __nv_bfloat16;

template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<bf16>(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16(v); }

// four consecutive elements as fp32
__device__ __forceinline__ float4 load4(const bf16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16(u.x), b = unpack_bf16(u.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void store4(bf16* p, const float4& v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}
__device__ __forceinline__ void store4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }

__device__ __forceinline__ float block_sum(float v, float* sh) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = (blockDim.x + 31) >> 5;
  __syncthreads();
  if (lane == 0) sh[warp] = v;
  __syncthreads();
  return warp_sum(lane < nw ? sh[lane] : 0.f);
}

// ------------------------------------------------------------------ conv_heads
template <typename T>
struct ConvHeads {
  const T* proj; long ld;               // [rows, ld]: q | k | v in the leading columns
  const T* w;                           // [C, taps] (nullptr: no convolution)
  int taps;
  int hq, hkv, d, e;                    // heads and widths
  int dp, ep;                           // row widths of the outputs and pools (≥ d, e; the rest is written as zero)
  float eps, coef; int every;           // query temperature (every = 0: none)
  const int64_t* pos;                   // place of every row in its sequence
  T *q, *k, *v;                         // [rows, hq, dp], [rows, hkv, dp] (may be null), [rows, hkv, ep]
  const T* v_first; const T* lam;       // [rows, hkv, ep], [1] (null: values are not mixed)
  T *k_pool, *v_pool; const int64_t* pool_row;   // [·, hkv, dp], [·, hkv, ep]; row of every token (< 0: not kept)
  T* hist; const int* slot; const int* left;     // [slots, taps − 1, C]; left[t] = later rows of the same sequence in this call
  int rows;
};

template <typename T>
__device__ __forceinline__ float query_factor(const ConvHeads<T>& p, int pos) {
  return p.every > 0 ? 1.f + p.coef * log1pf(static_cast<float>(static_cast<uint32_t>(pos + 1) / static_cast<uint32_t>(p.every))) : 1.f;
}

// Eight consecutive elements as they lie in memory.
template <typename T> struct Raw8;
template <> struct Raw8<bf16> {
  uint4 u;
  __device__ __forceinline__ void load(const bf16* p) { u = *reinterpret_cast<const uint4*>(p); }
  __device__ __forceinline__ void store(bf16* p) const { *reinterpret_cast<uint4*>(p) = u; }
  __device__ __forceinline__ void zero() { u = make_uint4(0u, 0u, 0u, 0u); }
  __device__ __forceinline__ void get(float (&x)[8]) const {
    const float2 a = unpack_bf16(u.x), b = unpack_bf16(u.y), c = unpack_bf16(u.z), d = unpack_bf16(u.w);
    x[0] = a.x; x[1] = a.y; x[2] = b.x; x[3] = b.y; x[4] = c.x; x[5] = c.y; x[6] = d.x; x[7] = d.y;
  }
  __device__ __forceinline__ void set(const float (&x)[8]) {
    u = make_uint4(pack_bf16(x[0], x[1]), pack_bf16(x[2], x[3]), pack_bf16(x[4], x[5]), pack_bf16(x[6], x[7]));
  }
};
template <> struct Raw8<float> {
  float4 a, b;
  __device__ __forceinline__ void load(const float* p) { a = reinterpret_cast<const float4*>(p)[0]; b = reinterpret_cast<const float4*>(p)[1]; }
  __device__ __forceinline__ void store(float* p) const { reinterpret_cast<float4*>(p)[0] = a; reinterpret_cast<float4*>(p)[1] = b; }
  __device__ __forceinline__ void zero() { a = b = make_float4(0.f, 0.f, 0.f, 0.f); }
  __device__ __forceinline__ void get(float (&x)[8]) const { x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w; x[4] = b.x; x[5] = b.y; x[6] = b.z; x[7] = b.w; }
  __device__ __forceinline__ void set(const float (&x)[8]) { a = make_float4(x[0], x[1], x[2], x[3]); b = make_float4(x[4], x[5], x[6], x[7]); }
};

// Half a warp per (head, run of `run` ≤ 32 rows); a lane owns NV groups of eight channels of the head.  Rows of a run are
// read once and slide through registers as history of the rows behind them (packed rows: the history of row t is t−1, t−2, …
// as far as its position allows).  STEP: every row is a sequence of its own and takes its history from the pool.  What
// depends on the row only (position, temperature, places in the cache) is worked out once per run, one row per lane.
template <typename T, int TAPS, int NV, bool STEP>
__global__ void __launch_bounds__(128, (NV == 1 && sizeof(T) == 2) ? 4 : 1) conv_heads_kernel(const ConvHeads<T> p, int run) {
  constexpr int H = TAPS - 1, AHEAD = STEP ? 1 : (NV == 1 ? 3 : 2);
  const int lane = threadIdx.x & 31, sub = lane & 15;
  const int heads = p.hq + 2 * p.hkv;
  int head = (blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5)) * 2 + (lane >> 4);
  const bool live = head < heads;
  head = min(head, heads - 1);                       // idle half-warps stay for the shuffles and store nothing
  const bool is_v = head >= p.hq + p.hkv, is_q = head < p.hq;
  const int width = is_v ? p.e : p.d;
  const int c0 = is_v ? (p.hq + p.hkv) * p.d + (head - p.hq - p.hkv) * p.e : head * p.d;   // first column of the head
  const int C = (p.hq + p.hkv) * p.d + p.hkv * p.e;
  const int gh = is_q ? head : (is_v ? head - p.hq - p.hkv : head - p.hq);                  // head inside its own tensor
  const int own_heads = is_q ? p.hq : p.hkv;
  const int t0 = blockIdx.x * run, t1 = min(t0 + run, p.rows);
  // one row per lane
  const int mine = min(t0 + lane, p.rows - 1);
  const int m_pos = static_cast<int>(p.pos[mine]);
  const float m_temp = query_factor(p, m_pos);
  const int m_row = p.pool_row != nullptr ? static_cast<int>(p.pool_row[mine]) : -1;
  int m_hist = -1, m_slot = 0;                       // row of the history pool this row is kept in (< 0: not kept)
  if constexpr (H > 0) {
    if (p.hist != nullptr) {
      m_slot = p.slot[mine];
      if (p.left[mine] < H) m_hist = m_slot * H + m_pos % H;
    }
  }
  bool own[NV];
  float w[NV][TAPS][8];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int el = (i * 16 + sub) * 8;
    own[i] = live && el < width;
    // the taps of eight channels are 8 · TAPS consecutive elements
#pragma unroll
    for (int n = 0; n < TAPS; ++n) {
      float v[8] = {1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f};
      if (own[i] && p.w != nullptr) {
        Raw8<T> r;
        r.load(p.w + static_cast<size_t>(c0 + el) * TAPS + n * 8);
        r.get(v);
      }
#pragma unroll
      for (int c = 0; c < 8; ++c) w[i][(n * 8 + c) % TAPS][(n * 8 + c) / TAPS] = v[c];
    }
  }
  const bool mixes = is_v && p.v_first != nullptr;
  const float lam = mixes ? to_f(p.lam[0]) : 0.f, inv_width = 1.f / width;
  const T* src = p.proj + c0 + sub * 8;              // + t · ld
  T* dst = is_q ? p.q : (is_v ? p.v : p.k);          // + t · own_heads · width (keys of single steps have no copy of their own)
  const size_t off = static_cast<size_t>(gh) * width + sub * 8, pitch = static_cast<size_t>(own_heads) * width;
  T* pool = is_v ? p.v_pool : p.k_pool;
  Raw8<T> h[H > 0 ? H : 1][NV];                      // h[j] = row t − 1 − j, kept as it lies in memory (half the registers)
  if constexpr (!STEP) {
#pragma unroll
    for (int j = 0; j < H; ++j)
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        h[j][i].zero();
        if (own[i] && t0 - 1 - j >= 0) h[j][i].load(src + static_cast<size_t>(t0 - 1 - j) * p.ld + i * 128);
      }
  }
  for (int tb = t0; tb < t1; tb += AHEAD) {
    Raw8<T> cur[AHEAD][NV], first[AHEAD][NV];
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
      const int t = min(tb + u, t1 - 1);
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        cur[u][i].zero();
        first[u][i].zero();
        if (own[i]) {
          cur[u][i].load(src + static_cast<size_t>(t) * p.ld + i * 128);
          if (mixes) first[u][i].load(p.v_first + static_cast<size_t>(t) * pitch + off + i * 128);
        }
      }
    }
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
      const int t = tb + u;
      if (t >= t1) break;
      const int pos = __shfl_sync(0xffffffffu, m_pos, t - t0), row = __shfl_sync(0xffffffffu, m_row, t - t0);
      const float temp = __shfl_sync(0xffffffffu, m_temp, t - t0);
      const int kept = H > 0 ? __shfl_sync(0xffffffffu, m_hist, t - t0) : -1;
      if constexpr (STEP && H > 0) {
        const int slot = __shfl_sync(0xffffffffu, m_slot, t - t0);
#pragma unroll
        for (int j = 0; j < H; ++j)
#pragma unroll
          for (int i = 0; i < NV; ++i) {
            h[j][i].zero();
            if (own[i] && j + 1 <= pos) h[j][i].load(p.hist + (static_cast<size_t>(slot) * H + (pos - 1 - j) % H) * C + c0 + sub * 8 + i * 128);
          }
      }
      float y[NV][8], ss = 0.f;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        float x[8];
        cur[u][i].get(x);
#pragma unroll
        for (int c = 0; c < 8; ++c) y[i][c] = w[i][H][c] * x[c];
#pragma unroll
        for (int j = 0; j < H; ++j) {
          if (j + 1 <= pos) {
            h[j][i].get(x);
#pragma unroll
            for (int c = 0; c < 8; ++c) y[i][c] += w[i][H - 1 - j][c] * x[c];
          }
        }
#pragma unroll
        for (int c = 0; c < 8; ++c) ss += own[i] ? y[i][c] * y[i][c] : 0.f;
      }
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);      // inside the half-warp
      const float f = is_v ? 1.f : rsqrtf(ss * inv_width + p.eps) * (is_q ? temp : 1.f);
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        if (own[i]) {
          if (mixes) {
            float v1[8];
            first[u][i].get(v1);
#pragma unroll
            for (int c = 0; c < 8; ++c) y[i][c] += lam * (v1[c] - y[i][c]);
          } else {
#pragma unroll
            for (int c = 0; c < 8; ++c) y[i][c] *= f;
          }
          Raw8<T> r;
          r.set(y[i]);
          if (dst != nullptr) r.store(dst + static_cast<size_t>(t) * pitch + off + i * 128);
          if (!is_q && row >= 0) r.store(pool + static_cast<size_t>(row) * pitch + off + i * 128);
          // the newest rows of a sequence are what its next step looks back at (the same thread read this place above)
          if (kept >= 0) cur[u][i].store(p.hist + static_cast<size_t>(kept) * C + c0 + sub * 8 + i * 128);
        }
      }
      if constexpr (!STEP && H > 0) {
#pragma unroll
        for (int i = 0; i < NV; ++i) {
#pragma unroll
          for (int j = H - 1; j > 0; --j) h[j][i] = h[j - 1][i];
          h[0][i] = cur[u][i];
        }
      }
    }
  }
}

// Any number of taps, any widths: one block per (row, head), element-wise loads.
template <typename T, bool STEP>
__global__ void __launch_bounds__(128) conv_heads_plain_kernel(const ConvHeads<T> p) {
  extern __shared__ float row_buf[];
  __shared__ float sh[32];
  const int t = blockIdx.x, head = blockIdx.y, H = p.taps > 0 ? p.taps - 1 : 0;
  const bool is_v = head >= p.hq + p.hkv, is_q = head < p.hq;
  const int width = is_v ? p.e : p.d, padded = is_v ? p.ep : p.dp;
  const int c0 = is_v ? (p.hq + p.hkv) * p.d + (head - p.hq - p.hkv) * p.e : head * p.d;
  const int C = (p.hq + p.hkv) * p.d + p.hkv * p.e;
  const int gh = is_q ? head : (is_v ? head - p.hq - p.hkv : head - p.hq);
  const int pos = static_cast<int>(p.pos[t]);
  const int64_t row = p.pool_row != nullptr ? p.pool_row[t] : -1;
  const bool keep = H > 0 && p.hist != nullptr && p.left[t] < H;
  float ss = 0.f;
  for (int el = threadIdx.x; el < width; el += blockDim.x) {
    const int c = c0 + el;
    const T now = p.proj[static_cast<size_t>(t) * p.ld + c];
    float y = to_f(now);
    if (p.w != nullptr) {
      y *= to_f(p.w[static_cast<size_t>(c) * p.taps + H]);
      for (int j = 1; j <= H && j <= pos; ++j) {
        const T b = STEP ? p.hist[(static_cast<size_t>(p.slot[t]) * H + (pos - j) % H) * C + c] : p.proj[static_cast<size_t>(t - j) * p.ld + c];
        y += to_f(p.w[static_cast<size_t>(c) * p.taps + H - j]) * to_f(b);
      }
    }
    if (keep) p.hist[(static_cast<size_t>(p.slot[t]) * H + pos % H) * C + c] = now;
    row_buf[el] = y;
    ss += y * y;
  }
  float f = 1.f;
  if (!is_v) {
    f = rsqrtf(block_sum(ss, sh) / width + p.eps);
    if (is_q) f *= query_factor(p, pos);
  }
  for (int el = threadIdx.x; el < padded; el += blockDim.x) {   // an element is finished by the thread that computed it
    float y = el < width ? row_buf[el] * f : 0.f;
    if (is_q) {
      p.q[(static_cast<size_t>(t) * p.hq + gh) * p.dp + el] = from_f<T>(y);
    } else if (!is_v) {
      if (p.k != nullptr) p.k[(static_cast<size_t>(t) * p.hkv + gh) * p.dp + el] = from_f<T>(y);
      if (row >= 0) p.k_pool[(static_cast<size_t>(row) * p.hkv + gh) * p.dp + el] = from_f<T>(y);
    } else {
      if (p.v_first != nullptr) y += to_f(p.lam[0]) * (to_f(p.v_first[(static_cast<size_t>(t) * p.hkv + gh) * p.ep + el]) - y);
      p.v[(static_cast<size_t>(t) * p.hkv + gh) * p.ep + el] = from_f<T>(y);
      if (row >= 0) p.v_pool[(static_cast<size_t>(row) * p.hkv + gh) * p.ep + el] = from_f<T>(y);
    }
  }
}

static bool aligned16(const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; }

template <typename T, int TAPS>
static void launch_conv_heads(const ConvHeads<T>& p, bool step, bool wide, cudaStream_t stream) {
  const int heads = p.hq + 2 * p.hkv;
  // enough warps to fill the device first, then longer runs (fewer history rows read twice)
  const long target = 16L * num_sms();               // warps; two heads each
  int run = step ? 1 : static_cast<int>(std::min<long>(32, std::max<long>(4, static_cast<long>(p.rows) * heads / 2 / target)));
  const dim3 grid((p.rows + run - 1) / run, (heads + 7) / 8);
  if (step) {
    if (wide) conv_heads_kernel<T, TAPS, 2, true><<<grid, 128, 0, stream>>>(p, run);
    else conv_heads_kernel<T, TAPS, 1, true><<<grid, 128, 0, stream>>>(p, run);
  } else {
    if (wide) conv_heads_kernel<T, TAPS, 2, false><<<grid, 128, 0, stream>>>(p, run);
    else conv_heads_kernel<T, TAPS, 1, false><<<grid, 128, 0, stream>>>(p, run);
  }
}

using OptT = c10::optional<torch::Tensor>;
static bool has(const OptT& t) { return t.has_value() && t->defined(); }

template <typename T>
static void conv_heads_t(ConvHeads<T>& p, bool step) {
  auto stream = at::cuda::getCurrentCUDAStream();
  const int wmax = std::max(p.dp, p.ep);
  const bool vec = p.d % 8 == 0 && p.e % 8 == 0 && p.ld % 8 == 0 && wmax <= 256 && p.taps <= 4 && aligned16(p.proj) && aligned16(p.w);
  if (vec) {
    switch (p.taps) {
      case 4: launch_conv_heads<T, 4>(p, step, wmax > 128, stream); break;
      case 3: launch_conv_heads<T, 3>(p, step, wmax > 128, stream); break;
      case 2: launch_conv_heads<T, 2>(p, step, wmax > 128, stream); break;
      default: launch_conv_heads<T, 1>(p, step, wmax > 128, stream); break;
    }
  } else {
    const dim3 grid(p.rows, p.hq + 2 * p.hkv);
    const size_t smem = static_cast<size_t>(wmax) * sizeof(float);
    TORCH_CHECK(smem <= 48 * 1024, "head width too large");
    if (step) conv_heads_plain_kernel<T, true><<<grid, 128, smem, stream>>>(p);
    else conv_heads_plain_kernel<T, false><<<grid, 128, smem, stream>>>(p);
  }
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
}

std::vector<torch::Tensor> conv_heads(const torch::Tensor& proj, const OptT& weight, const torch::Tensor& pos, int64_t hq, int64_t hkv, int64_t d, int64_t e,
                                      double eps, double coef, int64_t every, const OptT& v_first, const OptT& lam, bool step, const OptT& hist,
                                      const OptT& slot, const OptT& left, const OptT& pool_row, const OptT& k_pool, const OptT& v_pool, bool want_k) {
  const auto st = proj.scalar_type();
  TORCH_CHECK(proj.is_cuda() && proj.dim() == 2 && proj.stride(1) == 1 && (st == torch::kBFloat16 || st == torch::kFloat32), "proj [rows, N] bf16 or fp32");
  const int64_t rows = proj.size(0), C = (hq + hkv) * d + hkv * e, dp = (d + 7) / 8 * 8, ep = (e + 7) / 8 * 8;
  TORCH_CHECK(hq > 0 && hkv > 0 && d > 0 && e > 0 && proj.size(1) >= C, "projection narrower than its q | k | v columns");
  TORCH_CHECK(pos.is_cuda() && pos.scalar_type() == torch::kInt64 && pos.is_contiguous() && pos.numel() == rows, "positions int64 [rows]");
  int taps = 0;
  if (has(weight)) {
    TORCH_CHECK(weight->scalar_type() == st && weight->is_contiguous() && weight->dim() == 2 && weight->size(0) == C && weight->size(1) >= 1, "filters [C, taps]");
    taps = weight->size(1);
  }
  if (has(v_first)) {
    TORCH_CHECK(v_first->scalar_type() == st && v_first->is_contiguous() && v_first->numel() == rows * hkv * ep, "v_first [rows, hkv, ep]");
    TORCH_CHECK(has(lam) && lam->scalar_type() == st && lam->numel() == 1, "mixing weight [1]");
  }
  TORCH_CHECK(!step || taps <= 1 || has(hist), "single steps of a convolution need its history");
  if (has(hist) && taps > 1) {
    TORCH_CHECK(hist->scalar_type() == st && hist->is_contiguous() && hist->dim() == 3 && hist->size(1) == taps - 1 && hist->size(2) == C, "history [slots, taps-1, C]");
    TORCH_CHECK(has(slot) && has(left) && slot->scalar_type() == torch::kInt32 && left->scalar_type() == torch::kInt32 && slot->is_contiguous() &&
                    left->is_contiguous() && slot->numel() == rows && left->numel() == rows, "slot / left int32 [rows]");
  }
  if (has(pool_row)) {
    TORCH_CHECK(has(k_pool) && has(v_pool) && k_pool->scalar_type() == st && v_pool->scalar_type() == st && k_pool->is_contiguous() && v_pool->is_contiguous() &&
                    k_pool->size(-1) == dp && v_pool->size(-1) == ep && k_pool->size(-2) == hkv && v_pool->size(-2) == hkv, "pools [..., hkv, dp] and [..., hkv, ep]");
    TORCH_CHECK(pool_row->scalar_type() == torch::kInt64 && pool_row->is_contiguous() && pool_row->numel() == rows, "pool rows int64 [rows]");
  }
  c10::cuda::CUDAGuard guard(proj.device());
  auto q = torch::empty({rows, hq, dp}, proj.options());
  auto k = want_k ? torch::empty({rows, hkv, dp}, proj.options()) : torch::Tensor();
  auto v = torch::empty({rows, hkv, ep}, proj.options());
  TORCH_CHECK(every >= 0 && every < (int64_t(1) << 31) && (!has(pool_row) || k_pool->numel() / (hkv * dp) < (int64_t(1) << 31)) &&
                  (!has(hist) || hist->size(0) * std::max(taps - 1, 1) < (int64_t(1) << 31)), "32-bit row numbers");
  if (rows > 0) {
    auto fill = [&](auto tag) {
      using T = decltype(tag);
      auto ptr = [](const OptT& t) { return has(t) ? reinterpret_cast<T*>(t->data_ptr()) : static_cast<T*>(nullptr); };
      ConvHeads<T> p{};
      p.proj = reinterpret_cast<const T*>(proj.data_ptr()); p.ld = proj.stride(0); p.w = ptr(weight); p.taps = taps;
      p.hq = hq; p.hkv = hkv; p.d = d; p.e = e; p.dp = dp; p.ep = ep; p.eps = eps; p.coef = coef; p.every = every;
      p.pos = pos.data_ptr<int64_t>();
      p.q = reinterpret_cast<T*>(q.data_ptr()); p.k = want_k ? reinterpret_cast<T*>(k.data_ptr()) : nullptr; p.v = reinterpret_cast<T*>(v.data_ptr());
      p.v_first = ptr(v_first); p.lam = ptr(lam);
      if (has(pool_row)) { p.pool_row = pool_row->data_ptr<int64_t>(); p.k_pool = ptr(k_pool); p.v_pool = ptr(v_pool); }
      if (has(hist) && taps > 1) { p.hist = ptr(hist); p.slot = slot->data_ptr<int>(); p.left = left->data_ptr<int>(); }
      p.rows = rows;
      conv_heads_t<T>(p, step);
    };
    if (st == torch::kBFloat16) fill(bf16{}); else fill(float{});
  }
  if (want_k) return {q, k, v};
  return {q, v};
}

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

// ----------------------------------------------------------------- glu_columns
template <typename T, int V>
__global__ void __launch_bounds__(256) glu_columns_kernel(const T* __restrict__ p, long ld, int gate, int up, T* __restrict__ out, long rows, int I) {
  const int per_row = I / V;
  const long total = rows * per_row;
  for (long i = blockIdx.x * static_cast<long>(blockDim.x) + threadIdx.x; i < total; i += static_cast<long>(gridDim.x) * blockDim.x) {
    const long r = i / per_row;
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
        po[k] = pack_bf16(x.x / (1.f + __expf(-x.x)) * y.x, x.y / (1.f + __expf(-x.y)) * y.y);
      }
      *reinterpret_cast<uint4*>(o) = make_uint4(po[0], po[1], po[2], po[3]);
    } else {
#pragma unroll
      for (int k = 0; k < V; ++k) {
        const float x = to_f(g[k]);
        o[k] = from_f<T>(x / (1.f + __expf(-x)) * to_f(u[k]));
      }
    }
  }
}

torch::Tensor glu_columns(const torch::Tensor& p, int64_t gate, int64_t up, int64_t I) {
  const auto st = p.scalar_type();
  TORCH_CHECK(p.is_cuda() && p.dim() == 2 && p.stride(1) == 1 && (st == torch::kBFloat16 || st == torch::kFloat32), "projection [rows, N] bf16 or fp32");
  TORCH_CHECK(I > 0 && gate >= 0 && up >= 0 && gate + I <= p.size(1) && up + I <= p.size(1), "gate / up columns outside the projection");
  const long rows = p.size(0), ld = p.stride(0);
  c10::cuda::CUDAGuard guard(p.device());
  auto out = torch::empty({rows, I}, p.options());
  if (rows == 0) return out;
  auto stream = at::cuda::getCurrentCUDAStream();
  const bool vec = st == torch::kBFloat16 && I % 8 == 0 && gate % 8 == 0 && up % 8 == 0 && ld % 8 == 0 && aligned16(p.data_ptr());
  const long total = rows * (vec ? I / 8 : I);
  const int blocks = static_cast<int>(std::min<long>((total + 255) / 256, num_sms() * 16L));
  if (st == torch::kBFloat16) {
    const bf16* in = reinterpret_cast<const bf16*>(p.data_ptr());
    bf16* o = reinterpret_cast<bf16*>(out.data_ptr());
    if (vec) glu_columns_kernel<bf16, 8><<<blocks, 256, 0, stream>>>(in, ld, gate, up, o, rows, I);
    else glu_columns_kernel<bf16, 1><<<blocks, 256, 0, stream>>>(in, ld, gate, up, o, rows, I);
  } else {
    glu_columns_kernel<float, 1><<<blocks, 256, 0, stream>>>(p.data_ptr<float>(), ld, gate, up, out.data_ptr<float>(), rows, I);
  }
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return out;
}

}  // namespace tk
