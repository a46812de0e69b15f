// conv_heads: short causal convolution on q, k and v, q / k over their root mean square per head, query temperature, value mixing,
// and the writes into the paged K/V pools and the convolution history — one pass over the leading [q | k | v] columns of a fused
// projection.  Templated on the compute dtype (bf16 or fp32); a vector kernel where rows are made of whole vectors, a plain one
// otherwise.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/types.h>

#include "common.cuh"
#include "host.h"
#include "vec.cuh"

namespace tk {

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

}  // namespace tk
