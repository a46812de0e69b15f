// Heads that do not rotate: [q | k | v] columns of a fused projection (or [q | k], when the values are the projected keys) to queries, keys
// and values, with bias, RMS norm of q and k per head or over all heads together, values over their root mean square, and the writes into
// the paged K/V pools — one pass.  Templated on the compute dtype (bf16 or fp32); a vector kernel where rows are made of whole vectors, a
// plain one otherwise.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/types.h>

#include "common.cuh"
#include "host.h"
#include "vec.cuh"

namespace tk {

template <typename T>
struct PlainHeads {
  const T* proj; long ld;                        // q | k | v from here on
  const T *bias, *qw, *kw;                       // (null: none)
  bool whole, value_norm, shared;                // norms over all heads; values normed; values are the projected keys
  int hq, hkv, d, e, dp, ep;                     // heads, widths, and row widths of outputs and pools (the rest is written as zero)
  float eps;
  T *q, *k, *v;                                  // k and v may be null
  T *k_pool, *v_pool; const int64_t* pool_row;   // (null: not kept)
};

// One block per row.  LANES threads per head, eight elements each; the sums of norms over all heads take a pass of their own over the row,
// which stays in the first-level cache for the second.
template <typename T, int LANES>
__global__ void __launch_bounds__(256) plain_heads_kernel(const PlainHeads<T> p) {
  constexpr int GROUPS = 256 / LANES;
  __shared__ float sh[32], sh2[32];
  const int t = blockIdx.x, sub = threadIdx.x % LANES, el = sub * 8, nq = p.hq * p.d, nk = p.hkv * p.d;
  const int heads = p.hq + p.hkv + (p.shared ? 0 : p.hkv);
  const T* row = p.proj + static_cast<size_t>(t) * p.ld;
  const int64_t kept = p.pool_row != nullptr ? p.pool_row[t] : -1;
  auto element8 = [&](int c, float (&y)[8]) {
    Raw8<T> r;
    r.load(row + c);
    r.get(y);
    if (p.bias != nullptr) {
      float b[8];
      r.load(p.bias + c);
      r.get(b);
#pragma unroll
      for (int i = 0; i < 8; ++i) y[i] += b[i];
    }
  };
  float all_q = 0.f, all_k = 0.f;
  if (p.whole) {
    for (int c = threadIdx.x * 8; c < nq + nk; c += 2048) {
      float y[8], ss = 0.f;
      element8(c, y);
#pragma unroll
      for (int i = 0; i < 8; ++i) ss += y[i] * y[i];
      if (c < nq) all_q += ss; else all_k += ss;
    }
    all_q = rsqrtf(block_sum(all_q, sh) / nq + p.eps);
    all_k = rsqrtf(block_sum(all_k, sh2) / nk + p.eps);
  }
  for (int h0 = 0; h0 < heads; h0 += GROUPS) {     // the same number of rounds for the whole block
    const int head = h0 + threadIdx.x / LANES;
    const bool is_q = head < p.hq, is_v = head >= p.hq + p.hkv;
    const int width = is_v ? p.e : p.d, g = is_q ? head : (is_v ? head - p.hq - p.hkv : head - p.hq);
    const bool own = head < heads && el < width;
    float y[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f}, ss = 0.f;
    if (own) element8(is_v ? nq + nk + g * p.e + el : head * p.d + el, y);
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += y[i] * y[i];
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!own) continue;                            // no barrier or shuffle follows for this round's heads
    const float per_head = rsqrtf(ss / width + p.eps);
    Raw8<T> r;
    auto put_value = [&](float (&v)[8]) {
      if (p.value_norm) {
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] *= per_head;
      }
      r.set(v);
      if (p.v != nullptr) r.store(p.v + (static_cast<size_t>(t) * p.hkv + g) * p.e + el);
      if (kept >= 0) r.store(p.v_pool + (static_cast<size_t>(kept) * p.hkv + g) * p.e + el);
    };
    if (is_v) {
      put_value(y);
      continue;
    }
    if (!is_q && p.shared) {
      float v[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) v[i] = y[i];
      put_value(v);
    }
    const T* w = is_q ? p.qw : p.kw;
    if (w != nullptr) {
      const float f = !p.whole ? per_head : (is_q ? all_q : all_k);
      float s[8];
      r.load(w + (p.whole ? g * p.d : 0) + el);
      r.get(s);
#pragma unroll
      for (int i = 0; i < 8; ++i) y[i] *= f * s[i];
    }
    r.set(y);
    if (is_q) {
      r.store(p.q + (static_cast<size_t>(t) * p.hq + g) * p.d + el);
    } else {
      if (p.k != nullptr) r.store(p.k + (static_cast<size_t>(t) * p.hkv + g) * p.d + el);
      if (kept >= 0) r.store(p.k_pool + (static_cast<size_t>(kept) * p.hkv + g) * p.d + el);
    }
  }
}

// Any widths: one block per row, a warp per head, element-wise.
template <typename T>
__global__ void __launch_bounds__(256) plain_heads_any_kernel(const PlainHeads<T> p) {
  __shared__ float sh[32], sh2[32];
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nq = p.hq * p.d, nk = p.hkv * p.d;
  const T* row = p.proj + static_cast<size_t>(t) * p.ld;
  const int64_t kept = p.pool_row != nullptr ? p.pool_row[t] : -1;
  auto at = [&](int c) { return to_f(row[c]) + (p.bias != nullptr ? to_f(p.bias[c]) : 0.f); };
  float all_q = 0.f, all_k = 0.f;
  if (p.whole) {
    for (int c = threadIdx.x; c < nq + nk; c += 256) {
      const float y = at(c);
      if (c < nq) all_q += y * y; else all_k += y * y;
    }
    all_q = rsqrtf(block_sum(all_q, sh) / nq + p.eps);
    all_k = rsqrtf(block_sum(all_k, sh2) / nk + p.eps);
  }
  for (int head = warp; head < p.hq + 2 * p.hkv; head += 8) {
    const bool is_q = head < p.hq, is_v = head >= p.hq + p.hkv;
    const int width = is_v ? p.e : p.d, padded = is_v ? p.ep : p.dp, g = is_q ? head : (is_v ? head - p.hq - p.hkv : head - p.hq);
    const int c0 = is_q ? g * p.d : (is_v && !p.shared ? nq + nk + g * p.e : nq + g * p.d);
    const T* w = is_v ? nullptr : (is_q ? p.qw : p.kw);
    float f = 1.f;
    if (w != nullptr && p.whole) {
      f = is_q ? all_q : all_k;
    } else if (w != nullptr || (is_v && p.value_norm)) {
      float ss = 0.f;
      for (int i = lane; i < width; i += 32) ss += at(c0 + i) * at(c0 + i);
      f = rsqrtf(warp_sum(ss) / width + p.eps);
    }
    T *out = is_q ? p.q : (is_v ? p.v : p.k), *pool = is_q ? nullptr : (is_v ? p.v_pool : p.k_pool);
    const int own = is_q ? p.hq : p.hkv;
    for (int i = lane; i < padded; i += 32) {
      const T y = from_f<T>(i < width ? at(c0 + i) * f * (w != nullptr ? to_f(w[(p.whole ? g * p.d : 0) + i]) : 1.f) : 0.f);
      if (out != nullptr) out[(static_cast<size_t>(t) * own + g) * padded + i] = y;
      if (pool != nullptr && kept >= 0) pool[(static_cast<size_t>(kept) * own + g) * padded + i] = y;
    }
  }
}

// proj [rows, N].  qw / kw: [d] (per head) or [heads · d] (over all heads).  Returns {q} or, with want_kv, {q, k, v}.
std::vector<torch::Tensor> plain_heads(const torch::Tensor& proj, int64_t first, const OptT& bias, const OptT& qw, const OptT& kw, bool value_norm, bool shared, int64_t hq,
                                       int64_t hkv, int64_t d, int64_t e, double eps, const OptT& k_pool, const OptT& v_pool, const OptT& pool_row, bool want_kv) {
  const auto st = proj.scalar_type();
  TORCH_CHECK(proj.is_cuda() && proj.dim() == 2 && proj.stride(1) == 1 && (st == torch::kBFloat16 || st == torch::kFloat32), "proj [rows, N] bf16 or fp32");
  const int64_t rows = proj.size(0), C = (hq + hkv) * d + (shared ? 0 : hkv * e), dp = (d + 7) / 8 * 8, ep = (e + 7) / 8 * 8;
  TORCH_CHECK(hq > 0 && hkv > 0 && d > 0 && e > 0 && first >= 0 && proj.size(1) >= first + C, "projection narrower than its q | k | v columns");
  TORCH_CHECK(!shared || d == e, "values that are the keys are as wide");
  auto vector = [&](const OptT& t, int64_t len) { return t->is_cuda() && t->scalar_type() == st && t->is_contiguous() && t->numel() == len; };
  TORCH_CHECK(!has(bias) || vector(bias, C), "bias [q | k | v columns] in the projection's dtype");
  TORCH_CHECK(has(qw) == has(kw), "norm weights of q and k go together");
  // with one head each, both kinds of norm are the same
  const bool whole = has(qw) && !(vector(qw, d) && vector(kw, d));
  TORCH_CHECK(!whole || (vector(qw, hq * d) && vector(kw, hkv * d)), "norm weights [d] or [heads * d] in the projection's dtype");
  if (has(pool_row)) {
    TORCH_CHECK(has(k_pool) && has(v_pool) && k_pool->scalar_type() == st && v_pool->scalar_type() == st && k_pool->is_contiguous() && v_pool->is_contiguous() &&
                    k_pool->size(-1) == dp && v_pool->size(-1) == ep && k_pool->size(-2) == hkv && v_pool->size(-2) == hkv, "pools [..., hkv, dp] and [..., hkv, ep]");
    TORCH_CHECK(pool_row->scalar_type() == torch::kInt64 && pool_row->is_contiguous() && pool_row->numel() == rows, "pool rows int64 [rows]");
  }
  c10::cuda::CUDAGuard guard(proj.device());
  std::vector<torch::Tensor> out{torch::empty({rows, hq, dp}, proj.options())};
  if (want_kv) {
    out.push_back(torch::empty({rows, hkv, dp}, proj.options()));
    out.push_back(torch::empty({rows, hkv, ep}, proj.options()));
  }
  if (rows == 0) return out;
  auto stream = at::cuda::getCurrentCUDAStream();
  auto run = [&](auto tag) {
    using T = decltype(tag);
    auto ptr = [](const OptT& t) { return has(t) ? reinterpret_cast<T*>(t->data_ptr()) : static_cast<T*>(nullptr); };
    PlainHeads<T> p{};
    p.proj = reinterpret_cast<const T*>(proj.data_ptr()) + first; p.ld = proj.stride(0); p.bias = ptr(bias); p.qw = ptr(qw); p.kw = ptr(kw);
    p.whole = whole; p.value_norm = value_norm; p.shared = shared;
    p.hq = hq; p.hkv = hkv; p.d = d; p.e = e; p.dp = dp; p.ep = ep; p.eps = eps;
    p.q = reinterpret_cast<T*>(out[0].data_ptr());
    if (want_kv) { p.k = reinterpret_cast<T*>(out[1].data_ptr()); p.v = reinterpret_cast<T*>(out[2].data_ptr()); }
    if (has(pool_row)) { p.pool_row = pool_row->data_ptr<int64_t>(); p.k_pool = ptr(k_pool); p.v_pool = ptr(v_pool); }
    const int widest = std::max(d, e);
    const bool vec = d % 8 == 0 && e % 8 == 0 && p.ld % 8 == 0 && widest <= 256 && aligned16(p.proj) && aligned16(p.bias) && aligned16(p.qw) && aligned16(p.kw);
    if (!vec) plain_heads_any_kernel<T><<<rows, 256, 0, stream>>>(p);
    else if (widest <= 64) plain_heads_kernel<T, 8><<<rows, 256, 0, stream>>>(p);
    else if (widest <= 128) plain_heads_kernel<T, 16><<<rows, 256, 0, stream>>>(p);
    else plain_heads_kernel<T, 32><<<rows, 256, 0, stream>>>(p);
  };
  if (st == torch::kBFloat16) run(bf16{}); else run(float{});
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return out;
}

}  // namespace tk
