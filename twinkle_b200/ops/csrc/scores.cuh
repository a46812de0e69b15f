// What may happen to an attention score beyond its scale, shared by the attention kernels: a factor per head, cap · tanh(s / cap), and a
// number for the distance between query and key.
#pragma once
#include <c10/util/Optional.h>
#include <torch/types.h>

#include "common.cuh"

namespace tk {

struct ScoreTerms {
  float cap, inv_cap;             // 0: not capped
  const void *temp;               // [H] (null: 1)
  const void *slope, *rate;       // [H]: −slope ln(1 + rate · n)
  const void *table;              // [rows, H]: table[bucket[min(n, far)]]
  const int* bucket;
  int far, heads;
  bool used;                      // any of them
};

inline ScoreTerms score_terms(double cap, const c10::optional<torch::Tensor>& temp, const c10::optional<torch::Tensor>& slope, const c10::optional<torch::Tensor>& rate,
                              const c10::optional<torch::Tensor>& table, const c10::optional<torch::Tensor>& bucket, int64_t heads, torch::ScalarType st) {
  ScoreTerms s{};
  TORCH_CHECK(cap >= 0, "score cap: 0 (none) or positive");
  s.cap = static_cast<float>(cap);
  s.inv_cap = cap > 0 ? static_cast<float>(1.0 / cap) : 0.f;
  s.heads = static_cast<int>(heads);
  auto per_head = [&](const c10::optional<torch::Tensor>& t) -> const void* {
    if (!t.has_value() || !t->defined()) return nullptr;
    TORCH_CHECK(t->is_cuda() && t->scalar_type() == st && t->is_contiguous() && t->numel() == heads, "score terms: a number per query head in the queries' dtype");
    return t->data_ptr();
  };
  s.temp = per_head(temp);
  s.slope = per_head(slope);
  s.rate = per_head(rate);
  TORCH_CHECK((s.slope == nullptr) == (s.rate == nullptr), "slope and rate go together");
  if (table.has_value() && table->defined()) {
    TORCH_CHECK(bucket.has_value() && bucket->is_cuda() && bucket->scalar_type() == torch::kInt32 && bucket->is_contiguous() && bucket->numel() > 0, "buckets int32 [distances]");
    TORCH_CHECK(table->is_cuda() && table->scalar_type() == st && table->is_contiguous() && table->dim() == 2 && table->size(1) == heads, "distance table [rows, heads]");
    s.table = table->data_ptr();
    s.bucket = bucket->data_ptr<int>();
    s.far = static_cast<int>(bucket->numel()) - 1;
  }
  s.used = s.cap > 0 || s.temp != nullptr || s.slope != nullptr || s.table != nullptr;
  return s;
}

__device__ __forceinline__ float score_ld(const float* p) { return *p; }
__device__ __forceinline__ float score_ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }

// tanh(u) for |u| ≤ kTanhNear: u times a polynomial in u² through the Chebyshev nodes of [0, kTanhNear²]; relative error 3e-9.
constexpr float kTanhNear = 0.6f;
__device__ __forceinline__ float tanh_near(float u) {
  const float v = u * u;
  float r = fmaf(v, -0.00584964390839844f, 0.02075134910436602f);
  r = fmaf(v, r, -0.053767983507834786f);
  r = fmaf(v, r, 0.13331679634553723f);
  r = fmaf(v, r, -0.33333282834325195f);
  r = fmaf(v, r, 0.999999997480156f);
  return u * r;
}
// tanh(u) for |u| not small: 1 − 2 / (1 + e^{2|u|}) with the sign of u
__device__ __forceinline__ float tanh_far(float u) {
  const float e = fast_exp2(fabsf(u) * 2.885390081777927f);
  return copysignf(1.f - __fdividef(2.f, 1.f + e), u);
}
__device__ __forceinline__ float tanh_any(float u) { return fabsf(u) <= kTanhNear ? tanh_near(u) : tanh_far(u); }

// The number of one head for a distance n ≥ 0.
template <typename T>
struct DistanceNumber {
  float slope, rate;
  const T* table;                 // this head's column
  const int* bucket;
  int far, heads;
  __device__ __forceinline__ DistanceNumber(const ScoreTerms& s, int head) : slope(0.f), rate(0.f), table(nullptr), bucket(s.bucket), far(s.far), heads(s.heads) {
    if (s.slope != nullptr) {
      slope = score_ld(reinterpret_cast<const T*>(s.slope) + head);
      rate = score_ld(reinterpret_cast<const T*>(s.rate) + head);
    }
    if (s.table != nullptr) table = reinterpret_cast<const T*>(s.table) + head;
  }
  __device__ __forceinline__ float at(int n) const {
    float y = -slope * __logf(fmaf(rate, static_cast<float>(n), 1.f));
    if (table != nullptr) y += score_ld(table + static_cast<size_t>(bucket[min(n, far)]) * heads);
    return y;
  }
};

template <typename T>
__device__ __forceinline__ float score_temp(const ScoreTerms& s, int head) {
  return s.temp != nullptr ? score_ld(reinterpret_cast<const T*>(s.temp) + head) : 1.f;
}

// Sigmoid gates on the output: one per head (e = 0) or one per element of a head (e = their number); null: none.
struct OutGate {
  const void* p;
  long ld;
  int e;
};
inline OutGate out_gate(const c10::optional<torch::Tensor>& gate, int64_t rows, int64_t heads, int64_t row_width, torch::ScalarType st) {
  OutGate g{};
  if (!gate.has_value() || !gate->defined()) return g;
  TORCH_CHECK(gate->is_cuda() && gate->scalar_type() == st && gate->dim() == 2 && gate->size(0) == rows && gate->stride(1) == 1 && gate->size(1) % heads == 0, "gate [T, Hq] or [T, Hq * e]");
  const int64_t e = gate->size(1) / heads;
  TORCH_CHECK(gate->size(1) == heads || e <= row_width, "gates wider than the output's heads");
  g.p = gate->data_ptr();
  g.ld = gate->stride(0);
  g.e = gate->size(1) == heads ? 0 : static_cast<int>(e);
  return g;
}
__device__ __forceinline__ float sigmoid_of(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }

}  // namespace tk
