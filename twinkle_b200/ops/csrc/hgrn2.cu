// HGRN2 linear attention between its projections.  Per head, with state S ∈ R^{dim × vdim} in fp32:
//
//   q = silu(q_raw),  k = (1 − lower) σ(−(f_raw + bias)) = 1 − forget gate,  S ← S + k ⊙ (v − S)  (rows by k),  o = Sᵀ q,
//   output = o / rms(o) · weight                                        (rms over the head's vdim)
//
// Forming k instead of the forget gate keeps the digits of gates close to one, and the update above needs no decay beside it.
//
//   hgrn2_prefill  packed prompts.  A block owns one head of one sequence (or of one time segment of it) and keeps the state in
//                  registers: RS neighbouring lanes share two columns, each with RPT of the rows, so a token costs three
//                  operations per state element, two 16-byte shared-memory broadcasts per twelve of them and a shuffle per column.
//                  Sixteen tokens at a time are brought in by asynchronous copies while the sixteen before are worked on.
//                  When sequences × heads do not fill the device, sequences are cut into time segments: a first pass forms each
//                  segment's own contribution and decay, a scan over segments gives every segment its starting state.
//   hgrn2_step     one token of every sequence: the state passes once through the block, 16 bytes per access.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/types.h>

#include "common.cuh"
#include "host.h"

namespace tk {

using bf16 = __nv_bfloat16;
using OptT = c10::optional<torch::Tensor>;

namespace hg {
constexpr int CH = 16;          // tokens per round

__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(bf16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float silu(float z) { return z / (1.f + __expf(-z)); }
__device__ __forceinline__ float let_in(float z, float low) { return (1.f - low) / (1.f + __expf(z)); }

// asynchronous copy of 16 bytes into shared memory
__device__ __forceinline__ void copy16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void copies_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void copies_wait() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }
}  // namespace hg

template <typename T>
struct Hgrn2 {
  const T *q, *f, *v;              // column ranges of the projection, row stride ld
  long ld;
  const T *bias, *lower, *weight;  // [H·dim], [H·dim], [vdim]
  T* o;                            // [rows, H·vdim]
  float* raw;                      // [rows, H·vdim]: outputs before their norm, when a block does not hold a whole head
  const int* cu;                   // [n+1]
  float* pool;                     // [slots, H, dim, vdim] (null: last states are not kept)
  const int* slot;                 // [rows]
  float *part, *decay;             // [n, segments − 1, H, dim, vdim], [n, segments − 1, H, dim]
  int H, dim, vdim, seg_len, segments, slices, cols;
  float eps;
};

// PART: only the state a segment builds up from nothing and its decay; otherwise outputs.
template <typename T, int RPT, int RS, bool VEC, bool PART>
__global__ void __launch_bounds__(256) hgrn2_prefill_kernel(const Hgrn2<T> p) {
  using namespace hg;
  extern __shared__ __align__(16) uint8_t sm_raw[];
  constexpr int DP = RPT * RS;
  const int head = blockIdx.x / p.slices, slice = blockIdx.x - head * p.slices, seg = blockIdx.y, seq = blockIdx.z;
  const int s0 = p.cu[seq], len = p.cu[seq + 1] - s0;
  const int a = seg * p.seg_len, b = min(len, a + p.seg_len);
  if (a >= len || (PART && b >= len)) return;         // the last segment of a sequence is nobody's past
  const int col0 = slice * p.cols, ncol = min(p.cols, p.vdim - col0);
  const int VP = p.cols;
  float* s_q = reinterpret_cast<float*>(sm_raw);      // [CH][DP]
  float* s_k = s_q + CH * DP;                         // [CH][DP]
  float* s_v = s_k + CH * DP;                         // [CH][VP]: values, then outputs
  float* s_low = s_v + CH * VP;                       // [DP] lower bound, [DP] bias
  float* s_bias = s_low + DP;
  T* r_q = reinterpret_cast<T*>(s_bias + DP);         // the next tokens as they lie in memory: [CH][dim], [CH][dim], [CH][ncol]
  T* r_f = r_q + CH * p.dim;
  T* r_v = r_f + CH * p.dim;
  const int tid = threadIdx.x, rs = tid % RS, c0 = tid / RS * 2;
  const bool mine = c0 < ncol, two = c0 + 1 < ncol;
  for (int i = tid; i < DP; i += blockDim.x) {
    s_low[i] = i < p.dim ? ld(p.lower + static_cast<size_t>(head) * p.dim + i) : 1.f;
    s_bias[i] = i < p.dim ? ld(p.bias + static_cast<size_t>(head) * p.dim + i) : 0.f;
  }
  for (int i = tid; i < CH * DP; i += blockDim.x) {   // rows that fill up the head's width stay zero
    s_q[i] = 0.f;
    s_k[i] = 0.f;
  }
  const T* gq = p.q + static_cast<size_t>(s0) * p.ld + static_cast<size_t>(head) * p.dim;
  const T* gf = p.f + static_cast<size_t>(s0) * p.ld + static_cast<size_t>(head) * p.dim;
  const T* gv = p.v + static_cast<size_t>(s0) * p.ld + static_cast<size_t>(head) * p.vdim + col0;
  auto fetch = [&](int t0) {
    if constexpr (VEC) {
      constexpr int E = 16 / sizeof(T);
      const int n = min(CH, b - t0), dv = p.dim / E, vv = ncol / E;
      for (int i = tid; i < n * dv; i += blockDim.x) {
        const int t = i / dv, c = (i - t * dv) * E;
        const size_t g = static_cast<size_t>(t0 + t) * p.ld + c;
        if constexpr (!PART) copy16(r_q + t * p.dim + c, gq + g);
        copy16(r_f + t * p.dim + c, gf + g);
      }
      for (int i = tid; i < n * vv; i += blockDim.x) {
        const int t = i / vv, c = (i - t * vv) * E;
        copy16(r_v + t * ncol + c, gv + static_cast<size_t>(t0 + t) * p.ld + c);
      }
      copies_commit();
    }
  };
  float S0[RPT], S1[RPT];
  const size_t head_state = static_cast<size_t>(p.dim) * p.vdim;
  // row of register i: RS lanes take turns in groups of four
  auto row_of = [&](int i) { return ((i >> 2) * RS + rs) * 4 + (i & 3); };
  {
    const float* init = (!PART && seg > 0) ? p.part + ((static_cast<size_t>(seq) * (p.segments - 1) + seg - 1) * p.H + head) * head_state + col0 : nullptr;
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int r = row_of(i);
      S0[i] = init != nullptr && mine && r < p.dim ? init[static_cast<size_t>(r) * p.vdim + c0] : 0.f;
      S1[i] = init != nullptr && two && r < p.dim ? init[static_cast<size_t>(r) * p.vdim + c0 + 1] : 0.f;
    }
  }
  float keep[(DP + 31) / 32];                         // PART: decay of the rows this thread follows (blocks have at least 32 threads)
  if constexpr (PART) {
#pragma unroll
    for (int i = 0; i < (DP + 31) / 32; ++i) keep[i] = 1.f;
  }
  fetch(a);
  for (int t0 = a; t0 < b; t0 += CH) {
    const int n = min(CH, b - t0);
    if constexpr (VEC) copies_wait();
    __syncthreads();
    for (int i = tid; i < n * p.dim; i += blockDim.x) {
      const int t = i / p.dim, c = i - t * p.dim;
      const size_t g = static_cast<size_t>(t0 + t) * p.ld + c;
      if constexpr (!PART) s_q[t * DP + c] = silu(ld(VEC ? r_q + i : gq + g));
      s_k[t * DP + c] = let_in(ld(VEC ? r_f + i : gf + g) + s_bias[c], s_low[c]);
    }
    for (int i = tid; i < n * ncol; i += blockDim.x) {
      const int t = i / ncol, c = i - t * ncol;
      s_v[t * VP + c] = ld(VEC ? r_v + i : gv + static_cast<size_t>(t0 + t) * p.ld + c);
    }
    __syncthreads();
    if (t0 + CH < b) fetch(t0 + CH);
    for (int t = 0; t < n; ++t) {
      const float v0 = mine ? s_v[t * VP + c0] : 0.f, v1 = two ? s_v[t * VP + c0 + 1] : 0.f;
      float o0 = 0.f, o1 = 0.f, u0 = 0.f, u1 = 0.f;
#pragma unroll
      for (int i = 0; i < RPT; i += 4) {
        const float4 kk = *reinterpret_cast<const float4*>(s_k + t * DP + ((i >> 2) * RS + rs) * 4);
        S0[i] = fmaf(kk.x, v0 - S0[i], S0[i]);
        S1[i] = fmaf(kk.x, v1 - S1[i], S1[i]);
        S0[i + 1] = fmaf(kk.y, v0 - S0[i + 1], S0[i + 1]);
        S1[i + 1] = fmaf(kk.y, v1 - S1[i + 1], S1[i + 1]);
        S0[i + 2] = fmaf(kk.z, v0 - S0[i + 2], S0[i + 2]);
        S1[i + 2] = fmaf(kk.z, v1 - S1[i + 2], S1[i + 2]);
        S0[i + 3] = fmaf(kk.w, v0 - S0[i + 3], S0[i + 3]);
        S1[i + 3] = fmaf(kk.w, v1 - S1[i + 3], S1[i + 3]);
        if constexpr (!PART) {
          const float4 qq = *reinterpret_cast<const float4*>(s_q + t * DP + ((i >> 2) * RS + rs) * 4);
          o0 = fmaf(qq.x, S0[i], o0); o1 = fmaf(qq.x, S1[i], o1);
          u0 = fmaf(qq.y, S0[i + 1], u0); u1 = fmaf(qq.y, S1[i + 1], u1);
          o0 = fmaf(qq.z, S0[i + 2], o0); o1 = fmaf(qq.z, S1[i + 2], o1);
          u0 = fmaf(qq.w, S0[i + 3], u0); u1 = fmaf(qq.w, S1[i + 3], u1);
        }
      }
      if constexpr (!PART) {
        o0 += u0;
        o1 += u1;
#pragma unroll
        for (int o = 1; o < RS; o <<= 1) {
          o0 += __shfl_xor_sync(0xffffffffu, o0, o);
          o1 += __shfl_xor_sync(0xffffffffu, o1, o);
        }
        // every lane that shares the columns has read its values by now: outputs take their place
        if (rs == 0 && mine) s_v[t * VP + c0] = o0;
        if (rs == RS - 1 && two) s_v[t * VP + c0 + 1] = o1;
      }
    }
    if constexpr (PART) {
#pragma unroll
      for (int i = 0; i < (DP + 31) / 32; ++i) {
        const int r = i * blockDim.x + tid;
        if (r < p.dim)
          for (int t = 0; t < n; ++t) keep[i] *= 1.f - s_k[t * DP + r];
      }
    } else {
      __syncthreads();
      const int warp = tid >> 5, lane = tid & 31;
      for (int t = warp; t < n; t += blockDim.x >> 5) {
        const size_t at = static_cast<size_t>(s0 + t0 + t) * p.H * p.vdim + static_cast<size_t>(head) * p.vdim + col0;
        if (p.raw != nullptr) {
          for (int c = lane; c < ncol; c += 32) p.raw[at + c] = s_v[t * VP + c];
          continue;
        }
        float ss = 0.f;
        for (int c = lane; c < ncol; c += 32) ss += s_v[t * VP + c] * s_v[t * VP + c];
        const float r = rsqrtf(warp_sum(ss) / p.vdim + p.eps);
        for (int c = lane; c < ncol; c += 32) st(p.o + at + c, s_v[t * VP + c] * r * ld(p.weight + c));
      }
    }
  }
  float* out = nullptr;
  if constexpr (PART) {
    out = p.part + ((static_cast<size_t>(seq) * (p.segments - 1) + seg) * p.H + head) * head_state + col0;
    if (slice == 0) {
      float* d = p.decay + ((static_cast<size_t>(seq) * (p.segments - 1) + seg) * p.H + head) * p.dim;
#pragma unroll
      for (int i = 0; i < (DP + 31) / 32; ++i) {
        const int r = i * blockDim.x + tid;
        if (r < p.dim) d[r] = keep[i];
      }
    }
  } else if (p.pool != nullptr && b == len) {
    const int sl = p.slot[s0];
    if (sl > 0) out = p.pool + (static_cast<size_t>(sl) * p.H + head) * head_state + col0;
  }
  if (out != nullptr) {
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int r = row_of(i);
      if (r < p.dim) {
        if (mine) out[static_cast<size_t>(r) * p.vdim + c0] = S0[i];
        if (two) out[static_cast<size_t>(r) * p.vdim + c0 + 1] = S1[i];
      }
    }
  }
}

// part[s] becomes the state behind segment s: a scan over the segments of every sequence, one thread per state element.
__global__ void __launch_bounds__(256) hgrn2_scan_kernel(float* part, const float* __restrict__ decay, const int* __restrict__ cu, int H, int dim, int vdim,
                                                         int seg_len, int segments) {
  const int seq = blockIdx.y, len = cu[seq + 1] - cu[seq];
  const long per = static_cast<long>(H) * dim * vdim, i = blockIdx.x * 256L + threadIdx.x;
  if (i >= per) return;
  float S = 0.f;
  for (int s = 0; s < segments - 1 && (s + 1) * seg_len < len; ++s) {
    const size_t at = (static_cast<size_t>(seq) * (segments - 1) + s) * per + i;
    S = fmaf(decay[(static_cast<size_t>(seq) * (segments - 1) + s) * H * dim + i / vdim], S, part[at]);
    part[at] = S;
  }
}

// Norm of heads whose columns were split over blocks: one warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(256) hgrn2_norm_kernel(const float* __restrict__ raw, const T* __restrict__ weight, T* __restrict__ o, long heads, int vdim, float eps) {
  const long i = blockIdx.x * 8L + (threadIdx.x >> 5);
  if (i >= heads) return;
  const int lane = threadIdx.x & 31;
  float ss = 0.f;
  for (int c = lane; c < vdim; c += 32) ss += raw[i * vdim + c] * raw[i * vdim + c];
  const float r = rsqrtf(warp_sum(ss) / vdim + eps);
  for (int c = lane; c < vdim; c += 32) hg::st(o + i * vdim + c, raw[i * vdim + c] * r * hg::ld(weight + c));
}

// One token per sequence: block = (head, sequence), V consecutive columns per access.  Slot 0: a row that fills up a batch.
template <typename T, int V>
__global__ void __launch_bounds__(256) hgrn2_step_kernel(const Hgrn2<T> p) {
  using namespace hg;
  extern __shared__ __align__(16) float sm_step[];
  __shared__ float s_part[8];
  const int head = blockIdx.x, row = blockIdx.y, tid = threadIdx.x, dim = p.dim, vdim = p.vdim;
  T* o = p.o + static_cast<size_t>(row) * p.H * vdim + static_cast<size_t>(head) * vdim;
  const int slot = p.slot[row];
  if (slot <= 0) {
    for (int c = tid; c < vdim; c += 256) st(o + c, 0.f);
    return;
  }
  float *s_q = sm_step, *s_k = s_q + dim, *s_v = s_k + dim, *s_o = s_v + (vdim + 3) / 4 * 4;
  const size_t g = static_cast<size_t>(row) * p.ld, hd = static_cast<size_t>(head) * dim;
  for (int c = tid; c < dim; c += 256) {
    s_q[c] = silu(ld(p.q + g + hd + c));
    s_k[c] = let_in(ld(p.f + g + hd + c) + ld(p.bias + hd + c), ld(p.lower + hd + c));
  }
  for (int c = tid; c < vdim; c += 256) s_v[c] = ld(p.v + g + static_cast<size_t>(head) * vdim + c);
  const int cg = vdim / V, rg = 256 / cg, c = tid % cg * V, r0 = tid / cg;
  float* S = p.pool + (static_cast<size_t>(slot) * p.H + head) * dim * vdim + c;
  float acc[V];
#pragma unroll
  for (int i = 0; i < V; ++i) acc[i] = 0.f;
  __syncthreads();
  if (r0 < rg) {
    constexpr int U = 8;
    for (int rb = r0; rb < dim; rb += rg * U) {
      float x[U][V];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int r = rb + u * rg;
        if (r < dim) {
          if constexpr (V == 4) {
            const float4 w = *reinterpret_cast<const float4*>(S + static_cast<size_t>(r) * vdim);
            x[u][0] = w.x; x[u][1] = w.y; x[u][2] = w.z; x[u][3] = w.w;
          } else {
            x[u][0] = S[static_cast<size_t>(r) * vdim];
          }
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int r = rb + u * rg;
        if (r < dim) {
          const float k = s_k[r], q = s_q[r];
#pragma unroll
          for (int i = 0; i < V; ++i) {
            x[u][i] = fmaf(k, s_v[c + i] - x[u][i], x[u][i]);
            acc[i] = fmaf(q, x[u][i], acc[i]);
          }
          if constexpr (V == 4) *reinterpret_cast<float4*>(S + static_cast<size_t>(r) * vdim) = make_float4(x[u][0], x[u][1], x[u][2], x[u][3]);
          else S[static_cast<size_t>(r) * vdim] = x[u][0];
        }
      }
    }
#pragma unroll
    for (int i = 0; i < V; ++i) s_o[r0 * vdim + c + i] = acc[i];
  }
  __syncthreads();
  float y = 0.f;                                  // vdim ≤ 256: a thread finishes one column
  if (tid < vdim)
    for (int r = 0; r < rg; ++r) y += s_o[r * vdim + tid];
  const float part = warp_sum(y * y);
  if ((tid & 31) == 0) s_part[tid >> 5] = part;
  __syncthreads();
  float ss = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) ss += s_part[w];
  if (tid < vdim) st(o + tid, y * rsqrtf(ss / vdim + p.eps) * ld(p.weight + tid));
}

namespace {

template <typename T>
Hgrn2<T> hgrn2_args(const torch::Tensor& proj, int64_t q0, int64_t f0, int64_t v0, int64_t H, int64_t dim, int64_t vdim, const torch::Tensor& bias,
                    const torch::Tensor& lower, const torch::Tensor& weight, double eps, torch::Tensor& o, const OptT& pool, const OptT& slot) {
  Hgrn2<T> p{};
  const T* base = reinterpret_cast<const T*>(proj.data_ptr());
  p.q = base + q0; p.f = base + f0; p.v = base + v0; p.ld = proj.stride(0);
  p.bias = reinterpret_cast<const T*>(bias.data_ptr()); p.lower = reinterpret_cast<const T*>(lower.data_ptr());
  p.weight = reinterpret_cast<const T*>(weight.data_ptr()); p.o = reinterpret_cast<T*>(o.data_ptr());
  if (pool.has_value() && pool->defined()) { p.pool = pool->data_ptr<float>(); p.slot = slot->data_ptr<int>(); }
  p.H = H; p.dim = dim; p.vdim = vdim; p.eps = eps;
  return p;
}

void hgrn2_check(const torch::Tensor& proj, int64_t q0, int64_t f0, int64_t v0, int64_t H, int64_t dim, int64_t vdim, const torch::Tensor& bias,
                 const torch::Tensor& lower, const torch::Tensor& weight, const OptT& pool, const OptT& slot) {
  const auto st = proj.scalar_type();
  TORCH_CHECK(proj.is_cuda() && proj.dim() == 2 && proj.stride(1) == 1 && (st == torch::kBFloat16 || st == torch::kFloat32), "projection [rows, N] bf16 or fp32");
  TORCH_CHECK(H > 0 && dim > 0 && vdim > 0 && dim <= 256 && vdim <= 256, "hgrn2: head widths up to 256");
  TORCH_CHECK(q0 >= 0 && f0 >= 0 && v0 >= 0 && q0 + H * dim <= proj.size(1) && f0 + H * dim <= proj.size(1) && v0 + H * vdim <= proj.size(1), "columns outside the projection");
  for (const auto* t : {&bias, &lower}) TORCH_CHECK(t->scalar_type() == st && t->is_contiguous() && t->numel() == H * dim, "gate bias and lower bound [heads·dim]");
  TORCH_CHECK(weight.scalar_type() == st && weight.is_contiguous() && weight.numel() == vdim, "norm weight [vdim]");
  if (pool.has_value() && pool->defined()) {
    TORCH_CHECK(pool->scalar_type() == torch::kFloat32 && pool->is_contiguous() && pool->dim() == 4 && pool->size(1) == H && pool->size(2) == dim && pool->size(3) == vdim,
                "state pool [slots, heads, dim, vdim] fp32");
    TORCH_CHECK(slot.has_value() && slot->defined() && slot->scalar_type() == torch::kInt32 && slot->is_contiguous() && slot->numel() == proj.size(0), "slot int32 [rows]");
  }
}

bool on16(const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; }

}  // namespace

torch::Tensor hgrn2_prefill(const torch::Tensor& proj, int64_t q0, int64_t f0, int64_t v0, int64_t H, int64_t dim, int64_t vdim, const torch::Tensor& bias,
                            const torch::Tensor& lower, const torch::Tensor& weight, double eps, const torch::Tensor& cu, int64_t max_seqlen, const OptT& pool,
                            const OptT& slot) {
  hgrn2_check(proj, q0, f0, v0, H, dim, vdim, bias, lower, weight, pool, slot);
  TORCH_CHECK(cu.is_cuda() && cu.scalar_type() == torch::kInt32 && cu.is_contiguous(), "cu_seqlens int32 on device");
  c10::cuda::CUDAGuard guard(proj.device());
  const int rows = proj.size(0), n = cu.numel() - 1;
  auto o = torch::empty({rows, H * vdim}, proj.options());
  if (rows == 0 || n <= 0 || max_seqlen <= 0) return o;
  auto f32 = proj.options().dtype(torch::kFloat32);
  auto stream = at::cuda::getCurrentCUDAStream();
  auto run = [&](auto tag) {
    using T = decltype(tag);
    auto p = hgrn2_args<T>(proj, q0, f0, v0, H, dim, vdim, bias, lower, weight, eps, o, pool, slot);
    p.cu = cu.data_ptr<int>();
    const int rpt = dim <= 64 ? 32 : 64, rs = dim <= 32 ? 1 : (dim <= 128 ? 2 : 4);
    const int most = 256 / rs * 2;                               // columns a block can hold
    p.slices = (vdim + most - 1) / most;
    p.cols = p.slices == 1 ? (vdim + 1) / 2 * 2 : most;
    torch::Tensor raw, part, decay;
    if (p.slices > 1) { raw = torch::empty({rows, H * vdim}, f32); p.raw = raw.data_ptr<float>(); }
    // time segments: enough blocks for two per SM, none shorter than 128 tokens (a segment costs a second pass over its state)
    const long blocks = static_cast<long>(H) * p.slices * n;
    long segs = blocks >= num_sms() ? 1 : std::min<long>((2L * num_sms() + blocks - 1) / blocks, max_seqlen / 128);
    segs = std::max<long>(segs, 1);
    p.seg_len = static_cast<int>(((max_seqlen + segs - 1) / segs + hg::CH - 1) / hg::CH * hg::CH);
    p.segments = static_cast<int>((max_seqlen + p.seg_len - 1) / p.seg_len);
    if (p.segments > 1) {
      part = torch::empty({n, p.segments - 1, H, dim, vdim}, f32);
      decay = torch::empty({n, p.segments - 1, H, dim}, f32);
      p.part = part.data_ptr<float>(); p.decay = decay.data_ptr<float>();
    }
    TORCH_CHECK(n <= 65535, "too many sequences in one call");
    constexpr int E = 16 / sizeof(T);
    const bool vec = dim % E == 0 && vdim % E == 0 && p.cols % E == 0 && p.ld % E == 0 && on16(p.q) && on16(p.f) && on16(p.v);
    const int threads = (((std::min<int>(p.cols, vdim) + 1) / 2) * rs + 31) / 32 * 32, dp = rpt * rs;
    const size_t smem = sizeof(float) * (2 * hg::CH * dp + hg::CH * p.cols + 2 * dp) + (vec ? sizeof(T) * hg::CH * (2 * dim + p.cols) : 0);
    auto go = [&](auto kern, int segments) {
      TK_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
      kern<<<dim3(H * p.slices, segments, n), threads, smem, stream>>>(p);
      count_launch();
      TK_CUDA_CHECK(cudaGetLastError());
    };
#define TK_HGRN2(PART, SEGS)                                                                                             \
  do {                                                                                                                   \
    if (vec) {                                                                                                           \
      if (rpt == 32 && rs == 1) go(hgrn2_prefill_kernel<T, 32, 1, true, PART>, SEGS);                                    \
      else if (rpt == 32) go(hgrn2_prefill_kernel<T, 32, 2, true, PART>, SEGS);                                          \
      else if (rs == 2) go(hgrn2_prefill_kernel<T, 64, 2, true, PART>, SEGS);                                            \
      else go(hgrn2_prefill_kernel<T, 64, 4, true, PART>, SEGS);                                                         \
    } else {                                                                                                             \
      if (rpt == 32 && rs == 1) go(hgrn2_prefill_kernel<T, 32, 1, false, PART>, SEGS);                                   \
      else if (rpt == 32) go(hgrn2_prefill_kernel<T, 32, 2, false, PART>, SEGS);                                         \
      else if (rs == 2) go(hgrn2_prefill_kernel<T, 64, 2, false, PART>, SEGS);                                           \
      else go(hgrn2_prefill_kernel<T, 64, 4, false, PART>, SEGS);                                                        \
    }                                                                                                                    \
  } while (0)
    if (p.segments > 1) {
      TK_HGRN2(true, p.segments - 1);
      hgrn2_scan_kernel<<<dim3(static_cast<unsigned>((H * dim * vdim + 255) / 256), n), 256, 0, stream>>>(p.part, p.decay, cu.data_ptr<int>(), H, dim, vdim, p.seg_len,
                                                                                                          p.segments);
      count_launch();
    }
    TK_HGRN2(false, p.segments);
#undef TK_HGRN2
    if (p.raw != nullptr) {
      const long heads = static_cast<long>(rows) * H;
      hgrn2_norm_kernel<T><<<static_cast<unsigned>((heads + 7) / 8), 256, 0, stream>>>(p.raw, p.weight, p.o, heads, vdim, p.eps);
      count_launch();
    }
    TK_CUDA_CHECK(cudaGetLastError());
  };
  if (proj.scalar_type() == torch::kBFloat16) run(bf16{}); else run(float{});
  return o;
}

torch::Tensor hgrn2_step(const torch::Tensor& proj, int64_t q0, int64_t f0, int64_t v0, int64_t H, int64_t dim, int64_t vdim, const torch::Tensor& bias,
                         const torch::Tensor& lower, const torch::Tensor& weight, double eps, const torch::Tensor& pool, const torch::Tensor& slot) {
  hgrn2_check(proj, q0, f0, v0, H, dim, vdim, bias, lower, weight, pool, slot);
  c10::cuda::CUDAGuard guard(proj.device());
  const int rows = proj.size(0);
  auto o = torch::empty({rows, H * vdim}, proj.options());
  if (rows == 0) return o;
  TORCH_CHECK(rows <= 65535, "too many sequences in one step");
  auto stream = at::cuda::getCurrentCUDAStream();
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const auto p = hgrn2_args<T>(proj, q0, f0, v0, H, dim, vdim, bias, lower, weight, eps, o, pool, slot);
    const int v = vdim % 4 == 0 ? 4 : 1, rg = 256 / static_cast<int>(vdim / v);
    const size_t smem = sizeof(float) * (2 * dim + (vdim + 3) / 4 * 4 + static_cast<size_t>(rg) * vdim);
    if (v == 4) hgrn2_step_kernel<T, 4><<<dim3(H, rows), 256, smem, stream>>>(p);
    else hgrn2_step_kernel<T, 1><<<dim3(H, rows), 256, smem, stream>>>(p);
  };
  if (proj.scalar_type() == torch::kBFloat16) run(bf16{}); else run(float{});
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return o;
}

}  // namespace tk
