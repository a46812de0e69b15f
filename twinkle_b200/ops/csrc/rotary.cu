// Rotated heads:
//   rotary_table    cosine and sine of position times frequency for every rotation of a stack, once per forward (fp64 inside, so that
//                   large positions keep their digits)
//   rotary_heads    [q | k | v] columns of a fused projection: bias, RMS norm of q and k per head, rotation, and the writes into the
//                   paged K/V pools — one pass
//   latent_rotary   for latent attention: rotated parts of the queries (in place for prompts, next to the query's place in latent space
//                   for steps), RMS norm of the latent, rotated key part, and the write into the paged pool — one pass
// A pair of dimensions is (2i, 2i + 1) (INTER) or (i, i + n).  Templated on the compute dtype (bf16 or fp32); vector kernels where rows
// are made of whole vectors, plain ones otherwise.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/types.h>

#include "common.cuh"
#include "host.h"
#include "vec.cuh"

namespace tk {

// ---------------------------------------------------------------- rotary_table
__global__ void __launch_bounds__(256) rotary_table_kernel(const int64_t* __restrict__ pos, const double* __restrict__ freq, float2* __restrict__ out, long total, int n) {
  const long i = blockIdx.x * 256L + threadIdx.x;
  if (i >= total) return;
  const long t = i / n;
  double s, c;
  sincos(static_cast<double>(pos[t]) * freq[i - t * n], &s, &c);
  out[i] = make_float2(static_cast<float>(c), static_cast<float>(s));
}

torch::Tensor rotary_table(const torch::Tensor& pos, const torch::Tensor& freq) {
  TORCH_CHECK(pos.is_cuda() && pos.scalar_type() == torch::kInt64 && pos.is_contiguous() && pos.dim() == 1, "positions int64 [rows]");
  TORCH_CHECK(freq.is_cuda() && freq.scalar_type() == torch::kFloat64 && freq.is_contiguous() && freq.dim() == 1, "frequencies fp64 [pairs]");
  c10::cuda::CUDAGuard guard(pos.device());
  auto out = torch::empty({pos.numel(), freq.numel(), 2}, freq.options().dtype(torch::kFloat32));
  const long total = pos.numel() * freq.numel();
  if (total == 0) return out;
  rotary_table_kernel<<<static_cast<unsigned>((total + 255) / 256), 256, 0, at::cuda::getCurrentCUDAStream()>>>(
      pos.data_ptr<int64_t>(), freq.data_ptr<double>(), reinterpret_cast<float2*>(out.data_ptr<float>()), total, static_cast<int>(freq.numel()));
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return out;
}

// ---------------------------------------------------------------- rotary_heads
template <typename T>
struct RotaryHeads {
  const T* proj; long ld;                        // q | k | v from here on
  const T *bias, *qw, *kw;                       // (null: none)
  const float2* table; int table_ld;             // this rotation's first pair; pairs per row of the table
  int pairs, hq, hkv, d, e, dp, ep;              // heads, widths, and row widths of outputs and pools (the rest is written as zero)
  float eps;
  T *q, *k, *v;                                  // k and v may be null
  T *k_pool, *v_pool; const int64_t* pool_row;   // (null: not kept)
  int rows;
};

// LANES threads per (row, head), eight elements each.  All heads of a group of threads belong to one row, so the row's angles are read
// once; the next head's elements are on their way while one is worked on.
template <typename T, int LANES, bool INTER>
__global__ void __launch_bounds__(128) rotary_heads_kernel(const RotaryHeads<T> p) {
  constexpr int GROUPS = 128 / LANES;
  const int t = blockIdx.x, sub = threadIdx.x % LANES, el = sub * 8, step = gridDim.y * GROUPS;
  const int heads = p.hq + 2 * p.hkv;
  int head = blockIdx.y * GROUPS + threadIdx.x / LANES;
  const int rounds = (heads - static_cast<int>(blockIdx.y) * GROUPS + step - 1) / step;     // the same for the whole block
  const T* row = p.proj + static_cast<size_t>(t) * p.ld;
  const int64_t kept = p.pool_row != nullptr ? p.pool_row[t] : -1;
  const int n = p.pairs, dims = 2 * n;
  float cs[8], sn[8];
  {
    // rotate-half: el < 2n and n a multiple of 8, so the eight pairs lie side by side
    const float2* a = p.table + static_cast<size_t>(t) * p.table_ld + (INTER ? el / 2 : (el < n ? el : el - n));
#pragma unroll
    for (int c = 0; c < 8; ++c) {
      float2 v = make_float2(1.f, 0.f);
      if (el + c < dims) v = a[INTER ? c / 2 : c];
      cs[c] = v.x; sn[c] = v.y;
    }
  }
  // rotate-half: n is a multiple of 8, so the partners of these eight elements are another thread's eight
  const bool lower = el < n, turns = el < dims;
  const float inv_d = 1.f / p.d;
  const int lane = threadIdx.x & 31, partner = INTER || !turns ? lane : (lower ? lane + n / 8 : lane - n / 8);
  auto column = [&](int h) { return h < p.hq + p.hkv ? h * p.d : (p.hq + p.hkv) * p.d + (h - p.hq - p.hkv) * p.e; };
  auto fetch = [&](int h, Raw8<T>& r) {
    r.zero();
    if (h < heads && el < (h < p.hq + p.hkv ? p.d : p.e)) r.load(row + column(h) + el);
  };
  Raw8<T> cur, nxt;
  fetch(head, cur);
  for (int i = 0; i < rounds; ++i, head += step) {
    fetch(head + step, nxt);
    const bool live = head < heads, is_v = head >= p.hq + p.hkv, is_q = head < p.hq;
    const int width = is_v ? p.e : p.d;
    const bool own = live && el < width;
    float y[8];
    cur.get(y);
    if (p.bias != nullptr && own) {
      float b[8];
      Raw8<T> r;
      r.load(p.bias + column(head) + el);
      r.get(b);
#pragma unroll
      for (int c = 0; c < 8; ++c) y[c] += b[c];
    }
    const T* w = is_q ? p.qw : p.kw;
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < 8; ++c) ss += y[c] * y[c];
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!is_v && w != nullptr && own) {
      float g[8];
      Raw8<T> r;
      r.load(w + el);
      r.get(g);
      const float f = rsqrtf(ss * inv_d + p.eps);
#pragma unroll
      for (int c = 0; c < 8; ++c) y[c] *= f * g[c];
    }
    if constexpr (INTER) {
      if (!is_v) {
#pragma unroll
        for (int c = 0; c < 8; c += 2) {
          const float u = y[c], v = y[c + 1];
          y[c] = u * cs[c] - v * sn[c];
          y[c + 1] = v * cs[c] + u * sn[c];
        }
      }
    } else {
#pragma unroll
      for (int c = 0; c < 8; ++c) {
        const float other = __shfl_sync(0xffffffffu, y[c], partner);
        if (!is_v && turns) y[c] = lower ? y[c] * cs[c] - other * sn[c] : y[c] * cs[c] + other * sn[c];
      }
    }
    if (own) {
      Raw8<T> r;
      r.set(y);
      if (is_q) {
        r.store(p.q + (static_cast<size_t>(t) * p.hq + head) * p.d + el);
      } else {
        const int g = is_v ? head - p.hq - p.hkv : head - p.hq;
        T *out = is_v ? p.v : p.k, *pool = is_v ? p.v_pool : p.k_pool;
        if (out != nullptr) r.store(out + (static_cast<size_t>(t) * p.hkv + g) * width + el);
        if (kept >= 0) r.store(pool + (static_cast<size_t>(kept) * p.hkv + g) * width + el);
      }
    }
    cur = nxt;
  }
}

// Any widths: one block per (row, head), element-wise.
template <typename T, bool INTER>
__global__ void __launch_bounds__(128) rotary_heads_plain_kernel(const RotaryHeads<T> p) {
  extern __shared__ float head_buf[];
  __shared__ float sh[32];
  const int t = blockIdx.x, head = blockIdx.y;
  const bool is_v = head >= p.hq + p.hkv, is_q = head < p.hq;
  const int width = is_v ? p.e : p.d, padded = is_v ? p.ep : p.dp, g = is_q ? head : (is_v ? head - p.hq - p.hkv : head - p.hq);
  const int c0 = is_v ? (p.hq + p.hkv) * p.d + g * p.e : head * p.d;
  const T* row = p.proj + static_cast<size_t>(t) * p.ld + c0;
  float ss = 0.f;
  for (int el = threadIdx.x; el < width; el += 128) {
    const float y = to_f(row[el]) + (p.bias != nullptr ? to_f(p.bias[c0 + el]) : 0.f);
    head_buf[el] = y;
    ss += y * y;
  }
  const T* w = is_v ? nullptr : (is_q ? p.qw : p.kw);
  const float f = rsqrtf(block_sum(ss, sh) / width + p.eps);
  __syncthreads();
  const int64_t kept = p.pool_row != nullptr && !is_q ? p.pool_row[t] : -1;
  T* out = is_q ? p.q : (is_v ? p.v : p.k);
  T* pool = is_v ? p.v_pool : p.k_pool;
  const int own = is_q ? p.hq : p.hkv;
  auto normed = [&](int el) { return w != nullptr ? head_buf[el] * f * to_f(w[el]) : head_buf[el]; };
  for (int el = threadIdx.x; el < padded; el += 128) {
    float y = el < width ? normed(el) : 0.f;
    if (!is_v && el < 2 * p.pairs) {
      const bool lower = INTER ? (el & 1) == 0 : el < p.pairs;
      const float2 a = p.table[static_cast<size_t>(t) * p.table_ld + (INTER ? el / 2 : el % p.pairs)];
      const float other = normed(INTER ? el ^ 1 : (lower ? el + p.pairs : el - p.pairs));
      y = lower ? y * a.x - other * a.y : y * a.x + other * a.y;
    }
    if (out != nullptr) out[(static_cast<size_t>(t) * own + g) * padded + el] = from_f<T>(y);
    if (kept >= 0) pool[(static_cast<size_t>(kept) * own + g) * padded + el] = from_f<T>(y);
  }
}

template <typename T, bool INTER>
static void launch_rotary_heads(const RotaryHeads<T>& p) {
  auto stream = at::cuda::getCurrentCUDAStream();
  const int heads = p.hq + 2 * p.hkv, widest = std::max(p.d, p.hkv > 0 ? p.e : 0);
  const bool vec = p.d % 8 == 0 && p.e % 8 == 0 && p.ld % 8 == 0 && widest <= 256 && (INTER || p.pairs % 8 == 0) && aligned16(p.proj) && aligned16(p.bias) &&
                   aligned16(p.qw) && aligned16(p.kw);
  if (vec) {
    auto go = [&](auto kern, int lanes) {
      // up to four heads per group of threads once there are blocks enough to fill the device
      const int groups = 128 / lanes, most = (heads + groups - 1) / groups;
      const int want = static_cast<int>(std::min<long>(most, std::max<long>((heads + 4 * groups - 1) / (4 * groups), (num_sms() * 8L + p.rows - 1) / p.rows)));
      kern<<<dim3(p.rows, want), 128, 0, stream>>>(p);
    };
    if (widest <= 64) go(rotary_heads_kernel<T, 8, INTER>, 8);
    else if (widest <= 128) go(rotary_heads_kernel<T, 16, INTER>, 16);
    else go(rotary_heads_kernel<T, 32, INTER>, 32);
  } else {
    const size_t smem = sizeof(float) * std::max(p.d, p.e);
    TORCH_CHECK(smem <= 48 * 1024 && heads <= 65535, "head width or count too large");
    rotary_heads_plain_kernel<T, INTER><<<dim3(p.rows, heads), 128, smem, stream>>>(p);
  }
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
}

// proj [rows, N]; table [rows, all pairs, 2] fp32, of which columns at … at + pairs belong to this rotation.  hkv 0: queries only.
// Returns {q} or, with want_kv and hkv > 0, {q, k, v}.
std::vector<torch::Tensor> rotary_heads(const torch::Tensor& proj, int64_t first, const OptT& bias, const OptT& qw, const OptT& kw, const torch::Tensor& table, int64_t at,
                                        int64_t pairs, bool interleaved, int64_t hq, int64_t hkv, int64_t d, int64_t e, double eps, const OptT& k_pool, const OptT& v_pool,
                                        const OptT& pool_row, bool want_kv) {
  const auto st = proj.scalar_type();
  TORCH_CHECK(proj.is_cuda() && proj.dim() == 2 && proj.stride(1) == 1 && (st == torch::kBFloat16 || st == torch::kFloat32), "proj [rows, N] bf16 or fp32");
  const int64_t rows = proj.size(0), C = (hq + hkv) * d + hkv * e, dp = (d + 7) / 8 * 8, ep = (e + 7) / 8 * 8;
  TORCH_CHECK(hq > 0 && hkv >= 0 && d > 0 && e > 0 && first >= 0 && proj.size(1) >= first + C, "projection narrower than its q | k | v columns");
  TORCH_CHECK(table.is_cuda() && table.scalar_type() == torch::kFloat32 && table.is_contiguous() && table.dim() == 3 && table.size(0) == rows && table.size(2) == 2 && at >= 0 &&
                  pairs >= 1 && at + pairs <= table.size(1) && 2 * pairs <= d, "table of angles [rows, pairs, 2] fp32");
  auto vector = [&](const OptT& t, int64_t len) { return !has(t) || (t->is_cuda() && t->scalar_type() == st && t->is_contiguous() && t->numel() == len); };
  TORCH_CHECK(vector(bias, C) && vector(qw, d) && vector(kw, d), "bias [q | k | v columns] and norm weights [d] in the projection's dtype");
  if (has(pool_row)) {
    TORCH_CHECK(hkv > 0 && has(k_pool) && has(v_pool) && k_pool->scalar_type() == st && v_pool->scalar_type() == st && k_pool->is_contiguous() && v_pool->is_contiguous() &&
                    k_pool->size(-1) == dp && v_pool->size(-1) == ep && k_pool->size(-2) == hkv && v_pool->size(-2) == hkv, "pools [..., hkv, dp] and [..., hkv, ep]");
    TORCH_CHECK(pool_row->scalar_type() == torch::kInt64 && pool_row->is_contiguous() && pool_row->numel() == rows, "pool rows int64 [rows]");
  }
  c10::cuda::CUDAGuard guard(proj.device());
  const bool kv = want_kv && hkv > 0;
  std::vector<torch::Tensor> out{torch::empty({rows, hq, dp}, proj.options())};
  if (kv) {
    out.push_back(torch::empty({rows, hkv, dp}, proj.options()));
    out.push_back(torch::empty({rows, hkv, ep}, proj.options()));
  }
  if (rows == 0) return out;
  auto fill = [&](auto tag) {
    using T = decltype(tag);
    auto ptr = [](const OptT& t) { return has(t) ? reinterpret_cast<T*>(t->data_ptr()) : static_cast<T*>(nullptr); };
    RotaryHeads<T> p{};
    p.proj = reinterpret_cast<const T*>(proj.data_ptr()) + first; p.ld = proj.stride(0); p.bias = ptr(bias); p.qw = ptr(qw); p.kw = ptr(kw);
    p.table = reinterpret_cast<const float2*>(table.data_ptr<float>()) + at; p.table_ld = table.size(1);
    p.pairs = pairs; p.hq = hq; p.hkv = hkv; p.d = d; p.e = e; p.dp = dp; p.ep = ep; p.eps = eps; p.rows = rows;
    p.q = reinterpret_cast<T*>(out[0].data_ptr());
    if (kv) { p.k = reinterpret_cast<T*>(out[1].data_ptr()); p.v = reinterpret_cast<T*>(out[2].data_ptr()); }
    if (has(pool_row)) { p.pool_row = pool_row->data_ptr<int64_t>(); p.k_pool = ptr(k_pool); p.v_pool = ptr(v_pool); }
    if (interleaved) launch_rotary_heads<T, true>(p); else launch_rotary_heads<T, false>(p);
  };
  if (st == torch::kBFloat16) fill(bf16{}); else fill(float{});
  return out;
}

// --------------------------------------------------------------- latent_rotary
template <typename T>
struct LatentRotary {
  T* proj; long ld;
  int q0, heads, d, r, c0, nc, wide;             // wide: row width of kept and pool
  const T* w;
  const float2* table; int table_ld;
  T* ql; int ql_ld;                              // [rows, heads, ql_ld]: rotated queries go into the last r columns (null: in place)
  T* kept;                                       // [rows, wide] (null: not wanted)
  T* pool; const int64_t* pool_row;
  float eps;
};

// One block per row.  Warp 0: the latent and its key part.  The others (all four when the layer borrows): rotated parts of the
// queries, VEC: eight elements of an interleaved rotation per access, otherwise a pair per thread.
template <typename T, bool INTER, bool VEC>
__global__ void __launch_bounds__(128) latent_rotary_kernel(const LatentRotary<T> p) {
  const int t = blockIdx.x, lane = threadIdx.x & 31, n = p.r / 2;
  T* row = p.proj + static_cast<size_t>(t) * p.ld;
  const float2* a = p.table + static_cast<size_t>(t) * p.table_ld;
  if (p.nc > 0 && threadIdx.x < 32) {
    const T* c = row + p.c0;
    float ss = 0.f;
    for (int j = lane; j < p.nc; j += 32) { const float v = to_f(c[j]); ss += v * v; }
    const float f = rsqrtf(warp_sum(ss) / p.nc + p.eps);
    const int64_t place = p.pool != nullptr ? p.pool_row[t] : -1;
    T* kept = p.kept != nullptr ? p.kept + static_cast<size_t>(t) * p.wide : nullptr;
    T* pool = place >= 0 ? p.pool + static_cast<size_t>(place) * p.wide : nullptr;
    for (int j = lane; j < p.wide; j += 32) {
      float v = 0.f;
      if (j < p.nc) {
        v = to_f(c[j]) * f * to_f(p.w[j]);
      } else if (j < p.nc + p.r) {
        const int i = j - p.nc;
        const bool lower = INTER ? (i & 1) == 0 : i < n;
        const float2 g = a[INTER ? i / 2 : i % n];
        const float own = to_f(c[j]), other = to_f(c[p.nc + (INTER ? i ^ 1 : (lower ? i + n : i - n))]);
        v = lower ? own * g.x - other * g.y : own * g.x + other * g.y;
      }
      if (kept != nullptr) kept[j] = from_f<T>(v);
      if (pool != nullptr) pool[j] = from_f<T>(v);
    }
    return;
  }
  const int skip = p.nc > 0 ? 32 : 0, threads = 128 - skip, per = VEC ? p.r / 8 : n;
  for (int i = threadIdx.x - skip; i < p.heads * per; i += threads) {
    const int h = i / per, k = i - h * per;
    T* src = row + p.q0 + h * (p.d + p.r) + p.d;
    T* dst = p.ql != nullptr ? p.ql + (static_cast<size_t>(t) * p.heads + h) * p.ql_ld + p.ql_ld - p.r : src;
    if constexpr (VEC) {
      Raw8<T> raw;
      float y[8];
      raw.load(src + k * 8);
      raw.get(y);
#pragma unroll
      for (int c = 0; c < 8; c += 2) {
        const float2 g = a[k * 4 + c / 2];
        const float u = y[c], v = y[c + 1];
        y[c] = u * g.x - v * g.y;
        y[c + 1] = v * g.x + u * g.y;
      }
      raw.set(y);
      raw.store(dst + k * 8);
    } else {
      const int i0 = INTER ? 2 * k : k, i1 = INTER ? 2 * k + 1 : k + n;
      const float2 g = a[k];
      const float u = to_f(src[i0]), v = to_f(src[i1]);
      dst[i0] = from_f<T>(u * g.x - v * g.y);
      dst[i1] = from_f<T>(v * g.x + u * g.y);
    }
  }
}

// Queries [d | r] per head from column q0, [latent | key part] = [nc | r] from column c0 of proj [rows, N] (nc 0: none).  Without ql the rotated
// queries replace the projection's; with ql [rows, heads, ·] they go into its last r columns.  Returns [rows, (nc + r) rounded up to 8], or an
// empty tensor when there is none or it is not wanted.
torch::Tensor latent_rotary(const torch::Tensor& proj, int64_t q0, int64_t heads, int64_t d, int64_t r, int64_t c0, int64_t nc, const OptT& w, double eps, const OptT& table,
                            int64_t at, int64_t pairs, bool interleaved, const OptT& ql, const OptT& pool, const OptT& pool_row, bool want_kept) {
  const auto st = proj.scalar_type();
  TORCH_CHECK(proj.is_cuda() && proj.dim() == 2 && proj.stride(1) == 1 && (st == torch::kBFloat16 || st == torch::kFloat32), "proj [rows, N] bf16 or fp32");
  const int64_t rows = proj.size(0), wide = (nc + r + 7) / 8 * 8;
  TORCH_CHECK(heads > 0 && d > 0 && r >= 0 && r % 2 == 0 && nc >= 0 && q0 >= 0 && c0 >= 0 && q0 + heads * (d + r) <= proj.size(1) && (nc == 0 || c0 + nc + r <= proj.size(1)),
              "columns outside the projection");
  TORCH_CHECK(2 * pairs == r, "one pair for every two rotated dimensions");
  if (r > 0)
    TORCH_CHECK(has(table) && table->is_cuda() && table->scalar_type() == torch::kFloat32 && table->is_contiguous() && table->dim() == 3 && table->size(0) == rows &&
                    table->size(2) == 2 && at >= 0 && at + pairs <= table->size(1), "table of angles [rows, pairs, 2] fp32");
  if (nc > 0) TORCH_CHECK(has(w) && w->scalar_type() == st && w->is_contiguous() && w->numel() == nc, "latent norm weight");
  if (has(ql)) TORCH_CHECK(ql->scalar_type() == st && ql->is_contiguous() && ql->dim() == 3 && ql->size(0) == rows && ql->size(1) == heads && ql->size(2) >= r, "ql [rows, heads, .]");
  if (has(pool)) {
    TORCH_CHECK(nc > 0 && pool->scalar_type() == st && pool->is_contiguous() && pool->size(-1) == wide, "latent pool [..., latent and key part rounded up to 8]");
    TORCH_CHECK(has(pool_row) && pool_row->scalar_type() == torch::kInt64 && pool_row->is_contiguous() && pool_row->numel() == rows, "pool rows int64 [rows]");
  }
  c10::cuda::CUDAGuard guard(proj.device());
  auto kept = torch::empty({want_kept && nc > 0 ? rows : 0, wide}, proj.options());
  if (rows == 0 || (r == 0 && nc == 0)) return kept;
  auto stream = at::cuda::getCurrentCUDAStream();
  auto run = [&](auto tag) {
    using T = decltype(tag);
    LatentRotary<T> p{};
    p.proj = reinterpret_cast<T*>(proj.data_ptr()); p.ld = proj.stride(0); p.q0 = q0; p.heads = r > 0 ? heads : 0; p.d = d; p.r = r; p.c0 = c0; p.nc = nc; p.wide = wide;
    p.w = nc > 0 ? reinterpret_cast<const T*>(w->data_ptr()) : nullptr;
    if (r > 0) { p.table = reinterpret_cast<const float2*>(table->data_ptr<float>()) + at; p.table_ld = table->size(1); }
    if (has(ql)) { p.ql = reinterpret_cast<T*>(ql->data_ptr()); p.ql_ld = ql->size(2); }
    if (kept.numel() > 0) p.kept = reinterpret_cast<T*>(kept.data_ptr());
    if (has(pool)) { p.pool = reinterpret_cast<T*>(pool->data_ptr()); p.pool_row = pool_row->data_ptr<int64_t>(); }
    p.eps = eps;
    const bool vec = interleaved && r % 8 == 0 && r > 0 && d % 8 == 0 && q0 % 8 == 0 && p.ld % 8 == 0 && aligned16(p.proj) && p.ql_ld % 8 == 0 && aligned16(p.ql);
    if (vec) latent_rotary_kernel<T, true, true><<<rows, 128, 0, stream>>>(p);
    else if (interleaved) latent_rotary_kernel<T, true, false><<<rows, 128, 0, stream>>>(p);
    else latent_rotary_kernel<T, false, false><<<rows, 128, 0, stream>>>(p);
  };
  if (st == torch::kBFloat16) run(bf16{}); else run(float{});
  count_launch();
  TK_CUDA_CHECK(cudaGetLastError());
  return kept;
}

}  // namespace tk
