// Row-wise building blocks of ragged-batch language-model steps with an fp32 residual stream:
// embedding gather, RMS norm (plain or zero-centred weights, optional scatter into a paged pool),
// the gated + normed residual update, and the router / grouping kernels of routed experts.
// All arithmetic is fp32; tensors are read and written in the dtype their code names.
// These kernels (and the other ragged-batch kernels: glinear, latent_attn, hgrn2) are launched
// stream-serialised (launch_serial), not with programmatic dependent launch: overlapping them with the
// persistent GEMMs deadlocked in one measured configuration, so they neither start early nor release
// their successor early.
#include "../../include/vila_b200.h"
#include "common.cuh"
#include "kernels.h"
#include "dtype_any.cuh"

namespace vb {
namespace {

constexpr int kRowThreads = 256;
constexpr int kRowsPerCta = kRowThreads / 32;
constexpr int kWideCols = 512;  // rows at least this wide get a whole CTA, narrower ones a warp

// TPR threads share a row: 32 = one warp (8 rows per CTA), 256 = the whole CTA.
template <int TPR>
__device__ __forceinline__ float row_sum(float v, float* red) {
  v = warp_sum(v);
  if (TPR == 32) return v;
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
  __syncthreads();
  if (l == 0) red[w] = v;
  __syncthreads();
  float t = l < kRowsPerCta ? red[l] : 0.f;
  return warp_sum(t);
}
template <int TPR>
__device__ __forceinline__ int row_of() {
  return TPR == 32 ? blockIdx.x * kRowsPerCta + (threadIdx.x >> 5) : blockIdx.x;
}
template <int TPR>
__device__ __forceinline__ int col0_of() { return TPR == 32 ? (threadIdx.x & 31) : threadIdx.x; }

__global__ void __launch_bounds__(kRowThreads)
embed_rows_kernel(const void* __restrict__ table, int dt, const int32_t* __restrict__ ids,
                  float* __restrict__ out, int rows, int cols) {
  const int row = blockIdx.x * kRowsPerCta + (threadIdx.x >> 5);
  if (row >= rows) return;
  const size_t src = static_cast<size_t>(ids[row]) * cols;
  float* o = out + static_cast<size_t>(row) * cols;
  for (int c = lane_id(); c < cols; c += 32) o[c] = ld_any(table, dt, src + c);
}

template <int TPR>
__global__ void __launch_bounds__(kRowThreads)
rmsnorm_rows_kernel(const void* __restrict__ x, int x_dt, int64_t ldx, const void* __restrict__ w,
                    int w_dt, float w_off, float eps, void* __restrict__ out, int o_dt, int64_t ldo,
                    const int32_t* __restrict__ out_rows, int rows, int cols, int groups) {
  // groups > 1: `rows` counts (row, piece) pairs, `cols` is the width of a piece; piece g of row r
  // starts at column g * cols and uses the weights [g * cols, (g + 1) * cols)
  __shared__ float red[kRowsPerCta];
  const int vrow = row_of<TPR>();
  if (vrow >= rows) return;   // TPR == 256: uniform over the CTA
  const int row = vrow / groups, piece = vrow - row * groups;
  const size_t xb = static_cast<size_t>(row) * ldx + static_cast<size_t>(piece) * cols;
  if (w) w = static_cast<const char*>(w) + static_cast<size_t>(piece) * cols * (w_dt ? 4 : 2);
  float ss = 0.f;
  for (int c = col0_of<TPR>(); c < cols; c += TPR) {
    const float v = ld_any(x, x_dt, xb + c);
    ss += v * v;
  }
  ss = row_sum<TPR>(ss, red);
  const float r = 1.0f / sqrtf(ss / static_cast<float>(cols) + eps);
  const size_t ob = static_cast<size_t>(out_rows ? out_rows[row] : row) * ldo + static_cast<size_t>(piece) * cols;
  for (int c = col0_of<TPR>(); c < cols; c += TPR) {
    const float g = w ? ld_any(w, w_dt, c) + w_off : 1.0f;
    st_any(out, o_dt, ob + c, ld_any(x, x_dt, xb + c) * r * g);
  }
}

// Pre-norm residual step in one pass: x += a + sum_j part_j (a first, then the partials by index), then
// out = x / sqrt(mean(x^2) + eps) * w: the operand of the sublayer that reads x next.
template <int TPR>
__global__ void __launch_bounds__(kRowThreads)
residual_norm_rows_kernel(float* __restrict__ x, const void* __restrict__ a, int a_dt, int64_t lda,
                          const void* __restrict__ part, int p_dt, int64_t ldp, int np, const void* __restrict__ w,
                          int w_dt, float eps, void* __restrict__ out, int o_dt, int rows, int cols) {
  __shared__ float red[kRowsPerCta];
  const int row = row_of<TPR>();
  if (row >= rows) return;
  float* xr = x + static_cast<size_t>(row) * cols;
  float ss = 0.f;
  for (int c = col0_of<TPR>(); c < cols; c += TPR) {
    float y = a ? ld_any(a, a_dt, static_cast<size_t>(row) * lda + c) : 0.f;
    if (part)
      for (int j = 0; j < np; ++j) y += ld_any(part, p_dt, (static_cast<size_t>(row) * np + j) * ldp + c);
    const float v = xr[c] + y;
    xr[c] = v;
    ss += v * v;
  }
  ss = row_sum<TPR>(ss, red);
  const float r = 1.0f / sqrtf(ss / static_cast<float>(cols) + eps);
  for (int c = col0_of<TPR>(); c < cols; c += TPR)   // every thread re-reads the columns it wrote itself
    st_any(out, o_dt, static_cast<size_t>(row) * cols + c, xr[c] * r * (w ? ld_any(w, w_dt, c) : 1.0f));
}

__device__ __forceinline__ float gated_value(const void* part, int p_dt, int64_t ldp, int np,
                                             const void* gate, int g_dt, int64_t ldg,
                                             const void* gb, int b_dt, int row, int c) {
  float y = 0.f;
  for (int j = 0; j < np; ++j)
    y += ld_any(part, p_dt, (static_cast<size_t>(row) * np + j) * ldp + c);
  if (gate) {
    float z = ld_any(gate, g_dt, static_cast<size_t>(row) * ldg + c);
    if (gb) z += ld_any(gb, b_dt, c);
    y *= sigmoid_f(z);
  }
  return y;
}

template <int TPR>
__global__ void __launch_bounds__(kRowThreads)
gated_norm_residual_kernel(float* __restrict__ x, const void* __restrict__ part, int p_dt, int64_t ldp,
                           int np, const void* __restrict__ gate, int g_dt, int64_t ldg,
                           const void* __restrict__ gb, int b_dt, const void* __restrict__ w, int w_dt,
                           float w_off, float eps, float mult, int rows, int cols) {
  __shared__ float red[kRowsPerCta];
  const int row = row_of<TPR>();
  if (row >= rows) return;
  float ss = 0.f;
  for (int c = col0_of<TPR>(); c < cols; c += TPR) {
    const float y = gated_value(part, p_dt, ldp, np, gate, g_dt, ldg, gb, b_dt, row, c);
    ss += y * y;
  }
  ss = row_sum<TPR>(ss, red);
  const float r = 1.0f / sqrtf(ss / static_cast<float>(cols) + eps);
  float* xr = x + static_cast<size_t>(row) * cols;
  for (int c = col0_of<TPR>(); c < cols; c += TPR) {
    const float y = gated_value(part, p_dt, ldp, np, gate, g_dt, ldg, gb, b_dt, row, c);
    const float g = w ? ld_any(w, w_dt, c) + w_off : 1.0f;
    xr[c] += mult * (y * r * g);
  }
}

// ---- routed experts ------------------------------------------------------------------------------
// E logits per token (fp32 dot products over the row), then `top` rounds of arg-max.  TPR == 32: one
// warp per token; TPR == 256 (few tokens): the 8 warps of a CTA split the experts of ONE token.
template <int TPR>
__global__ void __launch_bounds__(kRowThreads)
moe_route_kernel(const void* __restrict__ x, int x_dt, int64_t ldx, const float* __restrict__ wr,
                 const float* __restrict__ bias, int32_t* __restrict__ idx, float* __restrict__ weight,
                 int rows, int cols, int experts, int top) {
  extern __shared__ float z_s[];  // TPR == 32: [kRowsPerCta][experts]; 256: [experts]
  const int wid = threadIdx.x >> 5, lane = lane_id();
  const int row = row_of<TPR>();
  if (row >= rows) return;
  float* z = TPR == 32 ? z_s + wid * experts : z_s;
  const size_t xb = static_cast<size_t>(row) * ldx;
  for (int e = (TPR == 32 ? 0 : wid); e < experts; e += (TPR == 32 ? 1 : kRowsPerCta)) {
    const float* we = wr + static_cast<size_t>(e) * cols;
    float s = 0.f;
    for (int c = lane; c < cols; c += 32) s += ld_any(x, x_dt, xb + c) * we[c];
    s = warp_sum(s);
    if (lane == 0) z[e] = s + (bias ? bias[e] : 0.f);
  }
  if (TPR == 32) __syncwarp();
  else {
    __syncthreads();
    if (wid != 0) return;
  }
  float first = 0.f, denom = 0.f;
  for (int j = 0; j < top; ++j) {
    float best = -INFINITY;
    int bi = 0x7fffffff;
    for (int e = lane; e < experts; e += 32) {
      const float v = z[e];
      if (v > best) { best = v; bi = e; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
    }
    if (j == 0) first = best;
    const float e_j = expf(best - first);
    denom += e_j;
    if (lane == 0) {
      idx[static_cast<size_t>(row) * top + j] = bi;
      weight[static_cast<size_t>(row) * top + j] = e_j;
      z[bi] = -INFINITY;
    }
    __syncwarp();
  }
  if (lane == 0)
    for (int j = 0; j < top; ++j) weight[static_cast<size_t>(row) * top + j] /= denom;
}

// Single CTA: per-expert counts, exclusive prefix, then a stable placement (pair ids stay ascending
// inside every expert's segment) with warp ballots.
__global__ void __launch_bounds__(1024)
moe_group_kernel(const int32_t* __restrict__ idx, int32_t* __restrict__ seg, int32_t* __restrict__ sorted,
                 int pairs, int experts) {
  extern __shared__ int cnt_s[];  // [experts + 1]
  const int wid = threadIdx.x >> 5, lane = lane_id(), nw = blockDim.x >> 5;
  for (int e = wid; e < experts; e += nw) {
    int n = 0;
    for (int p0 = 0; p0 < pairs; p0 += 32) {
      const int p = p0 + lane;
      n += __popc(__ballot_sync(0xffffffffu, p < pairs && idx[p] == e));
    }
    if (lane == 0) cnt_s[e + 1] = n;
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    cnt_s[0] = 0;
    for (int e = 0; e < experts; ++e) cnt_s[e + 1] += cnt_s[e];
  }
  __syncthreads();
  for (int e = threadIdx.x; e <= experts; e += blockDim.x) seg[e] = cnt_s[e];
  for (int e = wid; e < experts; e += nw) {
    int at = cnt_s[e];
    for (int p0 = 0; p0 < pairs; p0 += 32) {
      const int p = p0 + lane;
      const bool mine = p < pairs && idx[p] == e;
      const unsigned m = __ballot_sync(0xffffffffu, mine);
      if (mine) sorted[at + __popc(m & ((1u << lane) - 1u))] = p;
      at += __popc(m);
    }
  }
}

inline int row_grid(int rows) { return (rows + kRowsPerCta - 1) / kRowsPerCta; }

// ---- word row + hashed (previous, current) pair row ------------------------------------------------
__global__ void __launch_bounds__(kRowThreads)
embed_pair_rows_kernel(const void* __restrict__ table, int dt, const void* __restrict__ pair, int pdt,
                       const int32_t* __restrict__ ids, const int32_t* __restrict__ prev, long long mul_prev,
                       long long mul_cur, long long buckets, float* __restrict__ out, int rows, int cols) {
  const int row = blockIdx.x * kRowsPerCta + (threadIdx.x >> 5);
  if (row >= rows) return;
  const long long id = ids[row], pv = prev[row];
  long long r = buckets;
  if (pv >= 0) {
    r = (pv * mul_prev + id * mul_cur) % buckets;
    if (r < 0) r += buckets;
  }
  const size_t src = static_cast<size_t>(id) * cols, psrc = static_cast<size_t>(r) * cols;
  float* o = out + static_cast<size_t>(row) * cols;
  for (int c = lane_id(); c < cols; c += 32) o[c] = ld_any(table, dt, src + c) + ld_any(pair, pdt, psrc + c);
}

__global__ void __launch_bounds__(kRowThreads)
add_row_vector_kernel(float* __restrict__ x, const void* __restrict__ vec, int dt, size_t total, int cols) {
  for (size_t i = blockIdx.x * static_cast<size_t>(kRowThreads) + threadIdx.x; i < total;
       i += static_cast<size_t>(gridDim.x) * kRowThreads)
    x[i] += ld_any(vec, dt, i % cols);
}

// x += mult * (a + sum_j part_j): the sum runs in a fixed order (a first, then the partials by index)
__global__ void __launch_bounds__(kRowThreads)
residual_add_rows_kernel(float* __restrict__ x, const void* __restrict__ a, int a_dt, int64_t lda,
                         const void* __restrict__ part, int p_dt, int64_t ldp, int np, float mult,
                         void* __restrict__ copy, int c_dt, int rows, int cols) {
  const size_t total = static_cast<size_t>(rows) * cols;
  for (size_t i = blockIdx.x * static_cast<size_t>(kRowThreads) + threadIdx.x; i < total;
       i += static_cast<size_t>(gridDim.x) * kRowThreads) {
    const size_t r = i / cols, c = i % cols;
    float y = a ? ld_any(a, a_dt, r * lda + c) : 0.f;
    if (part)
      for (int j = 0; j < np; ++j) y += ld_any(part, p_dt, (r * np + j) * ldp + c);
    const float v = x[i] + mult * y;
    x[i] = v;
    if (copy) st_any(copy, c_dt, i, v);
  }
}

__global__ void __launch_bounds__(kRowThreads)
gelu_mul_gather_kernel(const void* __restrict__ z, int z_dt, const void* __restrict__ table, int dt, int64_t ldt,
                       const int32_t* __restrict__ ids, int col0, void* __restrict__ out, int o_dt, int rows,
                       int cols) {
  const size_t total = static_cast<size_t>(rows) * cols;
  for (size_t i = blockIdx.x * static_cast<size_t>(kRowThreads) + threadIdx.x; i < total;
       i += static_cast<size_t>(gridDim.x) * kRowThreads) {
    const size_t r = i / cols, c = i % cols;
    const float v = ld_any(z, z_dt, i);
    const float g = 0.5f * v * (1.0f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)));
    st_any(out, o_dt, i, g * ld_any(table, dt, static_cast<size_t>(ids[r]) * ldt + col0 + c));
  }
}

// ---- sigmoid / softmax router with group-limited choice ----------------------------------------------
// Logits in fp32 dot products over the row.  Then one warp per token: scores s = sigmoid(z) or softmax(z);
// choice c = s + correction; group score = the largest c of the group or the sum of its two largest; the
// `keep` best groups stay, the others' c become -inf; `top` rounds of arg-max over c (ties: lower index);
// the weight of a chosen expert is scale * s.
__device__ __forceinline__ void warp_argmax(float& best, int& bi) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, best, o);
    const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
    if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
  }
}

// four consecutive elements (16-byte aligned fp32, 8-byte aligned bf16)
__device__ __forceinline__ float4 ld4_any(const void* p, int dt, size_t i) {
  if (dt) return *reinterpret_cast<const float4*>(static_cast<const float*>(p) + i);
  const uint2 u = *reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(p) + i);
  return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16),
                     __uint_as_float(u.y & 0xffff0000u));
}
__device__ __forceinline__ void st4_any(void* p, int dt, size_t i, float4 v) {
  if (dt) {
    *reinterpret_cast<float4*>(static_cast<float*>(p) + i) = v;
    return;
  }
  __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<unsigned int*>(&lo);
  u.y = *reinterpret_cast<unsigned int*>(&hi);
  *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(p) + i) = u;
}

// A CTA takes NT tokens; its warps split the outputs, four at a time and for all the tokens (every weight is read once per
// CTA, the dot products overlap); the shared expert's gate, if there is one, is the output after the last.  Then a warp
// per token chooses.  A token's sums run in the same order whatever NT is.
template <int NT, int THREADS, bool VEC>
__global__ void __launch_bounds__(THREADS) moe_route_scores_kernel(const vila_moe_route_params p) {
  extern __shared__ float z_s[];  // per token: s [experts] | c [experts] | group score [groups]
  const int wid = threadIdx.x >> 5, lane = lane_id(), row0 = blockIdx.x * NT;
  const int experts = p.experts, groups = p.groups, keep = p.keep, cols = p.cols, per_tok = 2 * experts + groups;
  const int outs = experts + (p.gate_w ? 1 : 0);
  size_t xb[NT];
#pragma unroll
  for (int t = 0; t < NT; ++t) xb[t] = static_cast<size_t>(min(row0 + t, p.rows - 1)) * p.ldx;
  for (int e0 = 4 * wid; e0 < outs; e0 += 4 * (THREADS / 32)) {
    const float* we[4];
    float a[NT][4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int e = min(e0 + u, outs - 1);
      we[u] = e < experts ? p.w + static_cast<size_t>(e) * cols : p.gate_w;
#pragma unroll
      for (int t = 0; t < NT; ++t) a[t][u] = 0.f;
    }
    if (VEC) {
#pragma unroll 2
      for (int k = 4 * lane; k < cols; k += 128) {
        float4 wv[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) wv[u] = __ldg(reinterpret_cast<const float4*>(we[u] + k));
#pragma unroll
        for (int t = 0; t < NT; ++t) {
          const float4 xv = ld4_any(p.x, p.x_dtype, xb[t] + k);
#pragma unroll
          for (int u = 0; u < 4; ++u) {
            a[t][u] = fmaf(xv.x, wv[u].x, a[t][u]); a[t][u] = fmaf(xv.y, wv[u].y, a[t][u]);
            a[t][u] = fmaf(xv.z, wv[u].z, a[t][u]); a[t][u] = fmaf(xv.w, wv[u].w, a[t][u]);
          }
        }
      }
    } else {
      for (int k = lane; k < cols; k += 32) {
#pragma unroll
        for (int t = 0; t < NT; ++t) {
          const float xv = ld_any(p.x, p.x_dtype, xb[t] + k);
#pragma unroll
          for (int u = 0; u < 4; ++u) a[t][u] = fmaf(xv, we[u][k], a[t][u]);
        }
      }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1)
#pragma unroll
      for (int t = 0; t < NT; ++t)
#pragma unroll
        for (int u = 0; u < 4; ++u) a[t][u] += __shfl_xor_sync(0xffffffffu, a[t][u], o);
    if (lane == 0) {
#pragma unroll
      for (int t = 0; t < NT; ++t)
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const int e = e0 + u;
          if (e < experts) z_s[t * per_tok + e] = a[t][u];
          else if (e < outs && row0 + t < p.rows) p.gate[row0 + t] = sigmoid_f(a[t][u]);
        }
    }
  }
  __syncthreads();
  const int row = row0 + wid;
  if (wid >= NT || row >= p.rows) return;
  float* s = z_s + wid * per_tok;
  float* c = s + experts;
  float* gs = c + experts;
  float mx = 0.f, inv = 1.f;
  if (p.score == VILA_SCORE_SOFTMAX) {
    mx = -INFINITY;
    for (int e = lane; e < experts; e += 32) mx = fmaxf(mx, s[e]);
    mx = warp_max(mx);
    float sum = 0.f;
    for (int e = lane; e < experts; e += 32) sum += expf(s[e] - mx);
    inv = 1.0f / warp_sum(sum);
  }
  for (int e = lane; e < experts; e += 32) {   // a lane rewrites the entries that it read
    const float sv = p.score == VILA_SCORE_SOFTMAX ? expf(s[e] - mx) * inv : sigmoid_f(s[e]);
    s[e] = sv;
    c[e] = sv + (p.correction ? p.correction[e] : 0.f);
  }
  __syncwarp();
  const int gsize = experts / groups;
  if (keep < groups) {
    for (int g = lane; g < groups; g += 32) {
      float a = -INFINITY, b = -INFINITY;   // largest, second largest
      for (int e = g * gsize; e < (g + 1) * gsize; ++e) {
        const float v = c[e];
        if (v > a) { b = a; a = v; }
        else if (v > b) b = v;
      }
      gs[g] = (p.group_top >= 2 && gsize >= 2) ? a + b : a;
    }
    __syncwarp();
    // `keep` rounds of arg-max over the groups; a kept group is marked by +inf
    for (int j = 0; j < keep; ++j) {
      float best = -INFINITY;
      int bi = 0x7fffffff;
      for (int g = lane; g < groups; g += 32) {
        const float v = gs[g];
        if (v != INFINITY && v > best) { best = v; bi = g; }
      }
      warp_argmax(best, bi);
      if (lane == 0 && bi != 0x7fffffff) gs[bi] = INFINITY;
      __syncwarp();
    }
    for (int e = lane; e < experts; e += 32)
      if (gs[e / gsize] != INFINITY) c[e] = -INFINITY;
    __syncwarp();
  }
  for (int j = 0; j < p.top; ++j) {
    float best = -INFINITY;
    int bi = 0x7fffffff;
    for (int e = lane; e < experts; e += 32) {
      const float v = c[e];
      if (v > best) { best = v; bi = e; }
    }
    warp_argmax(best, bi);
    if (bi == 0x7fffffff) bi = 0;   // fewer selectable experts than `top` (refused by the launcher's callers)
    if (lane == 0) {
      p.idx[static_cast<size_t>(row) * p.top + j] = bi;
      p.weight[static_cast<size_t>(row) * p.top + j] = p.scale * s[bi];
      c[bi] = -INFINITY;
    }
    __syncwarp();
  }
}

inline int flat_grid(size_t total) {
  const size_t g = (total + kRowThreads - 1) / kRowThreads;
  return static_cast<int>(g < 1 ? 1 : (g > 148 * 16 ? 148 * 16 : g));
}

// ---- scaled embedding + sinusoidal positions ---------------------------------------------------------
// A warp (narrow rows) or a CTA (wide rows) per row; a thread takes column pairs (2i, 2i + 1) = (sin, cos) of ONE
// angle position * inv_freq[i].
// The angle is formed and brought into [-pi, pi] in double, so that far positions keep their phase (an fp32
// product loses it); sine and cosine of the reduced angle are evaluated in fp32.
template <int TPR>
__global__ void __launch_bounds__(kRowThreads)
embed_sincos_rows_kernel(const void* __restrict__ table, int dt, const int32_t* __restrict__ ids,
                         const int32_t* __restrict__ positions, const double* __restrict__ inv_freq, float scale,
                         float* __restrict__ out, void* __restrict__ copy, int c_dt, int rows, int cols) {
  const int row = row_of<TPR>();
  if (row >= rows) return;
  const size_t src = static_cast<size_t>(ids[row]) * cols, dst = static_cast<size_t>(row) * cols;
  const double pos = static_cast<double>(positions[row]);
  for (int i = col0_of<TPR>(); 2 * i < cols; i += TPR) {
    const double ang = pos * inv_freq[i];
    const float red = static_cast<float>(fma(-6.283185307179586476925, rint(ang * 0.15915494309189533577), ang));
    float sn, cs;
    sincosf(red, &sn, &cs);
    const float v0 = fmaf(ld_any(table, dt, src + 2 * i), scale, sn);
    out[dst + 2 * i] = v0;
    if (copy) st_any(copy, c_dt, dst + 2 * i, v0);
    if (2 * i + 1 < cols) {
      const float v1 = fmaf(ld_any(table, dt, src + 2 * i + 1), scale, cs);
      out[dst + 2 * i + 1] = v1;
      if (copy) st_any(copy, c_dt, dst + 2 * i + 1, v1);
    }
  }
}

// ---- post-normed residual update of one or two scaled branches ---------------------------------------
// x += rms(sa * a + sb * b) * w  (the norm sits on the sublayer's OUTPUT); optionally the updated row is
// also written in the dtype of the next projection's operand.
template <int TPR>
__global__ void __launch_bounds__(kRowThreads)
branch_norm_residual_kernel(float* __restrict__ x, const void* __restrict__ a, int a_dt, int64_t lda, float sa,
                            const void* __restrict__ b, int b_dt, int64_t ldb, float sb,
                            const void* __restrict__ w, int w_dt, float eps, void* __restrict__ copy, int c_dt,
                            int rows, int cols) {
  __shared__ float red[kRowsPerCta];
  const int row = row_of<TPR>();
  if (row >= rows) return;
  const size_t ab = static_cast<size_t>(row) * lda, bb = static_cast<size_t>(row) * ldb;
  float ss = 0.f;
  for (int c = col0_of<TPR>(); c < cols; c += TPR) {
    float y = sa * ld_any(a, a_dt, ab + c);
    if (b) y = fmaf(sb, ld_any(b, b_dt, bb + c), y);
    ss = fmaf(y, y, ss);
  }
  ss = row_sum<TPR>(ss, red);
  const float r = 1.0f / sqrtf(ss / static_cast<float>(cols) + eps);
  const size_t xb = static_cast<size_t>(row) * cols;
  for (int c = col0_of<TPR>(); c < cols; c += TPR) {
    float y = sa * ld_any(a, a_dt, ab + c);
    if (b) y = fmaf(sb, ld_any(b, b_dt, bb + c), y);
    const float v = x[xb + c] + y * r * (w ? ld_any(w, w_dt, c) : 1.0f);
    x[xb + c] = v;
    if (copy) st_any(copy, c_dt, xb + c, v);
  }
}

// ---- parallel-sublayer residual with per-channel scales ------------------------------------------------
// x += sa * a + sb * b (element by element; sa / sb one vector each, b may be missing), then, if out is given,
// out = x / sqrt(mean(x^2) + eps) * w: the operand of both sublayers of the next layer.  The vector form keeps
// the row in registers between the sum and the norm.
struct ScaledResidual {
  float* x;
  const void *a, *b;
  int64_t lda, ldb;
  const float *sa, *sb, *w;
  void* out;
  int a_dt, b_dt, o_dt, rows, cols;
  float eps;
};

template <int TPR>
__global__ void __launch_bounds__(kRowThreads) scaled_residual_norm_kernel(const ScaledResidual p) {
  __shared__ float red[kRowsPerCta];
  const int row = row_of<TPR>();
  if (row >= p.rows) return;
  float* xr = p.x + static_cast<size_t>(row) * p.cols;
  const size_t ab = static_cast<size_t>(row) * p.lda, bb = static_cast<size_t>(row) * p.ldb;
  float ss = 0.f;
  for (int c = col0_of<TPR>(); c < p.cols; c += TPR) {
    float y = p.sa[c] * ld_any(p.a, p.a_dt, ab + c);
    if (p.b) y = fmaf(p.sb[c], ld_any(p.b, p.b_dt, bb + c), y);
    const float v = xr[c] + y;
    xr[c] = v;
    ss = fmaf(v, v, ss);
  }
  if (!p.out) return;
  ss = row_sum<TPR>(ss, red);
  const float r = 1.0f / sqrtf(ss / static_cast<float>(p.cols) + p.eps);
  for (int c = col0_of<TPR>(); c < p.cols; c += TPR)
    st_any(p.out, p.o_dt, static_cast<size_t>(row) * p.cols + c, xr[c] * r * (p.w ? p.w[c] : 1.0f));
}

template <int TPR, int NV>   // cols <= 4 * TPR * NV, a multiple of 4, all rows aligned
__global__ void __launch_bounds__(kRowThreads) scaled_residual_norm_vec_kernel(const ScaledResidual p) {
  __shared__ float red[kRowsPerCta];
  const int row = row_of<TPR>();
  if (row >= p.rows) return;
  float* xr = p.x + static_cast<size_t>(row) * p.cols;
  const size_t ab = static_cast<size_t>(row) * p.lda, bb = static_cast<size_t>(row) * p.ldb;
  float4 v[NV];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int c = 4 * (col0_of<TPR>() + TPR * k);
    v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < p.cols) {
      const float4 x4 = *reinterpret_cast<const float4*>(xr + c), a4 = ld4_any(p.a, p.a_dt, ab + c);
      const float4 s4 = __ldg(reinterpret_cast<const float4*>(p.sa + c));
      float4 y = make_float4(s4.x * a4.x, s4.y * a4.y, s4.z * a4.z, s4.w * a4.w);
      if (p.b) {
        const float4 b4 = ld4_any(p.b, p.b_dt, bb + c), t4 = __ldg(reinterpret_cast<const float4*>(p.sb + c));
        y.x = fmaf(t4.x, b4.x, y.x); y.y = fmaf(t4.y, b4.y, y.y); y.z = fmaf(t4.z, b4.z, y.z); y.w = fmaf(t4.w, b4.w, y.w);
      }
      v[k] = make_float4(x4.x + y.x, x4.y + y.y, x4.z + y.z, x4.w + y.w);
      *reinterpret_cast<float4*>(xr + c) = v[k];
    }
    ss = fmaf(v[k].x, v[k].x, ss); ss = fmaf(v[k].y, v[k].y, ss);
    ss = fmaf(v[k].z, v[k].z, ss); ss = fmaf(v[k].w, v[k].w, ss);
  }
  if (!p.out) return;
  ss = row_sum<TPR>(ss, red);
  const float r = 1.0f / sqrtf(ss / static_cast<float>(p.cols) + p.eps);
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int c = 4 * (col0_of<TPR>() + TPR * k);
    if (c < p.cols) {
      float4 w4 = make_float4(1.f, 1.f, 1.f, 1.f);
      if (p.w) w4 = __ldg(reinterpret_cast<const float4*>(p.w + c));
      st4_any(p.out, p.o_dt, static_cast<size_t>(row) * p.cols + c,
              make_float4(v[k].x * r * w4.x, v[k].y * r * w4.y, v[k].z * r * w4.z, v[k].w * r * w4.w));
    }
  }
}

// ---- read-out of a recurrent mixer: per-head RMS norm, shared weight, gate -----------------------------------
// out[t, h, :] = o[t, h, :] / sqrt(mean(o[t, h, :]^2) + eps) * w * act(gate[t, h, :]), act = SiLU or sigmoid; a warp per
// (token, head), or a CTA where a head is wide
template <int TPR, bool VEC>
__global__ void __launch_bounds__(kRowThreads)
gated_head_norm_kernel(const float* __restrict__ o, const float* __restrict__ w, const void* __restrict__ gate, int g_dt,
                       int64_t ldg, float eps, void* __restrict__ out, int o_dt, int pairs, int H, int vdim, int gate_act) {
  __shared__ float red[kRowsPerCta];
  const int pair = row_of<TPR>();
  if (pair >= pairs) return;
  const int t = pair / H, h = pair - t * H, l = col0_of<TPR>();
  const size_t ob = static_cast<size_t>(pair) * vdim, gb = static_cast<size_t>(t) * ldg + static_cast<size_t>(h) * vdim;
  auto act = [&](float z) { return gate_act == VILA_ACT_SIGMOID ? sigmoid_f(z) : silu_exact_f(z); };
  float ss = 0.f;
  if (VEC) {
    for (int c = 4 * l; c < vdim; c += 4 * TPR) {
      const float4 v = *reinterpret_cast<const float4*>(o + ob + c);
      ss = fmaf(v.x, v.x, ss); ss = fmaf(v.y, v.y, ss); ss = fmaf(v.z, v.z, ss); ss = fmaf(v.w, v.w, ss);
    }
  } else {
    for (int c = l; c < vdim; c += TPR) ss = fmaf(o[ob + c], o[ob + c], ss);
  }
  ss = row_sum<TPR>(ss, red);
  const float r = 1.0f / sqrtf(ss / static_cast<float>(vdim) + eps);
  if (VEC) {
    for (int c = 4 * l; c < vdim; c += 4 * TPR) {
      const float4 v = *reinterpret_cast<const float4*>(o + ob + c), g = ld4_any(gate, g_dt, gb + c);
      const float4 w4 = __ldg(reinterpret_cast<const float4*>(w + c));
      st4_any(out, o_dt, ob + c, make_float4(v.x * r * w4.x * act(g.x), v.y * r * w4.y * act(g.y),
                                             v.z * r * w4.z * act(g.z), v.w * r * w4.w * act(g.w)));
    }
  } else {
    for (int c = l; c < vdim; c += TPR)
      st_any(out, o_dt, ob + c, o[ob + c] * r * w[c] * act(ld_any(gate, g_dt, gb + c)));
  }
}

// ---- parallel-sublayer residual + Dynamic Tanh norms (elementwise: nothing is reduced over the row) -----------
// x (or an embedding row) += mult * (sa * a + sb * (b * gate + routed partials, identity experts included)), then up to two
// norms tanh(alpha x) * w + bias of the result; V = 4 or 1 neighbouring columns per thread
template <int V>
struct Cols {
  float v[V];
};
template <int V>
__device__ __forceinline__ Cols<V> ldv(const void* p, int dt, size_t i) {
  Cols<V> r;
  if (V == 4) {
    const float4 u = ld4_any(p, dt, i);
    r.v[0] = u.x; r.v[V == 4 ? 1 : 0] = u.y; r.v[V == 4 ? 2 : 0] = u.z; r.v[V == 4 ? 3 : 0] = u.w;
  } else {
    r.v[0] = ld_any(p, dt, i);
  }
  return r;
}
template <int V>
__device__ __forceinline__ void stv(void* p, int dt, size_t i, const Cols<V>& c) {
  if (V == 4) st4_any(p, dt, i, make_float4(c.v[0], c.v[V == 4 ? 1 : 0], c.v[V == 4 ? 2 : 0], c.v[V == 4 ? 3 : 0]));
  else st_any(p, dt, i, c.v[0]);
}

template <int V>
__global__ void __launch_bounds__(kRowThreads) tanh_residual_kernel(const vila_tanh_residual_params p) {
  const int cv = p.cols / V;
  const size_t total = static_cast<size_t>(p.rows) * cv;
  for (size_t i = blockIdx.x * static_cast<size_t>(kRowThreads) + threadIdx.x; i < total;
       i += static_cast<size_t>(gridDim.x) * kRowThreads) {
    const int r = static_cast<int>(i / cv), c = static_cast<int>(i - static_cast<size_t>(r) * cv) * V;
    const size_t at = static_cast<size_t>(r) * p.cols + c;
    Cols<V> x = p.table ? ldv<V>(p.table, p.table_dtype, static_cast<size_t>(p.ids[r]) * p.cols + c) : ldv<V>(p.x, VILA_DT_F32, at);
    if (p.a) {
      const Cols<V> a = ldv<V>(p.a, p.a_dtype, static_cast<size_t>(r) * p.lda + c), sa = ldv<V>(p.a_scale, VILA_DT_F32, c);
      Cols<V> y;
#pragma unroll
      for (int k = 0; k < V; ++k) y.v[k] = sa.v[k] * a.v[k];
      if (p.b || p.part) {
        Cols<V> f;
#pragma unroll
        for (int k = 0; k < V; ++k) f.v[k] = 0.f;
        if (p.b) {
          const float g = p.b_gate ? p.b_gate[r] : 1.0f;
          const Cols<V> b = ldv<V>(p.b, p.b_dtype, static_cast<size_t>(r) * p.ldb + c);
#pragma unroll
          for (int k = 0; k < V; ++k) f.v[k] = g * b.v[k];
        }
        if (p.part) {
          const size_t pr = static_cast<size_t>(r) * p.n_partials;
          for (int j = 0; j < p.n_partials; ++j) {
            const bool self = p.idx != nullptr && p.idx[pr + j] >= p.experts;
            const float w = self ? p.weight[pr + j] : 1.0f;
            const Cols<V> q = self ? ldv<V>(p.h, p.h_dtype, static_cast<size_t>(r) * p.ldh + c)
                                   : ldv<V>(p.part, p.part_dtype, (pr + j) * p.ldp + c);
#pragma unroll
            for (int k = 0; k < V; ++k) f.v[k] = fmaf(w, q.v[k], f.v[k]);
          }
        }
        const Cols<V> sb = ldv<V>(p.b_scale, VILA_DT_F32, c);
#pragma unroll
        for (int k = 0; k < V; ++k) y.v[k] = fmaf(sb.v[k], f.v[k], y.v[k]);
      }
#pragma unroll
      for (int k = 0; k < V; ++k) x.v[k] = fmaf(p.mult, y.v[k], x.v[k]);
    }
    if (p.a || p.table) stv<V>(p.x, VILA_DT_F32, at, x);
#pragma unroll
    for (int o = 0; o < 2; ++o) {
      if (o < p.n_out) {
        const Cols<V> w = ldv<V>(p.w[o], VILA_DT_F32, c), b = ldv<V>(p.bias[o], VILA_DT_F32, c);
        Cols<V> n;
#pragma unroll
        for (int k = 0; k < V; ++k) n.v[k] = fmaf(tanhf(p.alpha[o] * x.v[k]), w.v[k], b.v[k]);
        stv<V>(p.out[o], p.out_dtype, at, n);
      }
    }
  }
}

inline bool aligned_to(const void* p, size_t n) { return reinterpret_cast<uintptr_t>(p) % n == 0; }
// rows of a [.., ld] tensor that start on a four-element boundary (8 bytes bf16, 16 bytes fp32)
inline bool rows4(const void* p, int64_t ld, int dt) { return ld % 4 == 0 && aligned_to(p, dt ? 16 : 8); }

}  // namespace

int scaled_residual_norm_rows(float* x, const void* a, int a_dt, int64_t lda, const float* sa, const void* b, int b_dt,
                              int64_t ldb, const float* sb, const float* w, float eps, void* out, int o_dt, int rows,
                              int cols, cudaStream_t stream) {
  if (rows <= 0) return 0;
  VB_CHECK(cols > 0 && a != nullptr && sa != nullptr && (b == nullptr || sb != nullptr), "scaled_residual_norm_rows: cols=%d", cols);
  const ScaledResidual p = {x, a, b, lda, ldb, sa, sb, w, out, a_dt, b_dt, o_dt, rows, cols, eps};
  const bool vec = cols % 4 == 0 && aligned_to(x, 16) && aligned_to(sa, 16) && rows4(a, lda, a_dt) &&
                   (b == nullptr || (rows4(b, ldb, b_dt) && aligned_to(sb, 16))) && (w == nullptr || aligned_to(w, 16)) &&
                   (out == nullptr || aligned_to(out, o_dt ? 16 : 8));
#define VB_SRN(K, G) VB_CUDA(launch_serial(K, dim3(G), dim3(kRowThreads), 0, stream, p))
  if (cols >= kWideCols) {
    if (vec && cols <= 1024) VB_SRN((scaled_residual_norm_vec_kernel<256, 1>), rows);
    else if (vec && cols <= 2048) VB_SRN((scaled_residual_norm_vec_kernel<256, 2>), rows);
    else if (vec && cols <= 4096) VB_SRN((scaled_residual_norm_vec_kernel<256, 4>), rows);
    else if (vec && cols <= 8192) VB_SRN((scaled_residual_norm_vec_kernel<256, 8>), rows);
    else VB_SRN(scaled_residual_norm_kernel<256>, rows);
  } else if (vec) {
    VB_SRN((scaled_residual_norm_vec_kernel<32, 4>), row_grid(rows));
  } else {
    VB_SRN(scaled_residual_norm_kernel<32>, row_grid(rows));
  }
#undef VB_SRN
  return 0;
}

int gated_head_norm_rows(const float* o, const float* w, const void* gate, int g_dt, int64_t ldg, float eps, void* out,
                         int o_dt, int rows, int H, int vdim, int gate_act, cudaStream_t stream) {
  if (rows <= 0) return 0;
  VB_CHECK(H >= 1 && vdim >= 1 && w != nullptr && gate != nullptr, "gated_head_norm_rows: H=%d vdim=%d", H, vdim);
  VB_CHECK(static_cast<long>(rows) * H < (1L << 31), "gated_head_norm_rows: rows=%d H=%d", rows, H);
  VB_CHECK(gate_act == VILA_ACT_SILU || gate_act == VILA_ACT_SIGMOID, "gated_head_norm_rows: gate activation %d", gate_act);
  const int pairs = rows * H;
  const bool vec = vdim % 4 == 0 && aligned_to(o, 16) && aligned_to(w, 16) && rows4(gate, ldg, g_dt) && aligned_to(out, o_dt ? 16 : 8);
#define VB_GHN(K, G)                                                                                                      \
  VB_CUDA(launch_serial(K, dim3(G), dim3(kRowThreads), 0, stream, o, w, gate, g_dt, ldg, eps, out, o_dt, pairs, H, vdim, gate_act))
  if (vdim >= kWideCols) {
    if (vec) VB_GHN((gated_head_norm_kernel<256, true>), pairs);
    else VB_GHN((gated_head_norm_kernel<256, false>), pairs);
  } else if (vec) {
    VB_GHN((gated_head_norm_kernel<32, true>), row_grid(pairs));
  } else {
    VB_GHN((gated_head_norm_kernel<32, false>), row_grid(pairs));
  }
#undef VB_GHN
  return 0;
}

int tanh_residual_rows(const vila_tanh_residual_params& p, cudaStream_t stream) {
  if (p.rows <= 0) return 0;
  VB_CHECK(p.cols > 0 && p.x != nullptr && p.n_out >= 0 && p.n_out <= 2 && (p.table == nullptr || p.ids != nullptr),
           "tanh_residual_rows: cols=%d n_out=%d", p.cols, p.n_out);
  VB_CHECK((p.a == nullptr || p.a_scale != nullptr) && ((p.b == nullptr && p.part == nullptr) || (p.a != nullptr && p.b_scale != nullptr)),
           "tanh_residual_rows: a branch without its scale, or a second branch without the first");
  VB_CHECK(p.part == nullptr || (p.n_partials >= 1 && (p.idx == nullptr || (p.weight != nullptr && p.h != nullptr))),
           "tanh_residual_rows: n_partials=%d; indices need weights and the experts' input", p.n_partials);
  bool vec = p.cols % 4 == 0 && aligned_to(p.x, 16) && (!p.table || aligned_to(p.table, p.table_dtype ? 16 : 8)) &&
             (!p.a || (rows4(p.a, p.lda, p.a_dtype) && aligned_to(p.a_scale, 16))) && (!p.b || rows4(p.b, p.ldb, p.b_dtype)) &&
             (!p.part || rows4(p.part, p.ldp, p.part_dtype)) && (!p.h || rows4(p.h, p.ldh, p.h_dtype)) &&
             (!p.b_scale || aligned_to(p.b_scale, 16));
  for (int k = 0; k < p.n_out; ++k) {
    VB_CHECK(p.w[k] != nullptr && p.bias[k] != nullptr && p.out[k] != nullptr, "tanh_residual_rows: norm %d is incomplete", k);
    vec = vec && aligned_to(p.w[k], 16) && aligned_to(p.bias[k], 16) && aligned_to(p.out[k], p.out_dtype ? 16 : 8);
  }
  const size_t total = static_cast<size_t>(p.rows) * (vec ? p.cols / 4 : p.cols);
  if (vec) VB_CUDA(launch_serial(tanh_residual_kernel<4>, dim3(flat_grid(total)), dim3(kRowThreads), 0, stream, p));
  else VB_CUDA(launch_serial(tanh_residual_kernel<1>, dim3(flat_grid(total)), dim3(kRowThreads), 0, stream, p));
  return 0;
}

int embed_rows(const void* table, int dt, const int32_t* ids, float* out, int rows, int cols,
               cudaStream_t stream) {
  if (rows <= 0) return 0;
  VB_CUDA(launch_serial(embed_rows_kernel, dim3(row_grid(rows)), dim3(kRowThreads), 0, stream, table, dt,
                     ids, out, rows, cols));
  return 0;
}

int rmsnorm_rows(const void* x, int x_dt, int64_t ldx, const void* w, int w_dt, float w_off, float eps,
                 void* out, int o_dt, int64_t ldo, const int32_t* out_rows, int rows, int cols,
                 cudaStream_t stream, int groups) {
  if (rows <= 0) return 0;
  VB_CHECK(cols > 0 && groups >= 1 && cols % groups == 0, "rmsnorm_rows: cols=%d groups=%d", cols, groups);
  const int vrows = rows * groups, vcols = cols / groups;
  if (vcols >= kWideCols)
    VB_CUDA(launch_serial(rmsnorm_rows_kernel<256>, dim3(vrows), dim3(kRowThreads), 0, stream, x, x_dt, ldx, w,
                       w_dt, w_off, eps, out, o_dt, ldo, out_rows, vrows, vcols, groups));
  else
    VB_CUDA(launch_serial(rmsnorm_rows_kernel<32>, dim3(row_grid(vrows)), dim3(kRowThreads), 0, stream, x, x_dt,
                       ldx, w, w_dt, w_off, eps, out, o_dt, ldo, out_rows, vrows, vcols, groups));
  return 0;
}

int residual_norm_rows(float* x, const void* a, int a_dt, int64_t lda, const void* part, int p_dt, int64_t ldp, int np,
                       const void* w, int w_dt, float eps, void* out, int o_dt, int rows, int cols, cudaStream_t stream) {
  if (rows <= 0) return 0;
  VB_CHECK(cols > 0 && out != nullptr && (part == nullptr || np >= 1), "residual_norm_rows: cols=%d n_partials=%d", cols, np);
  if (cols >= kWideCols)
    VB_CUDA(launch_serial(residual_norm_rows_kernel<256>, dim3(rows), dim3(kRowThreads), 0, stream, x, a, a_dt, lda,
                          part, p_dt, ldp, np, w, w_dt, eps, out, o_dt, rows, cols));
  else
    VB_CUDA(launch_serial(residual_norm_rows_kernel<32>, dim3(row_grid(rows)), dim3(kRowThreads), 0, stream, x, a,
                          a_dt, lda, part, p_dt, ldp, np, w, w_dt, eps, out, o_dt, rows, cols));
  return 0;
}

int gated_norm_residual(float* x, const void* part, int p_dt, int64_t ldp, int np, const void* gate,
                        int g_dt, int64_t ldg, const void* gb, int b_dt, const void* w, int w_dt,
                        float w_off, float eps, int rows, int cols, cudaStream_t stream, float mult) {
  if (rows <= 0) return 0;
  VB_CHECK(np >= 1 && cols > 0, "gated_norm_residual: n_partials=%d cols=%d", np, cols);
  if (cols >= kWideCols)
    VB_CUDA(launch_serial(gated_norm_residual_kernel<256>, dim3(rows), dim3(kRowThreads), 0, stream, x, part,
                       p_dt, ldp, np, gate, g_dt, ldg, gb, b_dt, w, w_dt, w_off, eps, mult, rows, cols));
  else
    VB_CUDA(launch_serial(gated_norm_residual_kernel<32>, dim3(row_grid(rows)), dim3(kRowThreads), 0, stream, x,
                       part, p_dt, ldp, np, gate, g_dt, ldg, gb, b_dt, w, w_dt, w_off, eps, mult, rows, cols));
  return 0;
}

int moe_route(const void* x, int x_dt, int64_t ldx, const float* wr, const float* bias, int32_t* idx,
              float* weight, int rows, int cols, int experts, int top, cudaStream_t stream) {
  if (rows <= 0) return 0;
  VB_CHECK(experts >= 1 && top >= 1 && top <= experts && experts <= 1024,
           "moe_route: experts=%d top=%d", experts, top);
  if (rows <= 1024)   // few tokens: a CTA per token, its warps split the experts
    VB_CUDA(launch_serial(moe_route_kernel<256>, dim3(rows), dim3(kRowThreads), sizeof(float) * experts, stream,
                       x, x_dt, ldx, wr, bias, idx, weight, rows, cols, experts, top));
  else
    VB_CUDA(launch_serial(moe_route_kernel<32>, dim3(row_grid(rows)), dim3(kRowThreads),
                       sizeof(float) * kRowsPerCta * experts, stream, x, x_dt, ldx, wr, bias, idx, weight, rows,
                       cols, experts, top));
  return 0;
}


int embed_pair_rows(const void* table, int dt, const void* pair, int pdt, const int32_t* ids,
                    const int32_t* prev, long long mul_prev, long long mul_cur, long long buckets, float* out,
                    int rows, int cols, cudaStream_t stream) {
  if (rows <= 0) return 0;
  VB_CHECK(buckets >= 1 && cols > 0, "embed_pair_rows: buckets=%lld cols=%d", buckets, cols);
  VB_CUDA(launch_serial(embed_pair_rows_kernel, dim3(row_grid(rows)), dim3(kRowThreads), 0, stream, table, dt,
                        pair, pdt, ids, prev, mul_prev, mul_cur, buckets, out, rows, cols));
  return 0;
}

int add_row_vector(float* x, const void* vec, int dt, int rows, int cols, cudaStream_t stream) {
  if (rows <= 0 || cols <= 0) return 0;
  const size_t total = static_cast<size_t>(rows) * cols;
  VB_CUDA(launch_serial(add_row_vector_kernel, dim3(flat_grid(total)), dim3(kRowThreads), 0, stream, x, vec, dt,
                        total, cols));
  return 0;
}

int residual_add_rows(float* x, const void* a, int a_dt, int64_t lda, const void* part, int p_dt, int64_t ldp,
                      int np, float mult, void* copy, int c_dt, int rows, int cols, cudaStream_t stream) {
  if (rows <= 0 || cols <= 0) return 0;
  VB_CHECK(part == nullptr || np >= 1, "residual_add_rows: n_partials=%d", np);
  VB_CUDA(launch_serial(residual_add_rows_kernel, dim3(flat_grid(static_cast<size_t>(rows) * cols)),
                        dim3(kRowThreads), 0, stream, x, a, a_dt, lda, part, p_dt, ldp, np, mult, copy, c_dt, rows, cols));
  return 0;
}

int gelu_mul_gather(const void* z, int z_dt, const void* table, int dt, int64_t ldt, const int32_t* ids, int col0,
                    void* out, int o_dt, int rows, int cols, cudaStream_t stream) {
  if (rows <= 0 || cols <= 0) return 0;
  VB_CUDA(launch_serial(gelu_mul_gather_kernel, dim3(flat_grid(static_cast<size_t>(rows) * cols)),
                        dim3(kRowThreads), 0, stream, z, z_dt, table, dt, ldt, ids, col0, out, o_dt, rows, cols));
  return 0;
}

int moe_route_scores(const vila_moe_route_params& p, cudaStream_t stream) {
  if (p.rows <= 0) return 0;
  VB_CHECK(p.experts >= 1 && p.experts <= 1024 && p.groups >= 1 && p.experts % p.groups == 0 && p.keep >= 1 &&
               p.keep <= p.groups && p.top >= 1 && p.top <= p.keep * (p.experts / p.groups),
           "moe_route_scores: experts=%d top=%d groups=%d keep=%d", p.experts, p.top, p.groups, p.keep);
  VB_CHECK((p.score == VILA_SCORE_SIGMOID || p.score == VILA_SCORE_SOFTMAX) && (p.group_top == 1 || p.group_top == 2) &&
               (p.gate_w == nullptr || p.gate != nullptr),
           "moe_route_scores: score=%d group_top=%d", p.score, p.group_top);
  const size_t per_tok = sizeof(float) * (2 * p.experts + p.groups);
  const bool vec = p.cols % 4 == 0 && rows4(p.x, p.ldx, p.x_dtype) && aligned_to(p.w, 16) && (!p.gate_w || aligned_to(p.gate_w, 16));
#define VB_ROUTE(NT, TH, VEC)                                                                                       \
  VB_CUDA(launch_serial(moe_route_scores_kernel<NT, TH, VEC>, dim3((p.rows + NT - 1) / NT), dim3(TH), NT * per_tok, \
                        stream, p))
  if (p.rows <= 256 || 4 * per_tok > 48 * 1024) {   // few tokens (or very many experts): one per CTA of 32 warps
    if (vec) VB_ROUTE(1, 1024, true);
    else VB_ROUTE(1, 1024, false);
  } else {
    if (vec) VB_ROUTE(4, 256, true);
    else VB_ROUTE(4, 256, false);
  }
#undef VB_ROUTE
  return 0;
}

int moe_group(const int32_t* idx, int32_t* seg, int32_t* sorted, int pairs, int experts,
              cudaStream_t stream) {
  VB_CHECK(experts >= 1 && experts <= 8192 && pairs >= 0, "moe_group: experts=%d pairs=%d", experts, pairs);
  VB_CUDA(launch_serial(moe_group_kernel, dim3(1), dim3(1024), sizeof(int) * (experts + 1), stream, idx, seg,
                     sorted, pairs, experts));
  return 0;
}

int embed_sincos_rows(const void* table, int dt, const int32_t* ids, const int32_t* positions, const double* inv_freq,
                      float scale, float* out, void* copy, int c_dt, int rows, int cols, cudaStream_t stream) {
  if (rows <= 0) return 0;
  VB_CHECK(cols >= 1 && inv_freq != nullptr && positions != nullptr, "embed_sincos_rows: cols=%d", cols);
  if (cols >= kWideCols)
    VB_CUDA(launch_serial(embed_sincos_rows_kernel<256>, dim3(rows), dim3(kRowThreads), 0, stream, table, dt, ids,
                          positions, inv_freq, scale, out, copy, c_dt, rows, cols));
  else
    VB_CUDA(launch_serial(embed_sincos_rows_kernel<32>, dim3(row_grid(rows)), dim3(kRowThreads), 0, stream, table, dt,
                          ids, positions, inv_freq, scale, out, copy, c_dt, rows, cols));
  return 0;
}

int branch_norm_residual(float* x, const void* a, int a_dt, int64_t lda, float sa, const void* b, int b_dt,
                         int64_t ldb, float sb, const void* w, int w_dt, float eps, void* copy, int c_dt, int rows,
                         int cols, cudaStream_t stream) {
  if (rows <= 0) return 0;
  VB_CHECK(cols > 0 && a != nullptr, "branch_norm_residual: cols=%d", cols);
  if (cols >= kWideCols)
    VB_CUDA(launch_serial(branch_norm_residual_kernel<256>, dim3(rows), dim3(kRowThreads), 0, stream, x, a, a_dt, lda,
                          sa, b, b_dt, ldb, sb, w, w_dt, eps, copy, c_dt, rows, cols));
  else
    VB_CUDA(launch_serial(branch_norm_residual_kernel<32>, dim3(row_grid(rows)), dim3(kRowThreads), 0, stream, x, a,
                          a_dt, lda, sa, b, b_dt, ldb, sb, w, w_dt, eps, copy, c_dt, rows, cols));
  return 0;
}

}  // namespace vb
