// Recurrences over an outer-product state S [dim, vdim] per head on ragged batches (fp32 state in a slot of a
// caller-owned pool; a sequence at position 0 starts from zero and never reads its slot):
//
//   delta_scan   gated delta rule, one decay g and one step size beta per head and token:
//                  S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//                q and k are made unit vectors first (q also times q_scale), g = exp(-exp(A_log) softplus(a + dt_bias)),
//                beta = sigmoid(b); head h uses q / k head h / (H / G)
//   gla_scan     gated linear attention, one decay per key channel and token:
//                  S <- diag(alpha) S + k v^T;  o = S^T (q_scale q),   alpha = sigmoid(z + z_bias)^(1 / tau)
//   decay_scan   linear attention with one constant decay per head (lightning attention):
//                  S <- g S + k v^T;  o = S^T (q_scale q);  optionally SiLU on q, k and v as they are read
//
// The read-outs are taken from the state BEFORE the token's write, which is the same number and shortens the chain
// of dependent steps to one pass over the state per token:
//   delta:  S_new^T q = g (S^T q) + (k . q) u        so S^T k and S^T q are reduced together
//   gla:    S_new^T q = S^T (alpha q) + (k . q) v    so the state update does not wait for the reduction
//   decay:  S_new^T q = g (S^T q) + (k . q) v        likewise
//
// Grid (sequence, head, COLS columns of vdim).  Warps 0-3 own the state: R lanes share CPT columns, lane r
// keeps the float4 pieces r, r + R, .. of a column in registers (state layout [.., vdim, dim]: coalesced loads, and
// the lanes' reads of a token's k / q from shared memory fall into consecutive banks).  The 2 CPT (or CPT) column
// sums are reduced over the R lanes with a transposing tree: every step halves the number of values a lane carries.
// The other 4 or 8 warps stage the next 16 tokens (load, unit norms or decays, k . q, fp32 into the other shared-memory buffer)
// and write the previous 16 tokens' outputs while the owners run; one barrier per 16 tokens.
// A column's sum runs in the same order whatever CPT is, and time runs in order: a row's result depends neither on
// the batch nor on how its sequence was cut into steps.
#include "../../include/vila_b200.h"
#include "common.cuh"
#include "kernels.h"
#include "dtype_any.cuh"

namespace vb {
namespace {

constexpr int kOwnerWarps = 4;
constexpr int kChunk = 16;   // tokens per stage

__device__ __forceinline__ float softplus_f(float z) { return z > 20.0f ? z : log1pf(expf(z)); }

// four consecutive elements as raw bits (bf16: in .x / .y): nothing consumes the load until raw4_to_float
__device__ __forceinline__ uint4 ld_raw4(const void* p, int dt, size_t off, int i, int n, bool vec) {
  uint4 u = make_uint4(0u, 0u, 0u, 0u);
  if (i >= n) return u;
  if (vec) {
    if (dt) return __ldg(reinterpret_cast<const uint4*>(static_cast<const float*>(p) + off + i));
    const uint2 h = __ldg(reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(p) + off + i));
    u.x = h.x;
    u.y = h.y;
    return u;
  }
  uint32_t e[4];
#pragma unroll
  for (int k = 0; k < 4; ++k) e[k] = i + k < n ? ld_raw(p, dt, off + i + k) : 0u;
  if (dt) return make_uint4(e[0], e[1], e[2], e[3]);
  u.x = e[0] | (e[1] << 16);
  u.y = e[2] | (e[3] << 16);
  return u;
}
__device__ __forceinline__ float4 raw4_to_float(uint4 u, int dt) {
  if (dt) return make_float4(__uint_as_float(u.x), __uint_as_float(u.y), __uint_as_float(u.z), __uint_as_float(u.w));
  return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16),
                     __uint_as_float(u.y & 0xffff0000u));
}
__device__ __forceinline__ float4 silu4(float4 v) {
  return make_float4(silu_exact_f(v.x), silu_exact_f(v.y), silu_exact_f(v.z), silu_exact_f(v.w));
}
__device__ __forceinline__ float dot4(float4 a, float4 b, float s) {
  s = fmaf(a.x, b.x, s);
  s = fmaf(a.y, b.y, s);
  s = fmaf(a.z, b.z, s);
  return fmaf(a.w, b.w, s);
}

// Sum NV values per lane over the R lanes of a group.  Afterwards v[0] of lane r is the complete sum of value
// (r * NV) / R (R / NV neighbouring lanes hold the same one).
template <int R, int NV>
__device__ __forceinline__ void transpose_sum(float (&v)[NV], int r) {
  int n = NV;
#pragma unroll
  for (int off = R / 2; off >= 1; off >>= 1) {
    if (n > 1) {
      n >>= 1;
      const bool hi = (r & off) != 0;
#pragma unroll
      for (int i = 0; i < NV / 2; ++i) {
        if (i < n) {
          const float send = hi ? v[i] : v[i + n];
          const float keep = hi ? v[i + n] : v[i];
          v[i] = keep + __shfl_xor_sync(0xffffffffu, send, off);
        }
      }
    } else {
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], off);
    }
  }
}

enum Mode : int { kDelta, kGla, kDecay };

struct ScanArgs {
  const void *q, *k, *v;        // rows of the step; head offsets are added by the kernel
  int64_t ldq, ldk, ldv;
  const void *a, *b;            // delta: decay / step-size pre-activations, column h;  gla: a = z, H * dim columns
  int64_t lda, ldb;
  const float *A_log, *bias;    // delta: A_log [H], dt_bias [H];  gla: bias [H * dim] or NULL
  float* state;                 // [slots, H, vdim, dim]
  const int32_t* seqs;
  float* out;
  int64_t ldo;
  int in_dt, a_dt, H, G, dim, vdim;
  float q_scale, eps, inv_tau;
  const float* decay;           // decay: [H]
  int silu;                     // decay: q, k and v are pre-activations, SiLU is taken as they are read
  int vec_qk, vec_a;            // four-element loads of q | k and of z are aligned
};

template <int MODE, int R, int KPT, int CPT, int kStageWarps>
__global__ void __launch_bounds__(32 * (kOwnerWarps + kStageWarps)) outer_scan_kernel(const ScanArgs p) {
  extern __shared__ __align__(16) float sm[];
  constexpr bool DELTA = MODE == kDelta, GLA = MODE == kGla;
  constexpr int NP = R * KPT;                       // key channels the owners cover
  constexpr int NQ = KPT / 4;                       // float4 pieces per lane
  constexpr int GPW = 32 / R;                       // column groups per warp
  constexpr int COLS = kOwnerWarps * GPW * CPT;
  constexpr int NV = DELTA ? 2 * CPT : CPT;
  constexpr int NVEC = GLA ? 3 : 2;                 // staged vectors per token: k, q (, alpha)
  constexpr int TOK = NVEC * NP;
  constexpr int NG = NP > 128 ? NP / 128 : 1;       // four-element pieces a staging lane handles per vector
  constexpr int TPW = kChunk / kStageWarps;         // tokens of a stage per staging warp
  constexpr int TB = NG == 1 ? TPW : (NG == 2 ? 2 : 1);   // of which it has so many in flight
  float* vec_s = sm;                                // [2][kChunk][NVEC][NP]
  float* v_s = vec_s + 2 * kChunk * TOK;            // [2][kChunk][COLS]
  float* y_s = v_s + 2 * kChunk * COLS;             // [2][kChunk][COLS]
  float4* sc_s = reinterpret_cast<float4*>(y_s + 2 * kChunk * COLS);   // [2][kChunk]: (g, beta, k.q, -)

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int* sq = p.seqs + 4 * blockIdx.x;
  const int row0 = sq[0], n = sq[1], pos0 = sq[2], slot = sq[3];
  const int h = blockIdx.y, dim = p.dim, vdim = p.vdim, kh = h / (p.H / p.G);
  const int col0 = blockIdx.z * COLS;
  const int nchunks = (n + kChunk - 1) / kChunk;

  if (warp >= kOwnerWarps) {
    // ---------------- staging warps ----------------
    const int sw = warp - kOwnerWarps, st = threadIdx.x - kOwnerWarps * 32;
    const int dt = p.in_dt, adt = p.a_dt;
    const size_t qoff = static_cast<size_t>(kh) * dim, voff = static_cast<size_t>(h) * vdim;
    const size_t zoff = static_cast<size_t>(h) * dim;
    const float neg_a = DELTA ? -expf(p.A_log[h]) : 0.f, dbias = DELTA ? p.bias[h] : 0.f;
    float4 zb[NG];
#pragma unroll
    for (int j = 0; j < NG; ++j) {
      zb[j] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (GLA && p.bias) {
        const int i = 4 * (lane + 32 * j);
        float e[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) e[k] = i + k < dim ? p.bias[zoff + i + k] : 0.f;
        zb[j] = make_float4(e[0], e[1], e[2], e[3]);
      }
    }
    auto stage = [&](int ch) {
      const int t0 = ch * kChunk, nt = min(kChunk, n - t0), bf = ch & 1;
      float* vb_ = vec_s + bf * kChunk * TOK;
      // the value columns and (delta) the head's two scalars of every token: loads first
      constexpr int VN = (kChunk * COLS + kStageWarps * 32 - 1) / (kStageWarps * 32);
      uint32_t rv[VN], ra = 0u, rb = 0u;
#pragma unroll
      for (int k = 0; k < VN; ++k) {
        const int idx = st + k * kStageWarps * 32, t = idx / COLS, c = col0 + idx % COLS;
        rv[k] = (t < nt && c < vdim) ? ld_raw(p.v, dt, static_cast<size_t>(row0 + t0 + t) * p.ldv + voff + c) : 0u;
      }
      if (DELTA && st < nt) {
        ra = ld_raw(p.a, adt, static_cast<size_t>(row0 + t0 + st) * p.lda + h);
        rb = ld_raw(p.b, adt, static_cast<size_t>(row0 + t0 + st) * p.ldb + h);
      }
#pragma unroll 1
      for (int tb = 0; tb < TPW; tb += TB) {
        uint4 rk[TB][NG], rq[TB][NG], rz[TB][NG];
#pragma unroll
        for (int u = 0; u < TB; ++u) {
          const int t = sw + (tb + u) * kStageWarps;
          const size_t row = static_cast<size_t>(row0 + t0 + t);
#pragma unroll
          for (int j = 0; j < NG; ++j) {
            const int i = t < nt ? 4 * (lane + 32 * j) : dim;
            rk[u][j] = ld_raw4(p.k, dt, row * p.ldk + qoff, i, dim, p.vec_qk != 0);
            rq[u][j] = ld_raw4(p.q, dt, row * p.ldq + qoff, i, dim, p.vec_qk != 0);
            if (GLA) rz[u][j] = ld_raw4(p.a, adt, row * p.lda + zoff, i, dim, p.vec_a != 0);
          }
        }
#pragma unroll
        for (int u = 0; u < TB; ++u) {
          const int t = sw + (tb + u) * kStageWarps;
          if (t >= nt) break;
          float kq = 0.f, kk = 0.f, qq = 0.f;
          float4 kv[NG], qv[NG];
#pragma unroll
          for (int j = 0; j < NG; ++j) {
            kv[j] = raw4_to_float(rk[u][j], dt);
            qv[j] = raw4_to_float(rq[u][j], dt);
            if (MODE == kDecay && p.silu) {
              kv[j] = silu4(kv[j]);
              qv[j] = silu4(qv[j]);
            }
            kq = dot4(kv[j], qv[j], kq);
            if (DELTA) {
              kk = dot4(kv[j], kv[j], kk);
              qq = dot4(qv[j], qv[j], qq);
            }
          }
#pragma unroll
          for (int o = 16; o > 0; o >>= 1) {
            kq += __shfl_xor_sync(0xffffffffu, kq, o);
            if (DELTA) {
              kk += __shfl_xor_sync(0xffffffffu, kk, o);
              qq += __shfl_xor_sync(0xffffffffu, qq, o);
            }
          }
          const float ks = DELTA ? 1.0f / sqrtf(kk + p.eps) : 1.0f;
          const float qs = (DELTA ? 1.0f / sqrtf(qq + p.eps) : 1.0f) * p.q_scale;
          float* kd = vb_ + t * TOK;
#pragma unroll
          for (int j = 0; j < NG; ++j) {
            const int i = 4 * (lane + 32 * j);
            if (i < NP) {
              float4 q4 = make_float4(qv[j].x * qs, qv[j].y * qs, qv[j].z * qs, qv[j].w * qs);
              *reinterpret_cast<float4*>(kd + i) = make_float4(kv[j].x * ks, kv[j].y * ks, kv[j].z * ks, kv[j].w * ks);
              if (GLA) {
                const float4 z = raw4_to_float(rz[u][j], adt);
                const float4 al = make_float4(expf(-softplus_f(-(z.x + zb[j].x)) * p.inv_tau),
                                              expf(-softplus_f(-(z.y + zb[j].y)) * p.inv_tau),
                                              expf(-softplus_f(-(z.z + zb[j].z)) * p.inv_tau),
                                              expf(-softplus_f(-(z.w + zb[j].w)) * p.inv_tau));
                q4 = make_float4(q4.x * al.x, q4.y * al.y, q4.z * al.z, q4.w * al.w);
                *reinterpret_cast<float4*>(kd + 2 * NP + i) = al;
              }
              *reinterpret_cast<float4*>(kd + NP + i) = q4;
            }
          }
          if (lane == 0) reinterpret_cast<float*>(sc_s + bf * kChunk + t)[2] = kq * ks * qs;
        }
      }
#pragma unroll
      for (int k = 0; k < VN; ++k) {
        const int idx = st + k * kStageWarps * 32;
        const float v = raw_to_float(rv[k], dt);
        if (idx < kChunk * COLS) v_s[bf * kChunk * COLS + idx] = MODE == kDecay && p.silu ? silu_exact_f(v) : v;
      }
      if (DELTA && st < nt) {
        float* s = reinterpret_cast<float*>(sc_s + bf * kChunk + st);
        s[0] = expf(neg_a * softplus_f(raw_to_float(ra, adt) + dbias));
        s[1] = sigmoid_f(raw_to_float(rb, adt));
      }
    };
    auto flush = [&](int ch) {
      const int t0 = ch * kChunk, nt = min(kChunk, n - t0);
      const float* y = y_s + (ch & 1) * kChunk * COLS;
      for (int idx = st; idx < nt * COLS; idx += kStageWarps * 32) {
        const int t = idx / COLS, c = col0 + idx % COLS;
        if (c < vdim) p.out[static_cast<size_t>(row0 + t0 + t) * p.ldo + voff + c] = y[idx];
      }
    };
    stage(0);
    __syncthreads();
    for (int ch = 0; ch < nchunks; ++ch) {
      if (ch + 1 < nchunks) stage(ch + 1);
      if (ch > 0) flush(ch - 1);
      __syncthreads();
    }
    if (nchunks > 0) flush(nchunks - 1);
    return;
  }

  // ---------------- owners of the state ----------------
  const int r = lane & (R - 1), cg = (warp * GPW + lane / R) * CPT;   // first column of this lane's group
  float* stp = p.state + ((static_cast<size_t>(slot) * p.H + h) * vdim + col0 + cg) * dim;
  const bool vec_s4 = (dim & 3) == 0;
  float4 S[CPT][NQ];
#pragma unroll
  for (int c = 0; c < CPT; ++c)
#pragma unroll
    for (int j = 0; j < NQ; ++j) {
      S[c][j] = make_float4(0.f, 0.f, 0.f, 0.f);
      const int i = 4 * (r + R * j);
      if (pos0 > 0 && col0 + cg + c < vdim && i < dim) {
        const float* s = stp + static_cast<size_t>(c) * dim + i;
        if (vec_s4) S[c][j] = *reinterpret_cast<const float4*>(s);
        else {
          S[c][j].x = s[0];
          if (i + 1 < dim) S[c][j].y = s[1];
          if (i + 2 < dim) S[c][j].z = s[2];
          if (i + 3 < dim) S[c][j].w = s[3];
        }
      }
    }
  constexpr int kSpan = R / NV;                    // neighbouring lanes that end up with the same sum
  const int mine = r / kSpan;                      // which of the NV sums this lane ends up with
  const int my_col = DELTA ? mine - CPT : mine;    // its column, if it is a read-out
  const bool writes = my_col >= 0 && (r % kSpan) == 0;
  const float gh = MODE == kDecay ? p.decay[h] : 0.f;
  __syncthreads();
  for (int ch = 0; ch < nchunks; ++ch) {
    const int nt = min(kChunk, n - ch * kChunk), bf = ch & 1;
    const float* tok = vec_s + bf * kChunk * TOK;
    const float* vv = v_s + bf * kChunk * COLS;
    float* yy = y_s + bf * kChunk * COLS;
    const float4* sc = sc_s + bf * kChunk;
    float4 kn[NQ], qn[NQ], an[NQ];
#pragma unroll
    for (int j = 0; j < NQ; ++j) {
      kn[j] = reinterpret_cast<const float4*>(tok)[r + R * j];
      qn[j] = reinterpret_cast<const float4*>(tok + NP)[r + R * j];
      if (GLA) an[j] = reinterpret_cast<const float4*>(tok + 2 * NP)[r + R * j];
    }
    for (int t = 0; t < nt; ++t) {
      float4 kc[NQ], qc[NQ], ac[NQ];
      float vc[CPT];
      const float4 s4 = sc[t];
#pragma unroll
      for (int c = 0; c < CPT; ++c) vc[c] = vv[t * COLS + cg + c];
#pragma unroll
      for (int j = 0; j < NQ; ++j) {
        kc[j] = kn[j];
        qc[j] = qn[j];
        if (GLA) ac[j] = an[j];
      }
      // the next token's vectors (row kChunk of a buffer does not exist: the last token reads its own again)
      const float* nx = tok + (t + 1 < nt ? t + 1 : t) * TOK;
#pragma unroll
      for (int j = 0; j < NQ; ++j) {
        kn[j] = reinterpret_cast<const float4*>(nx)[r + R * j];
        qn[j] = reinterpret_cast<const float4*>(nx + NP)[r + R * j];
        if (GLA) an[j] = reinterpret_cast<const float4*>(nx + 2 * NP)[r + R * j];
      }
      float d[NV];
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        float4 ek = make_float4(0.f, 0.f, 0.f, 0.f), eq = ek;   // four partial sums: short chains
#pragma unroll
        for (int j = 0; j < NQ; ++j) {
          if (DELTA) {
            ek.x = fmaf(S[c][j].x, kc[j].x, ek.x); ek.y = fmaf(S[c][j].y, kc[j].y, ek.y);
            ek.z = fmaf(S[c][j].z, kc[j].z, ek.z); ek.w = fmaf(S[c][j].w, kc[j].w, ek.w);
          }
          eq.x = fmaf(S[c][j].x, qc[j].x, eq.x); eq.y = fmaf(S[c][j].y, qc[j].y, eq.y);
          eq.z = fmaf(S[c][j].z, qc[j].z, eq.z); eq.w = fmaf(S[c][j].w, qc[j].w, eq.w);
        }
        if (DELTA) d[c] = (ek.x + ek.y) + (ek.z + ek.w);
        d[NV - CPT + c] = (eq.x + eq.y) + (eq.z + eq.w);
      }
      transpose_sum<R, NV>(d, r);
      if (DELTA) {
        const float g = s4.x, beta = s4.y;
        float u[CPT], um = 0.f;
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
          const float dk = __shfl_sync(0xffffffffu, d[0], c * kSpan, R);
          u[c] = beta * (vc[c] - g * dk);
          if (c == my_col) um = u[c];
        }
        if (writes) yy[t * COLS + cg + my_col] = fmaf(g, d[0], s4.z * um);
#pragma unroll
        for (int c = 0; c < CPT; ++c)
#pragma unroll
          for (int j = 0; j < NQ; ++j) {
            S[c][j].x = fmaf(g, S[c][j].x, kc[j].x * u[c]);
            S[c][j].y = fmaf(g, S[c][j].y, kc[j].y * u[c]);
            S[c][j].z = fmaf(g, S[c][j].z, kc[j].z * u[c]);
            S[c][j].w = fmaf(g, S[c][j].w, kc[j].w * u[c]);
          }
      } else {
        float vm = 0.f;
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
          if (c == my_col) vm = vc[c];
#pragma unroll
          for (int j = 0; j < NQ; ++j) {
            S[c][j].x = fmaf(GLA ? ac[j].x : gh, S[c][j].x, kc[j].x * vc[c]);
            S[c][j].y = fmaf(GLA ? ac[j].y : gh, S[c][j].y, kc[j].y * vc[c]);
            S[c][j].z = fmaf(GLA ? ac[j].z : gh, S[c][j].z, kc[j].z * vc[c]);
            S[c][j].w = fmaf(GLA ? ac[j].w : gh, S[c][j].w, kc[j].w * vc[c]);
          }
        }
        if (writes) yy[t * COLS + cg + my_col] = fmaf(s4.z, vm, GLA ? d[0] : gh * d[0]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int c = 0; c < CPT; ++c)
#pragma unroll
    for (int j = 0; j < NQ; ++j) {
      const int i = 4 * (r + R * j);
      if (col0 + cg + c < vdim && i < dim) {
        float* s = stp + static_cast<size_t>(c) * dim + i;
        if (vec_s4) *reinterpret_cast<float4*>(s) = S[c][j];
        else {
          s[0] = S[c][j].x;
          if (i + 1 < dim) s[1] = S[c][j].y;
          if (i + 2 < dim) s[2] = S[c][j].z;
          if (i + 3 < dim) s[3] = S[c][j].w;
        }
      }
    }
}

template <int MODE, int R, int KPT, int CPT>
int launch_scan(const ScanArgs& p, int nseq, cudaStream_t stream) {
  constexpr int NP = R * KPT, COLS = kOwnerWarps * (32 / R) * CPT;
  constexpr size_t smem = sizeof(float) * (2 * kChunk * (MODE == kGla ? 3 : 2) * NP + 4 * kChunk * COLS + 2 * kChunk * 4);
  static_assert(smem <= 224 * 1024, "outer_scan: shared memory");
  // the staging work of a token is the same for 2 as for 4 columns per group: twice the warps for the narrow form,
  // where an SM holds one or two CTAs, fewer for the wide one, where CTAs share it
  constexpr int SW = CPT == 4 ? 4 : 8;
  auto kern = outer_scan_kernel<MODE, R, KPT, CPT, SW>;
  static PerDeviceOnce attr_once;
  if (smem > 48 * 1024 && attr_once.first())
    VB_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  const dim3 grid(nseq, p.H, (p.vdim + COLS - 1) / COLS);
  VB_CHECK(grid.y <= 65535 && grid.z <= 65535, "outer_scan: H=%d vdim=%d", p.H, p.vdim);
  VB_CUDA(launch_serial(kern, grid, dim3(32 * (kOwnerWarps + SW)), smem, stream, p));
  return 0;
}

// columns per lane group: four where the launch still fills the machine twice over, else fewer, so that one long
// prompt spreads over more CTAs
template <int MODE, int R, int KPT>
int pick_columns(const ScanArgs& p, int nseq, cudaStream_t stream) {
  const long groups = static_cast<long>(nseq) * p.H * ((p.vdim + 4 * (32 / R) - 1) / (4 * (32 / R)));   // CTAs at CPT = 1
  if (groups >= 8L * num_sms()) return launch_scan<MODE, R, KPT, 4>(p, nseq, stream);
  return launch_scan<MODE, R, KPT, 2>(p, nseq, stream);
}

template <int MODE>
int scan_by_dim(const ScanArgs& p, int nseq, cudaStream_t stream) {
  if (p.dim <= 32) return pick_columns<MODE, 8, 4>(p, nseq, stream);
  if (p.dim <= 64) return pick_columns<MODE, 16, 4>(p, nseq, stream);
  if (p.dim <= 128) return pick_columns<MODE, 16, 8>(p, nseq, stream);
  if (p.dim <= 256) return pick_columns<MODE, 16, 16>(p, nseq, stream);
  return pick_columns<MODE, 32, 16>(p, nseq, stream);
}

// rows that start on a four-element boundary of their dtype (8 bytes bf16, 16 bytes fp32)
bool rows_aligned4(const void* base, int64_t ld, int dt) {
  return ld % 4 == 0 && reinterpret_cast<uintptr_t>(base) % (dt ? 16 : 8) == 0;
}

}  // namespace

int delta_scan(const vila_delta_scan_params& p, cudaStream_t stream) {
  if (p.nseq <= 0) return 0;
  VB_CHECK(p.H >= 1 && p.G >= 1 && p.H % p.G == 0 && p.dim >= 1 && p.dim <= 512 && p.vdim >= 1 && p.A_log && p.dt_bias,
           "delta_scan: H=%d G=%d dim=%d (<= 512) vdim=%d", p.H, p.G, p.dim, p.vdim);
  const size_t es = p.in_dtype ? 4 : 2;
  const char* base = static_cast<const char*>(p.qkv);
  ScanArgs a = {};
  a.q = base;
  a.k = base + static_cast<size_t>(p.G) * p.dim * es;
  a.v = base + 2 * static_cast<size_t>(p.G) * p.dim * es;
  a.ldq = a.ldk = a.ldv = p.ld_qkv;
  a.a = p.a; a.lda = p.ld_a;
  a.b = p.b; a.ldb = p.ld_b;
  a.A_log = p.A_log; a.bias = p.dt_bias;
  a.state = p.state; a.seqs = p.seqs; a.out = p.out; a.ldo = p.ld_out;
  a.in_dt = p.in_dtype; a.a_dt = p.ab_dtype;
  a.H = p.H; a.G = p.G; a.dim = p.dim; a.vdim = p.vdim;
  a.q_scale = p.q_scale; a.eps = p.unit_eps;
  a.vec_qk = p.dim % 4 == 0 && rows_aligned4(a.q, p.ld_qkv, p.in_dtype) && rows_aligned4(a.k, p.ld_qkv, p.in_dtype);
  return scan_by_dim<kDelta>(a, p.nseq, stream);
}

int gla_scan(const vila_gla_scan_params& p, cudaStream_t stream) {
  if (p.nseq <= 0) return 0;
  VB_CHECK(p.H >= 1 && p.dim >= 1 && p.dim <= 512 && p.vdim >= 1 && p.tau > 0.f, "gla_scan: H=%d dim=%d (<= 512) vdim=%d tau=%f",
           p.H, p.dim, p.vdim, p.tau);
  ScanArgs a = {};
  a.q = p.q; a.k = p.k; a.v = p.v;
  a.ldq = p.ld_q; a.ldk = p.ld_k; a.ldv = p.ld_v;
  a.a = p.z; a.lda = p.ld_z;
  a.bias = p.z_bias;
  a.state = p.state; a.seqs = p.seqs; a.out = p.out; a.ldo = p.ld_out;
  a.in_dt = p.in_dtype; a.a_dt = p.z_dtype;
  a.H = p.H; a.G = p.H; a.dim = p.dim; a.vdim = p.vdim;
  a.q_scale = p.q_scale; a.inv_tau = 1.0f / p.tau;
  a.vec_qk = p.dim % 4 == 0 && rows_aligned4(a.q, p.ld_q, p.in_dtype) && rows_aligned4(a.k, p.ld_k, p.in_dtype);
  a.vec_a = p.dim % 4 == 0 && rows_aligned4(a.a, p.ld_z, p.z_dtype);
  return scan_by_dim<kGla>(a, p.nseq, stream);
}

int decay_scan(const vila_decay_scan_params& p, cudaStream_t stream) {
  if (p.nseq <= 0) return 0;
  VB_CHECK(p.H >= 1 && p.dim >= 1 && p.dim <= 512 && p.vdim >= 1 && p.decay != nullptr, "decay_scan: H=%d dim=%d (<= 512) vdim=%d",
           p.H, p.dim, p.vdim);
  ScanArgs a = {};
  a.q = p.q; a.k = p.k; a.v = p.v;
  a.ldq = p.ld_q; a.ldk = p.ld_k; a.ldv = p.ld_v;
  a.decay = p.decay;
  a.silu = p.silu;
  a.state = p.state; a.seqs = p.seqs; a.out = p.out; a.ldo = p.ld_out;
  a.in_dt = p.in_dtype;
  a.H = p.H; a.G = p.H; a.dim = p.dim; a.vdim = p.vdim;
  a.q_scale = p.q_scale;
  a.vec_qk = p.dim % 4 == 0 && rows_aligned4(a.q, p.ld_q, p.in_dtype) && rows_aligned4(a.k, p.ld_k, p.in_dtype);
  return scan_by_dim<kDecay>(a, p.nseq, stream);
}

}  // namespace vb
