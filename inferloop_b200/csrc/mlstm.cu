// The matrix memory of xLSTM (mLSTM): per head a matrix state with an exponential input gate and a forget gate a token,
// kept in range by a running maximum, and read out over a normaliser of its own.
//
// Per head, from the projections q, k (d channels) and v (dv channels) of a token and its two gate logits gi, gf (made
// elsewhere in 32-bit, or here for single tokens):
//     i = cap tanh((gi + bi) / cap),   f = logsigmoid(cap tanh((gf + bf) / cap))           logarithms of the gates
//     m_t = max(f + m_{t-1}, i)                                                            m_0 = 0
//     S_t = exp(f + m_{t-1} - m_t) S_{t-1} + exp(i - m_t) k v^T,     n_t likewise with k alone
//     o_t = S_t^T q / (max(|n_t . q|, exp(-m_t)) + eps),   q scaled by q_scale first
// Then o is divided by its root mean square per head, multiplied by a weight and by the sigmoid of an output gate.
// State per request and head: S [d, dv], n [d], m, all 32-bit.
//
//   mlstm_step     single tokens, from the layer's projections to what its output product reads: the gates' two dot products,
//                  the recurrence, the read-out, the norm and the output gate.  A block per (head, sequence).
//   mlstm_gates,   token by token, any sizes up to 256 rows: the gates' chain first (a warp per head and sequence, which owns
//   mlstm_scan     m), then a block per 32 columns with the state in registers, eight threads a column; the normaliser is one
//                  more column of its own.  For short portions and the 32-bit path.
//   mlstm_chunks   long portions of bfloat16 projections, 64 tokens at a time on the tensor cores, in three launches.  With F_t
//                  the sum of the chunk's log forget gates up to token t and m_in the maximum that comes in:
//                      m_t = F_t + max(m_in, max_{s<=t}(i_s - F_s))
//                      S_t^T q_t = exp(F_t + m_in - m_t) S_in^T q_t + sum_{s<=t} exp(F_t - F_s + i_s - m_t) (q_t . k_s) v_s
//                  (1) every chunk's own contribution, relative to its own maximum; (2) the chunks' incoming states, one after
//                  the other; (3) every chunk's outputs.  q, k and v are bfloat16 as stored; every 32-bit operand (the weighted
//                  keys, the weighted scores, the state) is cut into three exact bfloat16 pieces whose products are added in
//                  32-bit, the smallest piece first.
//
// Everything is 32-bit; the projections come in the compute dtype.  A sequence whose slot is negative (a dummy row that
// pads a recorded launch) starts from zero and stores nothing.
#include <math.h>
#include "common.cuh"
#include "sm100.cuh"

using namespace ilb;

constexpr int kMaxRows = 256;         // rows (key channels) of a head's state

__device__ __forceinline__ float log_gate_in(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_gate_forget(float z, float cap) {
  const float x = cap * tanhf(z / cap);
  return fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
}
__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }

// which sequence, and which of its tiles of `tile` tokens, block `b` works on; false: none
__device__ __forceinline__ bool find_tile(const int* __restrict__ cu_q, int n_seqs, int tile, int b, int& seq, int& index) {
  for (seq = 0; seq < n_seqs; ++seq) {
    const int n = (cu_q[seq + 1] - cu_q[seq] + tile - 1) / tile;
    if (b < n) { index = b; return true; }
    b -= n;
  }
  return false;
}

struct MlstmParams {
  const void* proj; int ld, col_q, col_k, col_v;             // [T, ld] of the compute dtype
  const float* gates; int ld_g;                              // [T, ld_g]: heads logits of the input gate, then heads of the forget gate
  const float* bias_i; const float* bias_f;                  // [heads]
  float* state; float* norm; float* max;                     // [slots, heads, d, dv], [slots, heads, d], [slots, heads]
  const int* cu_q; const int* slots;
  int n_seqs, heads, d, dv;
  float cap, q_scale, eps;
};

// ---------------------------------------------------------------- the gates' chain, token by token
// keep[t, h] = exp(f + m_{t-1} - m_t), add[t, h] = exp(i - m_t), floor[t, h] = exp(-m_t); m from and to the slot.  One warp per
// (head, sequence).
__global__ void __launch_bounds__(32)
mlstm_gates_kernel(const MlstmParams p, float* __restrict__ keep, float* __restrict__ add, float* __restrict__ floor_) {
  ilb::pdl_launch_dependents();
  ilb::pdl_wait();
  const int h = blockIdx.x, seq = blockIdx.y, lane = threadIdx.x;
  const int tok0 = p.cu_q[seq], end = p.cu_q[seq + 1], slot = p.slots[seq];
  if (end <= tok0) return;
  float* own = slot >= 0 ? p.max + (size_t)slot * p.heads + h : nullptr;
  float m = own != nullptr ? *own : 0.f;
  const float bi = p.bias_i[h], bf = p.bias_f[h];
  for (int t0 = tok0; t0 < end; t0 += 32) {
    const int t = min(t0 + lane, end - 1);
    const float i = log_gate_in(p.gates[(size_t)t * p.ld_g + h] + bi, p.cap);
    const float f = log_gate_forget(p.gates[(size_t)t * p.ld_g + p.heads + h] + bf, p.cap);
    float before = m, after = m;
    const int n = min(32, end - t0);
    for (int s = 0; s < n; ++s) {
      const float next = fmaxf(__shfl_sync(0xffffffffu, f, s) + m, __shfl_sync(0xffffffffu, i, s));
      if (lane == s) { before = m; after = next; }
      m = next;
    }
    if (lane < n) {
      const size_t at = (size_t)t * p.heads + h;
      keep[at] = expf(f + before - after);
      add[at] = expf(i - after);
      floor_[at] = expf(-after);
    }
  }
  if (own != nullptr && lane == 0) *own = m;
}

// ---------------------------------------------------------------- the recurrence, token by token
constexpr int kCols = 32;             // columns of the state per block
constexpr int kTile = 16;             // tokens in shared memory at a time

template <typename TI, int Q>         // Q: groups of four rows a thread holds; 32 Q rows in all
__global__ void __launch_bounds__(256)
mlstm_scan_kernel(const MlstmParams p, const float* __restrict__ keep, const float* __restrict__ add, const float* __restrict__ floor_,
                  float* __restrict__ y, float* __restrict__ den) {
  ilb::pdl_launch_dependents();
  ilb::pdl_wait();
  constexpr int D = 32 * Q;                              // rows, padded with zeros
  __shared__ __align__(16) float Ks[kTile * D], Qs[kTile * D];
  __shared__ float Vs[kTile * kCols], Aw[kTile], Kw[kTile];
  const int h = blockIdx.x, seq = blockIdx.z;
  const bool is_norm = blockIdx.y == gridDim.y - 1;      // the normaliser: one column whose value is one
  const int c0 = blockIdx.y * kCols;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, sl = lane & 7, cl = warp * 4 + (lane >> 3);
  const int width = is_norm ? 1 : p.dv, col = is_norm ? cl : c0 + cl;
  const int tok0 = p.cu_q[seq], end = p.cu_q[seq + 1], slot = p.slots[seq];
  float* own = nullptr;
  if (slot >= 0) own = is_norm ? p.norm + ((size_t)slot * p.heads + h) * p.d : p.state + ((size_t)slot * p.heads + h) * p.d * p.dv;
  const bool live = col < width;
  float4 S[Q];                                           // rows 4 (8 q + sl) + j
#pragma unroll
  for (int q = 0; q < Q; ++q) {
    float v[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = 4 * (8 * q + sl) + j;
      v[j] = (own != nullptr && live && n < p.d) ? own[(size_t)n * width + col] : 0.f;
    }
    S[q] = make_float4(v[0], v[1], v[2], v[3]);
  }
  const TI* proj = reinterpret_cast<const TI*>(p.proj);
  for (int t0 = tok0; t0 < end; t0 += kTile) {
    const int ts = min(kTile, end - t0);
    for (int i = threadIdx.x; i < ts * D; i += 256) {
      const int tt = i / D, n = i % D;
      const TI* row = proj + (size_t)(t0 + tt) * p.ld + h * p.d + n;
      Ks[i] = n < p.d ? to_float(row[p.col_k]) : 0.f;
      Qs[i] = n < p.d ? to_float(row[p.col_q]) * p.q_scale : 0.f;
    }
    for (int i = threadIdx.x; i < ts * kCols; i += 256) {
      const int tt = i / kCols, c = c0 + i % kCols;
      Vs[i] = is_norm ? 1.f : (c < p.dv ? to_float(proj[(size_t)(t0 + tt) * p.ld + p.col_v + h * p.dv + c]) : 0.f);
    }
    if (threadIdx.x < ts) {
      Kw[threadIdx.x] = keep[(size_t)(t0 + threadIdx.x) * p.heads + h];
      Aw[threadIdx.x] = add[(size_t)(t0 + threadIdx.x) * p.heads + h];
    }
    __syncthreads();
    for (int tt = 0; tt < ts; ++tt) {
      const float4* k4 = reinterpret_cast<const float4*>(Ks + tt * D) + sl;
      const float4* q4 = reinterpret_cast<const float4*>(Qs + tt * D) + sl;
      const float a = Kw[tt], b = Aw[tt] * Vs[tt * kCols + cl];
      float z0 = 0.f, z1 = 0.f;
#pragma unroll
      for (int q = 0; q < Q; ++q) {
        const float4 k = k4[8 * q], r = q4[8 * q];
        S[q].x = fmaf(a, S[q].x, b * k.x); z0 = fmaf(r.x, S[q].x, z0);
        S[q].y = fmaf(a, S[q].y, b * k.y); z1 = fmaf(r.y, S[q].y, z1);
        S[q].z = fmaf(a, S[q].z, b * k.z); z0 = fmaf(r.z, S[q].z, z0);
        S[q].w = fmaf(a, S[q].w, b * k.w); z1 = fmaf(r.w, S[q].w, z1);
      }
      float z = z0 + z1;
      z += __shfl_xor_sync(0xffffffffu, z, 1);
      z += __shfl_xor_sync(0xffffffffu, z, 2);
      z += __shfl_xor_sync(0xffffffffu, z, 4);
      if (sl == 0 && live) {
        if (is_norm) den[(size_t)(t0 + tt) * p.heads + h] = fmaxf(fabsf(z), floor_[(size_t)(t0 + tt) * p.heads + h]) + p.eps;
        else y[(size_t)(t0 + tt) * p.heads * p.dv + (size_t)h * p.dv + col] = z;
      }
    }
    __syncthreads();
  }
  if (own != nullptr && live) {
#pragma unroll
    for (int q = 0; q < Q; ++q) {
      const float v[4] = {S[q].x, S[q].y, S[q].z, S[q].w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int n = 4 * (8 * q + sl) + j;
        if (n < p.d) own[(size_t)n * width + col] = v[j];
      }
    }
  }
}

static int check_sizes(const MlstmParams& p, int dtype) {
  ILB_REQUIRE(p.heads > 0 && p.heads <= 65535 && p.d > 0 && p.d <= kMaxRows && p.dv > 0, "mlstm: %d heads of %d x %d (at most %d rows)", p.heads, p.d, p.dv, kMaxRows);
  ILB_REQUIRE(dtype == kF32 || dtype == kBF16, "mlstm: unknown dtype %d", dtype);
  ILB_REQUIRE(p.n_seqs >= 0 && p.n_seqs <= 65535, "mlstm: too many sequences");
  ILB_REQUIRE(p.ld >= p.col_q + p.heads * p.d && p.ld >= p.col_k + p.heads * p.d && p.ld >= p.col_v + p.heads * p.dv, "mlstm: the projection's rows are too short");
  ILB_REQUIRE(p.cap > 0.f && p.eps >= 0.f, "mlstm: the gates' bound must be positive");
  ILB_REQUIRE(p.state != nullptr && p.norm != nullptr && p.max != nullptr && p.bias_i != nullptr && p.bias_f != nullptr, "mlstm: missing tensors");
  return 0;
}

// proj [T, ld] of `dtype`; gates [T, ld_g] 32-bit; scratch: 3 * T * heads floats; y [T, heads * dv] = S^T q, den [T, heads] what
// it is to be divided by.
ILB_EXPORT int ilb_mlstm_scan(const void* proj, int dtype, int ld, int col_q, int col_k, int col_v, const float* gates, int ld_g,
                              const float* bias_i, const float* bias_f, float cap, float q_scale, float eps, float* state, float* norm,
                              float* max, float* scratch, float* y, float* den, const int* cu_q, const int* slots, int n_seqs, int n_tokens,
                              int heads, int d, int dv, cudaStream_t stream) {
  const MlstmParams p{proj, ld, col_q, col_k, col_v, gates, ld_g, bias_i, bias_f, state, norm, max, cu_q, slots, n_seqs, heads, d, dv, cap, q_scale, eps};
  if (int rc = check_sizes(p, dtype)) return rc;
  ILB_REQUIRE(gates != nullptr && ld_g >= 2 * heads && scratch != nullptr && y != nullptr && den != nullptr, "mlstm_scan: missing inputs");
  if (n_seqs == 0 || n_tokens == 0) return 0;
  float *keep = scratch, *add = keep + (size_t)n_tokens * heads, *floor_ = add + (size_t)n_tokens * heads;
  ilb::launch(mlstm_gates_kernel, dim3(heads, n_seqs), dim3(32), 0, stream, p, keep, add, floor_);
  if (int rc = check_launch("mlstm_gates")) return rc;
  const dim3 grid(heads, (dv + kCols - 1) / kCols + 1, n_seqs);
  ILB_REQUIRE(grid.y <= 65535, "mlstm_scan: too many columns");
#define ILB_MS(TI, Q) ilb::launch(mlstm_scan_kernel<TI, Q>, grid, dim3(256), 0, stream, p, (const float*)keep, (const float*)add, (const float*)floor_, y, den)
#define ILB_MSQ(TI) do { if (d <= 32) ILB_MS(TI, 1); else if (d <= 64) ILB_MS(TI, 2); else if (d <= 128) ILB_MS(TI, 4); else ILB_MS(TI, 8); } while (0)
  if (dtype == kF32) ILB_MSQ(float); else ILB_MSQ(__nv_bfloat16);
#undef ILB_MSQ
#undef ILB_MS
  return check_launch("mlstm_scan");
}

// ---------------------------------------------------------------- single tokens
struct MlstmStep {
  MlstmParams a;
  const void* x; int width;          // [T, width]: the mixer's input, of the compute dtype
  const void* w_gates;               // [2 heads, width]: rows of the input gate, then of the forget gate
  int col_g;                         // the output gate's columns in proj
  const float* norm_w; float norm_eps;
  void* out; int ld_out;
};

constexpr int kStepThreads = 256, kStepWarps = kStepThreads / 32, kStepRows = 16;

// A block per (head, sequence).  Warp w takes rows w, w + 8, ... of the state, lane l the columns VEC (l + 32 c) ...; up to
// kStepRows rows a thread are in flight together.
template <typename TI, int VEC>
__global__ void __launch_bounds__(kStepThreads)
mlstm_step_kernel(const MlstmStep q) {
  ilb::pdl_launch_dependents();
  ilb::pdl_wait();
  const MlstmParams& p = q.a;
  extern __shared__ float os[];                          // [dv] the head's output
  __shared__ float Ks[kMaxRows], Qs[kMaxRows];
  __shared__ float red[kStepWarps][32 * VEC];
  __shared__ float scratch[33];
  const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int t = p.cu_q[seq];
  if (p.cu_q[seq + 1] - t != 1) return;                  // single tokens only
  const int slot = p.slots[seq];
  const size_t head = (size_t)(slot >= 0 ? slot : 0) * p.heads + h;
  float* own = slot >= 0 ? p.state + head * p.d * p.dv : nullptr;
  const TI* row = reinterpret_cast<const TI*>(p.proj) + (size_t)t * p.ld;
  float S[kStepRows][VEC];
  auto load_rows = [&](int n0, int c) {
#pragma unroll
    for (int i = 0; i < kStepRows; ++i) {
      const int n = n0 + warp + kStepWarps * i;
      const bool on = own != nullptr && n < p.d && c < p.dv;
      if constexpr (VEC == 4) {
        const float4 v = on ? *reinterpret_cast<const float4*>(own + (size_t)n * p.dv + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        S[i][0] = v.x; S[i][1] = v.y; S[i][2] = v.z; S[i][3] = v.w;
      } else {
        S[i][0] = on ? own[(size_t)n * p.dv + c] : 0.f;
      }
    }
  };
  load_rows(0, VEC * lane);                              // the first rows' loads go out before the gates are formed
  // the two gates' logits
  float zi = 0.f, zf = 0.f;
  {
    const TI* x = reinterpret_cast<const TI*>(q.x) + (size_t)t * q.width;
    const TI* wi = reinterpret_cast<const TI*>(q.w_gates) + (size_t)h * q.width;
    const TI* wf = reinterpret_cast<const TI*>(q.w_gates) + (size_t)(p.heads + h) * q.width;
    if (sizeof(TI) == 2 && q.width % 8 == 0) {
      for (int c = tid * 8; c < q.width; c += kStepThreads * 8) {
        const uint4 a = *reinterpret_cast<const uint4*>(x + c), b = *reinterpret_cast<const uint4*>(wi + c), e = *reinterpret_cast<const uint4*>(wf + c);
        const uint32_t av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w}, ev[4] = {e.x, e.y, e.z, e.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float lo = __uint_as_float(av[j] << 16), hi = __uint_as_float(av[j] & 0xFFFF0000u);
          zi = fmaf(lo, __uint_as_float(bv[j] << 16), zi); zi = fmaf(hi, __uint_as_float(bv[j] & 0xFFFF0000u), zi);
          zf = fmaf(lo, __uint_as_float(ev[j] << 16), zf); zf = fmaf(hi, __uint_as_float(ev[j] & 0xFFFF0000u), zf);
        }
      }
    } else {
      for (int c = tid; c < q.width; c += kStepThreads) {
        const float v = to_float(x[c]);
        zi = fmaf(v, to_float(wi[c]), zi);
        zf = fmaf(v, to_float(wf[c]), zf);
      }
    }
  }
  for (int n = tid; n < p.d; n += kStepThreads) {
    Ks[n] = to_float(row[p.col_k + h * p.d + n]);
    Qs[n] = to_float(row[p.col_q + h * p.d + n]) * p.q_scale;
  }
  const float m_old = slot >= 0 ? p.max[head] : 0.f;
  zi = block_sum(zi, scratch);
  zf = block_sum(zf, scratch);
  const float li = log_gate_in(zi + p.bias_i[h], p.cap), lf = log_gate_forget(zf + p.bias_f[h], p.cap);
  const float m = fmaxf(lf + m_old, li), keep = expf(lf + m_old - m), add = expf(li - m);
  float nq = 0.f;
  for (int n = tid; n < p.d; n += kStepThreads) {
    const float v = fmaf(keep, slot >= 0 ? p.norm[head * p.d + n] : 0.f, add * Ks[n]);
    if (slot >= 0) p.norm[head * p.d + n] = v;
    nq = fmaf(v, Qs[n], nq);
  }
  nq = block_sum(nq, scratch);
  if (tid == 0 && slot >= 0) p.max[head] = m;
  const float inv_den = 1.0f / (fmaxf(fabsf(nq), expf(-m)) + p.eps);
  float ss = 0.f;
  for (int c0 = 0; c0 < p.dv; c0 += 32 * VEC) {
    const int c = c0 + VEC * lane;
    float v[VEC], part[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      v[e] = c + e < p.dv ? add * to_float(row[p.col_v + h * p.dv + c + e]) : 0.f;
      part[e] = 0.f;
    }
    for (int n0 = 0; n0 < p.d; n0 += kStepWarps * kStepRows) {
      if (c0 != 0 || n0 != 0) load_rows(n0, c);
#pragma unroll
      for (int i = 0; i < kStepRows; ++i) {
        const int n = n0 + warp + kStepWarps * i;
        if (n < p.d) {
          const float k = Ks[n], r = Qs[n];
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            S[i][e] = fmaf(keep, S[i][e], k * v[e]);
            part[e] = fmaf(r, S[i][e], part[e]);
          }
          if (own != nullptr && c < p.dv) {
            if constexpr (VEC == 4) *reinterpret_cast<float4*>(own + (size_t)n * p.dv + c) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
            else own[(size_t)n * p.dv + c] = S[i][0];
          }
        }
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) red[warp][VEC * lane + e] = part[e];
    __syncthreads();
    if (tid < 32 * VEC && c0 + tid < p.dv) {
      float o = 0.f;
#pragma unroll
      for (int w = 0; w < kStepWarps; ++w) o += red[w][tid];
      o *= inv_den;
      os[c0 + tid] = o;
      ss = fmaf(o, o, ss);
    }
    __syncthreads();
  }
  ss = block_sum(ss, scratch);
  const float f = 1.0f / sqrtf(ss / (float)p.dv + q.norm_eps);
  TI* dst = reinterpret_cast<TI*>(q.out) + (size_t)t * q.ld_out + h * p.dv;
  for (int c = tid; c < p.dv; c += kStepThreads)
    dst[c] = from_float<TI>(os[c] * f * q.norm_w[h * p.dv + c] * sigmoid_f(to_float(row[q.col_g + h * p.dv + c])));
}

// Single tokens from the layer's projections to what its output product reads; x [T, width] (contiguous rows) is what the
// projections read, w_gates [2 heads, width] of the same dtype.
ILB_EXPORT int ilb_mlstm_step(const void* proj, int dtype, int ld, int col_q, int col_k, int col_v, int col_g, const void* x, int width,
                              const void* w_gates, const float* bias_i, const float* bias_f, float cap, float q_scale, float eps,
                              const float* norm_w, float norm_eps, float* state, float* norm, float* max, void* out, int ld_out,
                              const int* cu_q, const int* slots, int n_seqs, int heads, int d, int dv, cudaStream_t stream) {
  const MlstmParams p{proj, ld, col_q, col_k, col_v, nullptr, 0, bias_i, bias_f, state, norm, max, cu_q, slots, n_seqs, heads, d, dv, cap, q_scale, eps};
  if (int rc = check_sizes(p, dtype)) return rc;
  ILB_REQUIRE(x != nullptr && w_gates != nullptr && width > 0 && norm_w != nullptr && norm_eps > 0.f && out != nullptr && ld_out >= heads * dv &&
              ld >= col_g + heads * dv, "mlstm_step: bad inputs");
  ILB_REQUIRE(dtype == kF32 || width % 8 != 0 || (((uintptr_t)x % 16 == 0) && ((uintptr_t)w_gates % 16 == 0)), "mlstm_step: rows must start on 16-byte boundaries");
  const size_t smem = sizeof(float) * dv;
  ILB_REQUIRE(smem <= 32 * 1024, "mlstm_step: %d value channels a head are too many", dv);
  if (n_seqs == 0) return 0;
  const MlstmStep q{p, x, width, w_gates, col_g, norm_w, norm_eps, out, ld_out};
  const bool vec = dv % 4 == 0 && (uintptr_t)state % 16 == 0;
#define ILB_ST(TI, V) ilb::launch(mlstm_step_kernel<TI, V>, dim3(heads, n_seqs), dim3(kStepThreads), smem, stream, q)
  if (dtype == kF32) { if (vec) ILB_ST(float, 4); else ILB_ST(float, 1); }
  else { if (vec) ILB_ST(__nv_bfloat16, 4); else ILB_ST(__nv_bfloat16, 1); }
#undef ILB_ST
  return check_launch("mlstm_step");
}

// ---------------------------------------------------------------- long portions, 64 tokens at a time
constexpr int kChunk = 64;            // tokens of a chunk
constexpr int kTileCols = 64;         // value columns per block
constexpr int kHalfCols = 32;         // ... and per warp
constexpr int kChunkThreads = 256;    // eight warps
constexpr int kLdV = kTileCols + 8;   // row stride of tiles with 64 columns in shared memory (elements)

// a = hi + mid + lo exactly, each a bfloat16 (8 + 8 + 8 significant bits); two numbers at a time
__device__ __forceinline__ void split3(float x, float y, uint32_t& hi, uint32_t& mid, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float rx = x - __low2float(h), ry = y - __high2float(h);
  const __nv_bfloat162 m = __floats2bfloat162_rn(rx, ry);
  const __nv_bfloat162 l = __floats2bfloat162_rn(rx - __low2float(m), ry - __high2float(m));
  hi = *reinterpret_cast<const uint32_t*>(&h);
  mid = *reinterpret_cast<const uint32_t*>(&m);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

struct ChunkScratch {
  float* state;      // [chunks, heads, d, dv]: (1) a chunk's own contribution, (2) what comes into it
  float* norm;       // [chunks, heads, d]
  float* max;        // [chunks, heads]: (1) the chunk's own maximum, (2) the one that comes in
  float* sum;        // [chunks, heads]: the sum of its log forget gates
};

// What a chunk's tokens share, in shared memory: log gates, prefix sums of the forget gates, prefix maxima of i - F.
struct ChunkGates { float i[kChunk], F[kChunk], M[kChunk]; };

// One warp: tokens lane and lane + 32 of the chunk (t0 .. t0 + n - 1); tokens past the end add nothing.
__device__ __forceinline__ void chunk_gates(const MlstmParams& p, int h, int t0, int n, ChunkGates& g) {
  const int lane = threadIdx.x & 31;
  const float bi = p.bias_i[h], bf = p.bias_f[h];
  float carry_f = 0.f, carry_m = -INFINITY;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int t = half * 32 + lane;
    const bool on = t < n;
    const float* row = p.gates + (size_t)(t0 + (on ? t : 0)) * p.ld_g + h;
    const float i = on ? log_gate_in(row[0] + bi, p.cap) : -INFINITY;
    float F = on ? log_gate_forget(row[p.heads] + bf, p.cap) : 0.f;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, F, o);
      if (lane >= o) F += v;
    }
    F += carry_f;
    float M = i - F;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, M, o);
      if (lane >= o) M = fmaxf(M, v);
    }
    M = fmaxf(M, carry_m);
    carry_f = __shfl_sync(0xffffffffu, F, 31);
    carry_m = __shfl_sync(0xffffffffu, M, 31);
    g.i[t] = i; g.F[t] = F; g.M[t] = M;
  }
}

// rows t0 .. t0 + n - 1, columns col .. col + width - 1 of proj into dst [64][ld_dst], zeros beyond n and width up to `padded` columns
__device__ __forceinline__ void load_tile(const __nv_bfloat16* __restrict__ proj, int ld, int t0, int n, int col, int width, int padded,
                                          __nv_bfloat16* dst, int ld_dst, bool vec) {
  const int p8 = padded / 8;
  constexpr int kFlight = 4;                             // units whose loads are in flight together
  for (int u0 = threadIdx.x; u0 < kChunk * p8; u0 += kFlight * kChunkThreads) {
    uint4 v[kFlight];
#pragma unroll
    for (int f = 0; f < kFlight; ++f) {
      const int u = u0 + f * kChunkThreads, r = u / p8, c = (u % p8) * 8;
      v[f] = make_uint4(0u, 0u, 0u, 0u);
      if (r < n && c < width) {
        const __nv_bfloat16* src = proj + (size_t)(t0 + r) * ld + col + c;
        if (vec && c + 8 <= width) v[f] = __ldg(reinterpret_cast<const uint4*>(src));
        else {
          __align__(16) __nv_bfloat16 e[8];
#pragma unroll
          for (int j = 0; j < 8; ++j) e[j] = c + j < width ? src[j] : __float2bfloat16_rn(0.f);
          v[f] = *reinterpret_cast<const uint4*>(e);
        }
      }
    }
#pragma unroll
    for (int f = 0; f < kFlight; ++f) {
      const int u = u0 + f * kChunkThreads;
      if (u < kChunk * p8) *reinterpret_cast<uint4*>(dst + (u / p8) * ld_dst + (u % p8) * 8) = v[f];
    }
  }
}

__host__ __device__ constexpr int padded16(int n) { return (n + 15) / 16 * 16; }
static inline size_t local_smem(int d) { return (size_t)2 * kChunk * (padded16(d) + 8 + kLdV); }
static inline size_t out_smem(int d) { return (size_t)2 * (2 * kChunk * (padded16(d) + 8) + kChunk * kLdV + 3 * padded16(d) * kLdV); }

// (1) chunk_state = sum_s (w_s k_s) v_s^T with w_s = exp(F_L - F_s + i_s - m), m = max_s (F_L - F_s + i_s); chunk_norm the same
// with k alone.  A block per (chunk, head, 64 columns); a warp takes 16 rows and 32 of the columns at a time.
__global__ void __launch_bounds__(kChunkThreads)
mlstm_local_kernel(const MlstmParams p, const ChunkScratch s, int vec) {
  ilb::pdl_launch_dependents();
  ilb::pdl_wait();
  extern __shared__ __align__(16) __nv_bfloat16 tiles[];
  __shared__ ChunkGates g;
  __shared__ float w[kChunk];
  const int DP = padded16(p.d), ldk = DP + 8;
  __nv_bfloat16* Ks = tiles;                             // [64][ldk]
  __nv_bfloat16* Vs = Ks + kChunk * ldk;                 // [64][kLdV]
  int seq, ci;
  if (!find_tile(p.cu_q, p.n_seqs, kChunk, blockIdx.x, seq, ci)) return;
  const int h = blockIdx.y, c0 = blockIdx.z * kTileCols;
  const int t0 = p.cu_q[seq] + ci * kChunk, n = min(kChunk, p.cu_q[seq + 1] - t0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, t4 = lane & 3;
  const __nv_bfloat16* proj = reinterpret_cast<const __nv_bfloat16*>(p.proj);
  load_tile(proj, p.ld, t0, n, p.col_k + h * p.d, p.d, DP, Ks, ldk, vec);
  load_tile(proj, p.ld, t0, n, p.col_v + h * p.dv + c0, min(kTileCols, p.dv - c0), kTileCols, Vs, kLdV, vec);
  if (warp == 0) chunk_gates(p, h, t0, n, g);
  __syncthreads();
  const float FL = g.F[kChunk - 1], m = FL + g.M[kChunk - 1];
  if (tid < kChunk) w[tid] = tid < n ? expf(FL - g.F[tid] + g.i[tid] - m) : 0.f;
  __syncthreads();
  const size_t at = (size_t)blockIdx.x * p.heads + h;
  if (blockIdx.z == 0) {
    for (int r = tid; r < p.d; r += kChunkThreads) {
      float v = 0.f;
      for (int t = 0; t < n; ++t) v = fmaf(w[t], __bfloat162float(Ks[t * ldk + r]), v);
      s.norm[at * p.d + r] = v;
    }
    if (tid == 0) { s.max[at] = m; s.sum[at] = FL; }
  }
  float wt[kChunk / 16][4];                              // weights of this lane's tokens: 16 kb + 2 t4, + 1, + 8, + 9
#pragma unroll
  for (int kb = 0; kb < kChunk / 16; ++kb) {
    wt[kb][0] = w[16 * kb + 2 * t4]; wt[kb][1] = w[16 * kb + 2 * t4 + 1];
    wt[kb][2] = w[16 * kb + 2 * t4 + 8]; wt[kb][3] = w[16 * kb + 2 * t4 + 9];
  }
  float* dst = s.state + at * p.d * p.dv;
  for (int unit = warp; unit < DP / 8; unit += kChunkThreads / 32) {
    const int r0 = (unit >> 1) * 16, n0 = (unit & 1) * kHalfCols;
    if (c0 + n0 >= p.dv) continue;
    float acc[kHalfCols / 8][4];
#pragma unroll
    for (int i = 0; i < kHalfCols / 8; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
#pragma unroll
    for (int kb = 0; kb < kChunk / 16; ++kb) {
      // A = K^T (rows: key channels, inner: tokens) from [token][channel]: transposed 8 x 8 blocks
      uint32_t k[4];
      ldmatrix_x4_trans(smem_u32(Ks + (16 * kb + (lane & 7) + ((lane >> 4) & 1) * 8) * ldk + r0 + ((lane >> 3) & 1) * 8), k[0], k[1], k[2], k[3]);
      uint32_t hi[4], mid[4], lo[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float wa = wt[kb][(e >> 1) * 2], wb = wt[kb][(e >> 1) * 2 + 1];
        split3(__uint_as_float(k[e] << 16) * wa, __uint_as_float(k[e] & 0xFFFF0000u) * wb, hi[e], mid[e], lo[e]);
      }
#pragma unroll
      for (int nd = 0; nd < kHalfCols / 16; ++nd) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(smem_u32(Vs + (16 * kb + (lane & 7) + ((lane >> 3) & 1) * 8) * kLdV + n0 + nd * 16 + (lane >> 4) * 8), b0, b1, b2, b3);
        mma_16816(acc[2 * nd], lo, b0, b1);
        mma_16816(acc[2 * nd + 1], lo, b2, b3);
        mma_16816(acc[2 * nd], mid, b0, b1);
        mma_16816(acc[2 * nd + 1], mid, b2, b3);
        mma_16816(acc[2 * nd], hi, b0, b1);
        mma_16816(acc[2 * nd + 1], hi, b2, b3);
      }
    }
    const int ra = r0 + (lane >> 2), rb = ra + 8;
#pragma unroll
    for (int i = 0; i < kHalfCols / 8; ++i) {
      const int c = c0 + n0 + i * 8 + 2 * t4;
      if (p.dv % 2 == 0) {
        if (c < p.dv) {
          if (ra < p.d) *reinterpret_cast<float2*>(dst + (size_t)ra * p.dv + c) = make_float2(acc[i][0], acc[i][1]);
          if (rb < p.d) *reinterpret_cast<float2*>(dst + (size_t)rb * p.dv + c) = make_float2(acc[i][2], acc[i][3]);
        }
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = e < 2 ? ra : rb, cc = c + (e & 1);
          if (r < p.d && cc < p.dv) dst[(size_t)r * p.dv + cc] = acc[i][e];
        }
      }
    }
  }
}

// (2) The chunks of a sequence one after the other: afterwards chunk_state, chunk_norm and chunk_max hold what comes INTO the
// chunk, and the slot holds state and normaliser after the last one (m stays: every block here reads it).  A thread owns an
// element (blocks beyond the state's: of the normaliser).
constexpr int kCarryBatch = 16;       // chunks whose loads are in flight together
constexpr int kCarryTile = 32;        // chunks whose factors are in shared memory at a time

__global__ void __launch_bounds__(256)
mlstm_carry_kernel(const MlstmParams p, const ChunkScratch s, float* __restrict__ max_in, int state_blocks) {
  ilb::pdl_launch_dependents();
  ilb::pdl_wait();
  __shared__ float keep[kCarryTile], add[kCarryTile];
  const int h = blockIdx.y, seq = blockIdx.z, lane = threadIdx.x & 31;
  const bool is_norm = (int)blockIdx.x >= state_blocks;
  const int size = is_norm ? p.d : p.d * p.dv;
  const int e = ((int)blockIdx.x - (is_norm ? state_blocks : 0)) * 256 + threadIdx.x;
  int first = 0;
  for (int i = 0; i < seq; ++i) first += (p.cu_q[i + 1] - p.cu_q[i] + kChunk - 1) / kChunk;
  const int n = (p.cu_q[seq + 1] - p.cu_q[seq] + kChunk - 1) / kChunk;
  const int slot = p.slots[seq];
  float m = slot >= 0 ? p.max[(size_t)slot * p.heads + h] : 0.f;      // (kept by the first warp)
  float* own = slot >= 0 ? (is_norm ? p.norm : p.state) + ((size_t)slot * p.heads + h) * size + e : nullptr;
  float* at = (is_norm ? s.norm : s.state) + e;
  const bool live = e < size;
  float run = own != nullptr && live ? *own : 0.f;
  for (int t0 = 0; t0 < n; t0 += kCarryTile) {
    const int tn = min(kCarryTile, n - t0);
    __syncthreads();                                     // everyone is done with the tile before
    if (threadIdx.x < 32) {
      const size_t c = (size_t)(first + t0 + min(lane, tn - 1)) * p.heads + h;
      const float lm = s.max[c], ls = s.sum[c];
      float before = m, after = m;
      for (int j = 0; j < tn; ++j) {
        const float next = fmaxf(__shfl_sync(0xffffffffu, ls, j) + m, __shfl_sync(0xffffffffu, lm, j));
        if (lane == j) { before = m; after = next; }
        m = next;
      }
      if (lane < tn) {
        keep[lane] = expf(ls + before - after);
        add[lane] = expf(lm - after);
        if (blockIdx.x == 0) max_in[c] = before;
      }
    }
    __syncthreads();
    for (int c0 = 0; c0 < tn; c0 += kCarryBatch) {
      float local[kCarryBatch];
#pragma unroll
      for (int j = 0; j < kCarryBatch; ++j)
        local[j] = live && c0 + j < tn ? at[((size_t)(first + t0 + c0 + j) * p.heads + h) * size] : 0.f;
#pragma unroll
      for (int j = 0; j < kCarryBatch; ++j) {
        if (c0 + j < tn) {
          if (live) at[((size_t)(first + t0 + c0 + j) * p.heads + h) * size] = run;
          run = fmaf(keep[c0 + j], run, add[c0 + j] * local[j]);
        }
      }
    }
  }
  if (own != nullptr && live && n > 0) *own = run;
}

// (3) A block per (chunk, head, 64 columns); warp w owns tokens 16 (w % 4) .. + 15 of the chunk and 32 of the columns.
__global__ void __launch_bounds__(kChunkThreads)
mlstm_out_kernel(const MlstmParams p, const ChunkScratch s, const float* __restrict__ max_in, float* __restrict__ y, int vec) {
  ilb::pdl_launch_dependents();
  ilb::pdl_wait();
  extern __shared__ __align__(16) __nv_bfloat16 tiles[];
  __shared__ ChunkGates g;
  __shared__ float nq[kChunk], ms[kChunk];
  const int DP = padded16(p.d), ldk = DP + 8;
  __nv_bfloat16* Qs = tiles;                             // [64][ldk]
  __nv_bfloat16* Ks = Qs + kChunk * ldk;                 // [64][ldk]
  __nv_bfloat16* Vs = Ks + kChunk * ldk;                 // [64][kLdV]
  __nv_bfloat16* Ss = Vs + kChunk * kLdV;                // [3][DP][kLdV]: the incoming state's pieces
  int seq, ci;
  if (!find_tile(p.cu_q, p.n_seqs, kChunk, blockIdx.x, seq, ci)) return;
  const int h = blockIdx.y, c0 = blockIdx.z * kTileCols;
  const int tok0 = p.cu_q[seq], q_len = p.cu_q[seq + 1] - tok0, t0 = tok0 + ci * kChunk, n = min(kChunk, q_len - ci * kChunk);
  const int tid = threadIdx.x, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3;
  const int warp = (tid >> 5) & 3, n0 = (tid >> 7) * kHalfCols;      // rows and columns of this warp
  const __nv_bfloat16* proj = reinterpret_cast<const __nv_bfloat16*>(p.proj);
  const size_t at = (size_t)blockIdx.x * p.heads + h;
  const float m_in = max_in[at];
  load_tile(proj, p.ld, t0, n, p.col_q + h * p.d, p.d, DP, Qs, ldk, vec);
  load_tile(proj, p.ld, t0, n, p.col_k + h * p.d, p.d, DP, Ks, ldk, vec);
  load_tile(proj, p.ld, t0, n, p.col_v + h * p.dv + c0, min(kTileCols, p.dv - c0), kTileCols, Vs, kLdV, vec);
  {
    const float* S = s.state + at * p.d * p.dv;
    const int plane = DP * kLdV;
    const bool fours = p.dv % 4 == 0;
    constexpr int kFlight = 8;                           // units of four columns whose loads are in flight together
    for (int u0 = tid; u0 < DP * (kTileCols / 4); u0 += kFlight * kChunkThreads) {
      float4 v[kFlight];
#pragma unroll
      for (int f = 0; f < kFlight; ++f) {
        const int u = u0 + f * kChunkThreads, r = u / (kTileCols / 4), c = c0 + (u % (kTileCols / 4)) * 4;
        v[f] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (r < p.d && c < p.dv) {
          const float* src = S + (size_t)r * p.dv + c;
          if (fours) v[f] = *reinterpret_cast<const float4*>(src);
          else {
            v[f].x = src[0];
            if (c + 1 < p.dv) v[f].y = src[1];
            if (c + 2 < p.dv) v[f].z = src[2];
            if (c + 3 < p.dv) v[f].w = src[3];
          }
        }
      }
#pragma unroll
      for (int f = 0; f < kFlight; ++f) {
        const int u = u0 + f * kChunkThreads;
        if (u < DP * (kTileCols / 4)) {
          uint2 hi, mid, lo;
          split3(v[f].x, v[f].y, hi.x, mid.x, lo.x);
          split3(v[f].z, v[f].w, hi.y, mid.y, lo.y);
          __nv_bfloat16* at = Ss + (u / (kTileCols / 4)) * kLdV + (u % (kTileCols / 4)) * 4;
          *reinterpret_cast<uint2*>(at) = hi;
          *reinterpret_cast<uint2*>(at + plane) = mid;
          *reinterpret_cast<uint2*>(at + 2 * plane) = lo;
        }
      }
    }
  }
  if (tid < 32) chunk_gates(p, h, t0, n, g);
  __syncthreads();
  if (tid < kChunk) ms[tid] = g.F[tid] + fmaxf(m_in, g.M[tid]);
  {   // n_in . q: four threads a token
    const int t = tid >> 2, part = tid & 3;
    const float* nin = s.norm + at * p.d;
    float v = 0.f;
#pragma unroll 8
    for (int r = part; r < p.d; r += 4) v = fmaf(nin[r], __bfloat162float(Qs[t * ldk + r]), v);
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    if (part == 0) nq[t] = v;
  }
  __syncthreads();
  const int ra = warp * 16 + g8, rb = ra + 8;            // this lane's two tokens
  if (warp * 16 < n && c0 + n0 < p.dv) {
    float P[kChunk / 8][4], O[kHalfCols / 8][4];
#pragma unroll
    for (int i = 0; i < kChunk / 8; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) P[i][e] = 0.f;
#pragma unroll
    for (int i = 0; i < kHalfCols / 8; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) O[i][e] = 0.f;
    for (int kb = 0; kb < DP / 16; ++kb) {
      uint32_t a[4];
      ldmatrix_x4(smem_u32(Qs + (warp * 16 + (lane & 15)) * ldk + kb * 16 + (lane >> 4) * 8), a[0], a[1], a[2], a[3]);
      // scores against the chunk's keys ([token][channel] as the column operand)
#pragma unroll
      for (int nd = 0; nd < kChunk / 16; ++nd) {
        if (nd * 16 <= warp * 16 + 15) {
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4(smem_u32(Ks + (nd * 16 + (lane & 7) + (lane >> 4) * 8) * ldk + kb * 16 + ((lane >> 3) & 1) * 8), b0, b1, b2, b3);
          mma_16816(P[2 * nd], a, b0, b1);
          mma_16816(P[2 * nd + 1], a, b2, b3);
        }
      }
      // the incoming state's read-out
#pragma unroll
      for (int piece = 2; piece >= 0; --piece) {
        const __nv_bfloat16* S = Ss + piece * DP * kLdV + n0;
#pragma unroll
        for (int nd = 0; nd < kHalfCols / 16; ++nd) {
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4_trans(smem_u32(S + (kb * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kLdV + nd * 16 + (lane >> 4) * 8), b0, b1, b2, b3);
          mma_16816(O[2 * nd], a, b0, b1);
          mma_16816(O[2 * nd + 1], a, b2, b3);
        }
      }
    }
    const float ma = ms[ra], mb = ms[rb], Fa = g.F[ra] - ma, Fb = g.F[rb] - mb;
    const float ga = __expf(Fa + m_in) * p.q_scale, gb = __expf(Fb + m_in) * p.q_scale;
#pragma unroll
    for (int i = 0; i < kHalfCols / 8; ++i) { O[i][0] *= ga; O[i][1] *= ga; O[i][2] *= gb; O[i][3] *= gb; }
    float suma = 0.f, sumb = 0.f;
#pragma unroll
    for (int i = 0; i < kChunk / 8; ++i) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = i * 8 + 2 * t4 + e;
        const float w = g.i[t] - g.F[t];
        P[i][e] = t <= ra ? P[i][e] * p.q_scale * __expf(Fa + w) : 0.f;
        P[i][2 + e] = t <= rb ? P[i][2 + e] * p.q_scale * __expf(Fb + w) : 0.f;
        suma += P[i][e];
        sumb += P[i][2 + e];
      }
    }
    suma += __shfl_xor_sync(0xffffffffu, suma, 1); suma += __shfl_xor_sync(0xffffffffu, suma, 2);
    sumb += __shfl_xor_sync(0xffffffffu, sumb, 1); sumb += __shfl_xor_sync(0xffffffffu, sumb, 2);
#pragma unroll
    for (int kb = 0; kb < kChunk / 16; ++kb) {
      if (kb <= warp) {
        uint32_t hi[4], mid[4], lo[4];
        split3(P[2 * kb][0], P[2 * kb][1], hi[0], mid[0], lo[0]);
        split3(P[2 * kb][2], P[2 * kb][3], hi[1], mid[1], lo[1]);
        split3(P[2 * kb + 1][0], P[2 * kb + 1][1], hi[2], mid[2], lo[2]);
        split3(P[2 * kb + 1][2], P[2 * kb + 1][3], hi[3], mid[3], lo[3]);
#pragma unroll
        for (int nd = 0; nd < kHalfCols / 16; ++nd) {
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4_trans(smem_u32(Vs + (16 * kb + (lane & 7) + ((lane >> 3) & 1) * 8) * kLdV + n0 + nd * 16 + (lane >> 4) * 8), b0, b1, b2, b3);
          mma_16816(O[2 * nd], lo, b0, b1);
          mma_16816(O[2 * nd + 1], lo, b2, b3);
          mma_16816(O[2 * nd], mid, b0, b1);
          mma_16816(O[2 * nd + 1], mid, b2, b3);
          mma_16816(O[2 * nd], hi, b0, b1);
          mma_16816(O[2 * nd + 1], hi, b2, b3);
        }
      }
    }
    const float da = 1.0f / (fmaxf(fabsf(fmaf(ga, nq[ra], suma)), expf(-ma)) + p.eps);
    const float db = 1.0f / (fmaxf(fabsf(fmaf(gb, nq[rb], sumb)), expf(-mb)) + p.eps);
    const int inner = p.heads * p.dv;
    float* ya = y + (size_t)(t0 + ra) * inner + (size_t)h * p.dv;
    float* yb = y + (size_t)(t0 + rb) * inner + (size_t)h * p.dv;
#pragma unroll
    for (int i = 0; i < kHalfCols / 8; ++i) {
      const int c = c0 + n0 + i * 8 + 2 * t4;
      if (p.dv % 2 == 0) {
        if (c < p.dv) {
          if (ra < n) *reinterpret_cast<float2*>(ya + c) = make_float2(O[i][0] * da, O[i][1] * da);
          if (rb < n) *reinterpret_cast<float2*>(yb + c) = make_float2(O[i][2] * db, O[i][3] * db);
        }
      } else {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          if (c + e < p.dv) {
            if (ra < n) ya[c + e] = O[i][e] * da;
            if (rb < n) yb[c + e] = O[i][2 + e] * db;
          }
        }
      }
    }
  }
  // nobody reads the slot's maximum in this launch: the sequence's last chunk leaves the new one
  if (blockIdx.z == 0 && tid == 0 && ci == (q_len - 1) / kChunk && p.slots[seq] >= 0) p.max[(size_t)p.slots[seq] * p.heads + h] = ms[n - 1];
}

// Floats of scratch that `n_chunks` chunks need.
static long long chunk_floats(int n_chunks, int heads, int d, int dv) { return (long long)n_chunks * heads * ((long long)d * dv + d + 4); }
ILB_EXPORT long long ilb_mlstm_chunk_floats(int n_chunks, int heads, int d, int dv) { return chunk_floats(n_chunks, heads, d, dv); }

// As ilb_mlstm_scan for bfloat16 projections, 64 tokens at a time; y [T, heads * dv] is divided already.  n_chunks = the sum
// over the sequences of ceil(tokens / 64).
ILB_EXPORT int ilb_mlstm_chunks(const void* proj, int ld, int col_q, int col_k, int col_v, const float* gates, int ld_g, const float* bias_i,
                                const float* bias_f, float cap, float q_scale, float eps, float* state, float* norm, float* max,
                                float* scratch, long long scratch_floats, float* y, const int* cu_q, const int* slots, int n_seqs,
                                int n_chunks, int heads, int d, int dv, cudaStream_t stream) {
  const MlstmParams p{proj, ld, col_q, col_k, col_v, gates, ld_g, bias_i, bias_f, state, norm, max, cu_q, slots, n_seqs, heads, d, dv, cap, q_scale, eps};
  if (int rc = check_sizes(p, kBF16)) return rc;
  ILB_REQUIRE(gates != nullptr && ld_g >= 2 * heads && y != nullptr && (uintptr_t)y % 8 == 0, "mlstm_chunks: bad inputs");
  ILB_REQUIRE(n_chunks >= 0 && scratch != nullptr && (uintptr_t)scratch % 16 == 0 && chunk_floats(n_chunks, heads, d, dv) <= scratch_floats, "mlstm_chunks: scratch too small");
  if (n_seqs == 0 || n_chunks == 0) return 0;
  const size_t nc = (size_t)n_chunks * heads;
  ChunkScratch s;
  s.state = scratch;
  s.norm = s.state + nc * d * dv;
  s.max = s.norm + nc * d;
  s.sum = s.max + nc;
  float* max_in = s.sum + nc;
  const int vec = ((uintptr_t)proj % 16 == 0 && ld % 8 == 0 && col_q % 8 == 0 && col_k % 8 == 0 && col_v % 8 == 0 && d % 8 == 0 && dv % 8 == 0) ? 1 : 0;
  const size_t sa = local_smem(d), sc = out_smem(d);
  static OncePerDevice once;
  if (once.first()) {
    if (cudaFuncSetAttribute(mlstm_local_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)local_smem(kMaxRows)) != cudaSuccess ||
        cudaFuncSetAttribute(mlstm_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)out_smem(kMaxRows)) != cudaSuccess) {
      once.forget();
      return fail("mlstm_chunks: cannot reserve shared memory");
    }
  }
  const int tiles = (dv + kTileCols - 1) / kTileCols;
  ilb::launch(mlstm_local_kernel, dim3(n_chunks, heads, tiles), dim3(kChunkThreads), sa, stream, p, s, vec);
  if (int rc = check_launch("mlstm_local")) return rc;
  const int sb = (d * dv + 255) / 256, nb = (d + 255) / 256;
  ilb::launch(mlstm_carry_kernel, dim3(sb + nb, heads, n_seqs), dim3(256), 0, stream, p, s, max_in, sb);
  if (int rc = check_launch("mlstm_carry")) return rc;
  ilb::launch(mlstm_out_kernel, dim3(n_chunks, heads, tiles), dim3(kChunkThreads), sc, stream, p, s, (const float*)max_in, y, vec);
  return check_launch("mlstm_out");
}

ILB_DEFINE_LAST_ERROR()
