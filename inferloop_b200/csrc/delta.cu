// The generalized delta rule: a matrix state per head that is decayed, partly read out and removed, and written to.
//
// Per head, with key channels n < d and value columns c < dv, from the projections r, k, v, a of a token and the
// low-rank map's output l (all made elsewhere):
//     w = exp(-log_decay * sigmoid(l + w0))          decay per key channel
//     g = sigmoid(a + ab)                            removal rate per key channel
//     u = k / sqrt(sum(k^2) + unit_eps)              unit key
//     S_t = diag(w) S_{t-1} - (g u)(u^T S_{t-1}) + k v^T          (both terms read the old state)
//     o_t = S_t^T r
// State [d, dv] per head, 32-bit, in the request's slot.  Columns of the state do not interact.
//
//   delta_scan   token by token, any sizes up to 256 rows.  A block owns 16 columns of a head's state of one sequence in
//                registers: eight threads a column, a warp four columns; the read-out u^T S and the output r^T S are sums
//                over the eight threads of a column.  The tokens' channel vectors are made 16 tokens at a time in shared
//                memory.  For short portions, and sizes that the two below do not take.
//   delta_prep, delta_chunks
//                long portions, 16 tokens at a time.  Inside a chunk let D_t be the product of the decays up to token t
//                (D_0 = 1 before the first) and S~_t = S_t / D_t.  With
//                    p_t = D_{t-1} u_t,   q_t = g_t u_t / D_t,   m_t = k_t / D_t,   s_t = D_t r_t
//                the recurrence reads  S~_t = S~_{t-1} - q_t z_t^T + m_t v_t^T,  z_t = S~_{t-1}^T p_t,  o_t = S~_t^T s_t, so
//                    z_t = S_0^T p_t + sum_{j<t} ((p_t.m_j) v_j - (p_t.q_j) z_j)
//                which is a triangular system over the chunk's tokens.  Its solution is linear in the chunk's incoming
//                state: Z = W S_0 + U, O = X S_0 + Y, with W, U, X, Y from the tokens alone.  delta_prep makes those (and
//                D_16 q_t, D_16 m_t, D_16) for every chunk and head side by side; delta_chunks walks a sequence's chunks with
//                a block per head and 16 columns of the state in registers: two thin products with the state, then
//                    S_16 = D_16 S_0 + sum_t (D_16 m_t) v_t^T - (D_16 q_t) z_t^T.
//                Decays of at least exp(-log_decay) a token keep every scale of a chunk within exp(16 log_decay).
//   delta_step   single tokens, everything between the projections of a layer: the low-rank map, the decay, the recurrence,
//                the norm of each head and the output gate; a block per (head, sequence) with the whole state in registers.
//
// Everything is 32-bit; the projections come in the compute dtype.  A sequence whose slot is negative (a dummy row that
// pads a recorded launch) starts from zero and stores nothing.
#include <math.h>
#include "common.cuh"
#include "sm100.cuh"

using namespace ilb;

constexpr int kCols = 16;             // columns of the state per block of the token-by-token scan
constexpr int kScanThreads = 128;
constexpr int kTile = 16;             // tokens whose vectors are in shared memory at a time

// Exact: the library's functions (the 32-bit path).  Fast: the hardware's exponential and reciprocal (a few units in the
// last place; still 32-bit arithmetic) for projections that were stored in bfloat16.
template <bool FAST> __device__ __forceinline__ float exp_t(float x) { return FAST ? __expf(x) : expf(x); }
template <bool FAST> __device__ __forceinline__ float sigmoid_t(float x) {
  return FAST ? __fdividef(1.0f, 1.0f + __expf(-x)) : 1.0f / (1.0f + expf(-x));
}

struct DeltaParams {
  const void* proj; int ld, col_r, col_k, col_v, col_a;      // [T, ld] of the compute dtype; each of r, k, a: heads * d columns, v: heads * dv
  const float* low;                                          // [T, heads * d]
  const float* w0; const float* ab;                          // [heads * d]
  float* state;                                              // [slots, heads, d, dv]
  float* y;                                                  // [T, heads * dv]
  const int* cu_q; const int* slots;
  int n_seqs, heads, d, dv;
  float log_decay, unit_eps;
};

static inline size_t scan_smem_floats(int rows) { return (size_t)5 * kTile * rows + kTile * kCols; }

template <typename TI, int Q>         // Q: groups of four rows a thread holds; 32 Q rows in all
__global__ void __launch_bounds__(kScanThreads)
delta_scan_kernel(const DeltaParams p) {
  ilb::pdl_launch_dependents();
  ilb::pdl_wait();
  constexpr bool FAST = sizeof(TI) == 2;
  constexpr int D = 32 * Q;                              // rows, padded with zeros
  extern __shared__ __align__(16) float sm[];
  float* Us = sm;                                        // [kTile][D] unit keys
  float* Ws = Us + kTile * D;                            // decays
  float* Gs = Ws + kTile * D;                            // -g u
  float* Ks = Gs + kTile * D;
  float* Rs = Ks + kTile * D;
  float* Vs = Rs + kTile * D;                            // [kTile][kCols]
  const int h = blockIdx.x, c0 = blockIdx.y * kCols, seq = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, sl = lane & 7, cl = warp * 4 + (lane >> 3), col = c0 + cl;
  const int tok0 = p.cu_q[seq], end = p.cu_q[seq + 1];
  const int slot = p.slots[seq];
  const int inner_k = p.heads * p.d, inner_v = p.heads * p.dv;
  float* own = slot >= 0 ? p.state + ((size_t)slot * p.heads + h) * p.d * p.dv : nullptr;
  const bool live = col < p.dv;
  // thread's rows: 4 (8 q + sl) + j, so that the eight threads of a column read neighbouring 16-byte pieces
  float4 S[Q];
#pragma unroll
  for (int q = 0; q < Q; ++q) {
    float v[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = 4 * (8 * q + sl) + j;
      v[j] = (own != nullptr && live && n < p.d) ? own[(size_t)n * p.dv + col] : 0.f;
    }
    S[q] = make_float4(v[0], v[1], v[2], v[3]);
  }
  const TI* proj = reinterpret_cast<const TI*>(p.proj);
  for (int t0 = tok0; t0 < end; t0 += kTile) {
    const int ts = min(kTile, end - t0);
    for (int i = threadIdx.x; i < ts * D; i += kScanThreads) {
      const int tt = i / D, n = i % D;
      float k = 0.f, w = 0.f, g = 0.f, r = 0.f;
      if (n < p.d) {
        const TI* row = proj + (size_t)(t0 + tt) * p.ld;
        const int ch = h * p.d + n;
        k = to_float(row[p.col_k + ch]);
        r = to_float(row[p.col_r + ch]);
        g = sigmoid_t<FAST>(to_float(row[p.col_a + ch]) + p.ab[ch]);
        w = exp_t<FAST>(-p.log_decay * sigmoid_t<FAST>(p.low[(size_t)(t0 + tt) * inner_k + ch] + p.w0[ch]));
      }
      Ks[i] = k; Rs[i] = r; Gs[i] = g; Ws[i] = w;
    }
    for (int i = threadIdx.x; i < ts * kCols; i += kScanThreads) {
      const int tt = i / kCols, c = c0 + i % kCols;
      Vs[i] = c < p.dv ? to_float(proj[(size_t)(t0 + tt) * p.ld + p.col_v + h * p.dv + c]) : 0.f;
    }
    __syncthreads();
    for (int tt = warp; tt < ts; tt += kScanThreads / 32) {
      float ss = 0.f;
      for (int n = lane; n < D; n += 32) ss = fmaf(Ks[tt * D + n], Ks[tt * D + n], ss);
      const float inv = 1.0f / sqrtf(warp_sum(ss) + p.unit_eps);
      for (int n = lane; n < D; n += 32) {
        const float u = Ks[tt * D + n] * inv;
        Us[tt * D + n] = u;
        Gs[tt * D + n] = -Gs[tt * D + n] * u;
      }
    }
    __syncthreads();
    for (int tt = 0; tt < ts; ++tt) {
      const float4* u4 = reinterpret_cast<const float4*>(Us + tt * D) + sl;
      const float4* w4 = reinterpret_cast<const float4*>(Ws + tt * D) + sl;
      const float4* g4 = reinterpret_cast<const float4*>(Gs + tt * D) + sl;
      const float4* k4 = reinterpret_cast<const float4*>(Ks + tt * D) + sl;
      const float4* r4 = reinterpret_cast<const float4*>(Rs + tt * D) + sl;
      float z0 = 0.f, z1 = 0.f;
#pragma unroll
      for (int q = 0; q < Q; ++q) {
        const float4 u = u4[8 * q];
        z0 = fmaf(u.x, S[q].x, z0); z1 = fmaf(u.y, S[q].y, z1); z0 = fmaf(u.z, S[q].z, z0); z1 = fmaf(u.w, S[q].w, z1);
      }
      float z = z0 + z1;
      z += __shfl_xor_sync(0xffffffffu, z, 1);
      z += __shfl_xor_sync(0xffffffffu, z, 2);
      z += __shfl_xor_sync(0xffffffffu, z, 4);
      const float v = Vs[tt * kCols + cl];
      float o0 = 0.f, o1 = 0.f;
#pragma unroll
      for (int q = 0; q < Q; ++q) {
        const float4 w = w4[8 * q], g = g4[8 * q], k = k4[8 * q], r = r4[8 * q];
        S[q].x = fmaf(w.x, S[q].x, fmaf(g.x, z, k.x * v)); S[q].y = fmaf(w.y, S[q].y, fmaf(g.y, z, k.y * v));
        S[q].z = fmaf(w.z, S[q].z, fmaf(g.z, z, k.z * v)); S[q].w = fmaf(w.w, S[q].w, fmaf(g.w, z, k.w * v));
        o0 = fmaf(r.x, S[q].x, o0); o1 = fmaf(r.y, S[q].y, o1); o0 = fmaf(r.z, S[q].z, o0); o1 = fmaf(r.w, S[q].w, o1);
      }
      float o = o0 + o1;
      o += __shfl_xor_sync(0xffffffffu, o, 1);
      o += __shfl_xor_sync(0xffffffffu, o, 2);
      o += __shfl_xor_sync(0xffffffffu, o, 4);
      if (sl == 0 && live) p.y[(size_t)(t0 + tt) * inner_v + h * p.dv + col] = o;
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
        if (n < p.d) own[(size_t)n * p.dv + col] = v[j];
      }
    }
  }
}

template <typename TI, int Q>
static int scan_launch(const DeltaParams& p, cudaStream_t stream) {
  const size_t smem = sizeof(float) * scan_smem_floats(32 * Q);
  static OncePerDevice once;
  if (smem > 48 * 1024 && once.first() &&
      cudaFuncSetAttribute(delta_scan_kernel<TI, Q>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
    once.forget();
    return fail("delta_scan: cannot reserve %zu bytes of shared memory", smem);
  }
  ilb::launch(delta_scan_kernel<TI, Q>, dim3(p.heads, (p.dv + kCols - 1) / kCols, p.n_seqs), dim3(kScanThreads), smem, stream, p);
  return check_launch("delta_scan");
}

static int check_sizes(const DeltaParams& p, int dtype) {
  ILB_REQUIRE(p.heads > 0 && p.d > 0 && p.dv > 0 && p.d <= 256, "delta rule: %d heads of %d x %d (at most 256 rows)", p.heads, p.d, p.dv);
  ILB_REQUIRE(p.n_seqs >= 0 && p.n_seqs <= 65535, "delta rule: too many sequences");
  ILB_REQUIRE(dtype == kF32 || dtype == kBF16, "delta rule: unknown dtype %d", dtype);
  ILB_REQUIRE(p.proj != nullptr && p.low != nullptr && p.w0 != nullptr && p.ab != nullptr && p.state != nullptr && p.y != nullptr,
              "delta rule: missing inputs");
  const int wk = p.heads * p.d, wv = p.heads * p.dv;
  ILB_REQUIRE(p.col_r >= 0 && p.col_k >= 0 && p.col_a >= 0 && p.col_v >= 0 && p.ld >= p.col_r + wk && p.ld >= p.col_k + wk &&
              p.ld >= p.col_a + wk && p.ld >= p.col_v + wv, "delta rule: the projection's rows are too short");
  return 0;
}

ILB_EXPORT int ilb_delta_scan(const void* proj, int dtype, int ld, int col_r, int col_k, int col_v, int col_a, const float* low,
                              const float* w0, const float* ab, float log_decay, float unit_eps, float* state, float* y,
                              const int* cu_q, const int* slots, int n_seqs, int heads, int d, int dv, cudaStream_t stream) {
  const DeltaParams p{proj, ld, col_r, col_k, col_v, col_a, low, w0, ab, state, y, cu_q, slots, n_seqs, heads, d, dv, log_decay, unit_eps};
  if (int rc = check_sizes(p, dtype)) return rc;
  if (n_seqs == 0) return 0;
  const int q = d <= 32 ? 1 : (d <= 64 ? 2 : (d <= 128 ? 4 : 8));
  if (dtype == kF32) {
    if (q == 1) return scan_launch<float, 1>(p, stream);
    if (q == 2) return scan_launch<float, 2>(p, stream);
    if (q == 4) return scan_launch<float, 4>(p, stream);
    return scan_launch<float, 8>(p, stream);
  }
  if (q == 1) return scan_launch<__nv_bfloat16, 1>(p, stream);
  if (q == 2) return scan_launch<__nv_bfloat16, 2>(p, stream);
  if (q == 4) return scan_launch<__nv_bfloat16, 4>(p, stream);
  return scan_launch<__nv_bfloat16, 8>(p, stream);
}

// ---------------------------------------------------------------- chunks
constexpr int kChunk = 16;

// Two 32-bit numbers side by side and the arithmetic on both at once (IEEE, as the scalar instructions).
__device__ __forceinline__ uint64_t pack2(float lo, float hi) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ void unpack2(uint64_t v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ float sum2(uint64_t v) {
  float lo, hi;
  unpack2(v, lo, hi);
  return lo + hi;
}

// Floats of one (chunk, head) in scratch: W, X, - D q, D m [16][KP], D [KP], then U, Y, V [16][DP]; KP rows, DP columns, padded.
__host__ __device__ __forceinline__ long long chunk_floats(int KP, int DP) { return (long long)4 * kChunk * KP + KP + (long long)3 * kChunk * DP; }
// The tensor-core form keeps W, X, D m, - D q as three bfloat16 pieces each (x = hi + mid + lo exactly), in the order in which the
// lanes of a warp hold the operands of mma.m16n8k16, 16 bytes a lane:
//   per 16 rows of the state: W, X (A operands, 16 tokens x 16 rows), pieces hi mid lo each       6 x 512 bytes
//   then per 16 rows:         D m, - D q (B operands, 16 tokens x 2 x 8 rows), hi mid lo each      6 x 512 bytes
//   then D [KP]; then per 16 columns: U, Y [16][16] in 32-bit, and V transposed (A operand, 16 columns x 16 tokens; exact), 512 bytes
constexpr int kFragFloats = 128;                         // 512 bytes
constexpr int kColFloats = 2 * kChunk * kCols + kFragFloats;
__host__ __device__ constexpr int row_floats_mma(int KP) { return (KP / 16) * 12 * kFragFloats + KP; }
__host__ __device__ __forceinline__ long long chunk_floats_mma(int KP, int DP) { return row_floats_mma(KP) + (long long)(DP / kCols) * kColFloats; }
__host__ __device__ __forceinline__ int padded_cols(int dv) { return (dv + kCols - 1) / kCols * kCols; }
static inline int padded_rows(int d) { return d <= 64 ? 64 : (d <= 128 ? 128 : 256); }

// which sequence, and which of its chunks, block `b` works on; false: none
__device__ __forceinline__ bool find_chunk(const int* __restrict__ cu_q, int n_seqs, int b, int& seq, int& index) {
  for (seq = 0; seq < n_seqs; ++seq) {
    const int n = (cu_q[seq + 1] - cu_q[seq] + kChunk - 1) / kChunk;
    if (b < n) { index = b; return true; }
    b -= n;
  }
  return false;
}

// (x, y) = hi + mid + lo exactly, each a pair of bfloat16.
__device__ __forceinline__ void split3(float x, float y, uint32_t& hi, uint32_t& mid, uint32_t& lo) {
  hi = pack_bf16(x, y);
  x -= __uint_as_float(hi << 16); y -= __uint_as_float(hi & 0xFFFF0000u);
  mid = pack_bf16(x, y);
  x -= __uint_as_float(mid << 16); y -= __uint_as_float(mid & 0xFFFF0000u);
  lo = pack_bf16(x, y);
}

constexpr int kPrepThreads = 128;

static inline size_t prep_smem_floats(int KP, int DP) { return (size_t)4 * kChunk * (KP + 4) + (size_t)kChunk * DP + 4 * kChunk * kChunk; }

template <typename TI>
__global__ void __launch_bounds__(kPrepThreads, 4)
delta_prep_kernel(const DeltaParams p, float* __restrict__ scratch, int KP) {
  ilb::pdl_wait();
  constexpr bool FAST = sizeof(TI) == 2;
  extern __shared__ __align__(16) float sm[];
  const int DP = padded_cols(p.dv), ld = KP + 4;
  float* P = sm;                                         // [16][ld] each
  float* R = P + kChunk * ld;
  float* Qv = R + kChunk * ld;
  float* M = Qv + kChunk * ld;
  float* V = M + kChunk * ld;                            // [16][DP]
  float* AC = V + kChunk * DP;                           // [16][16][2]: - p.q (j < t), - s.q (j <= t); zero elsewhere
  float* BE = AC + 2 * kChunk * kChunk;                  //              p.m (j < t), s.m (j <= t)
  __shared__ float inv_norm[kChunk], Ds[256];
  int seq, ci;
  if (!find_chunk(p.cu_q, p.n_seqs, blockIdx.x, seq, ci)) return;
  const int h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int tok0 = p.cu_q[seq] + ci * kChunk, ts = min(kChunk, p.cu_q[seq + 1] - tok0);
  const int inner_k = p.heads * p.d;
  const TI* proj = reinterpret_cast<const TI*>(p.proj);
  // FAST: the tensor-core form's layout, else the plain one
  float* out = scratch + ((size_t)blockIdx.x * p.heads + h) * (FAST ? chunk_floats_mma(KP, DP) : chunk_floats(KP, DP));
  float* outW = out; float* outX = outW + kChunk * KP; float* outQ = outX + kChunk * KP; float* outM = outQ + kChunk * KP;
  float* outD = FAST ? out + (KP / 16) * 12 * kFragFloats : outM + kChunk * KP;
  float* outU = outD + KP; float* outY = outU + kChunk * DP; float* outV = outY + kChunk * DP;

  // the raw inputs of a channel, all in flight together; this thread's first channel's before anything is waited for
  TI r_raw[kChunk], a_raw[kChunk];
  float l_raw[kChunk];
  auto fetch = [&](int n) {
    const int ch = h * p.d + (n < p.d ? n : 0);
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      const int tt = tok0 + (t < ts ? t : 0);
      const TI* row = proj + (size_t)tt * p.ld;
      r_raw[t] = row[p.col_r + ch];
      a_raw[t] = row[p.col_a + ch];
      l_raw[t] = p.low[(size_t)tt * inner_k + ch];
    }
  };
  fetch(tid);
  for (int n = tid; n < KP; n += kPrepThreads) {
#pragma unroll
    for (int t = 0; t < kChunk; ++t)
      M[t * ld + n] = (n < p.d && t < ts) ? to_float(proj[(size_t)(tok0 + t) * p.ld + p.col_k + h * p.d + n]) : 0.f;
  }
  for (int c = tid; c < DP; c += kPrepThreads) {
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      const float v = (c < p.dv && t < ts) ? to_float(proj[(size_t)(tok0 + t) * p.ld + p.col_v + h * p.dv + c]) : 0.f;
      V[t * DP + c] = v;
      if constexpr (!FAST) outV[t * DP + c] = v;
    }
  }
  __syncthreads();
  for (int t = warp; t < kChunk; t += kPrepThreads / 32) {
    float ss = 0.f;
    for (int n = lane; n < KP; n += 32) ss = fmaf(M[t * ld + n], M[t * ld + n], ss);
    ss = warp_sum(ss);
    if (lane == 0) inv_norm[t] = 1.0f / sqrtf(ss + p.unit_eps);
  }
  __syncthreads();
  for (int n = tid; n < KP; n += kPrepThreads) {
    const bool live = n < p.d;
    const int ch = h * p.d + (live ? n : 0);
    const float w0 = p.w0[ch], ab = p.ab[ch];
    if (n != tid) fetch(n);
    float D = 1.f;
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      const bool on = live && t < ts;
      const float k = M[t * ld + n], u = k * inv_norm[t];
      const float w = on ? exp_t<FAST>(-p.log_decay * sigmoid_t<FAST>(l_raw[t] + w0)) : 1.f;
      const float g = on ? sigmoid_t<FAST>(to_float(a_raw[t]) + ab) : 0.f;
      P[t * ld + n] = D * u;
      D *= w;
      const float inv = FAST ? __fdividef(1.0f, D) : 1.0f / D;
      Qv[t * ld + n] = g * u * inv;
      M[t * ld + n] = k * inv;
      R[t * ld + n] = on ? D * to_float(r_raw[t]) : 0.f;
    }
    outD[n] = D;
    Ds[n] = D;
  }
  __syncthreads();
  {   // rows of P and R against rows of Q and M: a thread takes four rows and one column of both
    const int j = tid & 15, rg = tid >> 4;               // rows 4 (rg & 3) .. + 3 of P (rg < 4) or of R
    const float* rows = (rg < 4 ? P : R) + (size_t)(rg & 3) * 4 * ld;
    uint64_t x2[4], y2[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) { x2[i] = 0; y2[i] = 0; }
#pragma unroll 4
    for (int n = 0; n < KP; n += 4) {
      const ulonglong2 q = *reinterpret_cast<const ulonglong2*>(Qv + j * ld + n), m = *reinterpret_cast<const ulonglong2*>(M + j * ld + n);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(rows + i * ld + n);
        x2[i] = fma2(v.y, q.y, fma2(v.x, q.x, x2[i]));
        y2[i] = fma2(v.y, m.y, fma2(v.x, m.x, y2[i]));
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int t = 4 * (rg & 3) + i;
      const bool keep = rg < 4 ? j < t : j <= t;
      AC[(t * kChunk + j) * 2 + (rg < 4 ? 0 : 1)] = keep ? -sum2(x2[i]) : 0.f;
      BE[(t * kChunk + j) * 2 + (rg < 4 ? 0 : 1)] = keep ? sum2(y2[i]) : 0.f;
    }
  }
  __syncthreads();
  // The pairs of row t, columns 0 .. t, from shared memory.  (The fence keeps the compiler from holding whole matrices in
  // registers across the columns' loop.)
  auto pairs = [&](const float* m, int t, uint64_t (&r)[kChunk]) {
    asm volatile("" ::: "memory");
#pragma unroll
    for (int j = 0; j < kChunk; j += 2) {
      if (j <= t) {
        const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(m + (t * kChunk + j) * 2);
        r[j] = v.x; r[j + 1] = v.y;
      }
    }
  };
  for (int n = tid; n < KP; n += kPrepThreads) {         // W = (I + A)^-1 P,  X = R - C W, column by column
    float w[kChunk];
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      uint64_t ac[kChunk], vx = pack2(P[t * ld + n], R[t * ld + n]);
      pairs(AC, t, ac);
#pragma unroll
      for (int j = 0; j < t; ++j) vx = fma2(ac[j], pack2(w[j], w[j]), vx);
      float c, zero, x;
      unpack2(ac[t], zero, c);
      unpack2(vx, w[t], x);
      x = fmaf(c, w[t], x);
      if constexpr (FAST) { P[t * ld + n] = w[t]; R[t * ld + n] = x; }      // (this thread's own column: nobody else reads it any more)
      else { outW[t * KP + n] = w[t]; outX[t * KP + n] = x; }
    }
    const float D = Ds[n];
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      if constexpr (FAST) { Qv[t * ld + n] *= -D; M[t * ld + n] *= D; }
      else { outQ[t * KP + n] = -Qv[t * ld + n] * D; outM[t * KP + n] = M[t * ld + n] * D; }
    }
  }
  for (int c0 = tid; c0 < DP; c0 += kPrepThreads) {      // U = (I + A)^-1 B V,  Y = E V - C U
    float u[kChunk], v[kChunk];
#pragma unroll
    for (int t = 0; t < kChunk; ++t) v[t] = V[t * DP + c0];
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      uint64_t ac[kChunk], be[kChunk], sy = 0;
      pairs(AC, t, ac);
      pairs(BE, t, be);
#pragma unroll
      for (int j = 0; j < t; ++j) sy = fma2(ac[j], pack2(u[j], u[j]), fma2(be[j], pack2(v[j], v[j]), sy));
      float c, e, zero, y;
      unpack2(ac[t], zero, c);
      unpack2(be[t], zero, e);
      unpack2(sy, u[t], y);
      y = fmaf(c, u[t], fmaf(e, v[t], y));
      if constexpr (FAST) {
        float* uy = outU + (c0 / kCols) * kColFloats + t * kCols + c0 % kCols;
        uy[0] = u[t]; uy[kChunk * kCols] = y;
      } else {
        outU[t * DP + c0] = u[t]; outY[t * DP + c0] = y;
      }
    }
  }
  if constexpr (FAST) {
    __syncthreads();
    uint4* frag = reinterpret_cast<uint4*>(out);
    // eight values of a lane, cut into three pieces, 16 bytes each
    auto emit = [&](size_t at, const float (&x)[8]) {
      uint32_t hi[4], mid[4], lo[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) split3(x[2 * i], x[2 * i + 1], hi[i], mid[i], lo[i]);
      frag[at] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      frag[at + 32] = make_uint4(mid[0], mid[1], mid[2], mid[3]);
      frag[at + 64] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    };
    const int slices = KP / 16;
    for (int i = tid; i < slices * 4 * 32; i += kPrepThreads) {
      const int ln = i & 31, what = (i >> 5) & 3, ks = i >> 7, g = ln >> 2, t4 = ln & 3;
      float x[8];
      if (what < 2) {                                    // A operand: rows are tokens g and g + 8, columns the state's rows
        const float* m = (what == 0 ? P : R) + ks * 16 + 2 * t4;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          x[e] = m[g * ld + e]; x[2 + e] = m[(g + 8) * ld + e]; x[4 + e] = m[g * ld + 8 + e]; x[6 + e] = m[(g + 8) * ld + 8 + e];
        }
        emit((size_t)((ks * 2 + what) * 3) * 32 + ln, x);
      } else {                                           // B operand: rows are tokens, columns the state's rows g and g + 8
        const float* m = (what == 2 ? M : Qv) + ks * 16 + g;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          x[e] = m[(2 * t4 + e) * ld]; x[2 + e] = m[(2 * t4 + 8 + e) * ld]; x[4 + e] = m[(2 * t4 + e) * ld + 8]; x[6 + e] = m[(2 * t4 + 8 + e) * ld + 8];
        }
        emit((size_t)(slices * 6 + (ks * 2 + what - 2) * 3) * 32 + ln, x);
      }
    }
    for (int i = tid; i < DP / 16 * 32; i += kPrepThreads) {
      const int ln = i & 31, g = ln >> 2, t4 = ln & 3;
      const float* m = V + (i >> 5) * 16 + g;
      reinterpret_cast<uint4*>(outU + (i >> 5) * kColFloats + 2 * kChunk * kCols)[ln] = make_uint4(pack_bf16(m[2 * t4 * DP], m[(2 * t4 + 1) * DP]), pack_bf16(m[2 * t4 * DP + 8], m[(2 * t4 + 1) * DP + 8]),
                            pack_bf16(m[(2 * t4 + 8) * DP], m[(2 * t4 + 9) * DP]), pack_bf16(m[(2 * t4 + 8) * DP + 8], m[(2 * t4 + 9) * DP + 8]));
    }
  }
  ilb::pdl_launch_dependents();                          // (the blocks of delta_chunks are few and large: they start when these are done)
}

__device__ __forceinline__ void delta_cp_async_16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

constexpr int kChunkThreads = 256;
constexpr int kChunkWarps = kChunkThreads / 32;

static inline size_t chunks_smem_floats(int KP) {
  return 2 * ((size_t)4 * kChunk * KP + KP + 3 * kChunk * kCols) + (size_t)kChunkWarps * 2 * kChunk * kCols + kChunk * kCols;
}

// RH: rows of the state a thread holds (of 16 RH), in pairs, for one column.  Thread (warp, lane): rows (2 warp + lane / 16) RH
// .., column lane % 16 of the block's 16.
template <int RH>
__global__ void __launch_bounds__(kChunkThreads)
delta_chunks_kernel(const DeltaParams p, const float* __restrict__ scratch) {
  ilb::pdl_launch_dependents();
  ilb::pdl_wait();
  constexpr int KP = 16 * RH, PH = RH / 2;
  constexpr int kVecs = 4 * kChunk * KP, kBuf = kVecs + KP + 3 * kChunk * kCols;      // floats of one buffer
  extern __shared__ __align__(16) float sm[];
  float* red = sm + 2 * kBuf;                            // [warps][32][kCols]: sums over a warp's rows, of W S then X S
  float* zs = red + kChunkWarps * 2 * kChunk * kCols;    // [16][kCols]
  const int h = blockIdx.x, c0 = blockIdx.y * kCols, seq = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, cl = lane & 15, r0 = (2 * warp + (lane >> 4)) * RH;
  const int DP = padded_cols(p.dv);
  const int tok0 = p.cu_q[seq], q_len = p.cu_q[seq + 1] - tok0, n_chunks = (q_len + kChunk - 1) / kChunk;
  if (n_chunks == 0) return;
  int first = 0;
  for (int i = 0; i < seq; ++i) first += (p.cu_q[i + 1] - p.cu_q[i] + kChunk - 1) / kChunk;
  const int slot = p.slots[seq];
  float* own = slot >= 0 ? p.state + ((size_t)slot * p.heads + h) * p.d * p.dv : nullptr;
  const int inner_v = p.heads * p.dv, col = c0 + cl;
  const long long per = chunk_floats(KP, DP);

  auto issue = [&](int ci) {
    const float* src = scratch + ((size_t)(first + ci) * p.heads + h) * per;
    float* dst = sm + (ci & 1) * kBuf;
    for (int i = tid; i < (kVecs + KP) / 4; i += kChunkThreads) delta_cp_async_16(dst + 4 * i, src + 4 * i);
    const float* cols = src + kVecs + KP + c0;           // U, Y, V: this block's 16 columns of each
    for (int i = tid; i < 3 * kChunk * kCols / 4; i += kChunkThreads)
      delta_cp_async_16(dst + kVecs + KP + 4 * i, cols + (size_t)(i / (kCols / 4)) * DP + (i % (kCols / 4)) * 4);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  issue(0);
  uint64_t S[PH];                                        // rows r0 + 2 i, r0 + 2 i + 1 of this thread's column
#pragma unroll
  for (int i = 0; i < PH; ++i) {
    const int n = r0 + 2 * i;
    const bool in = own != nullptr && col < p.dv;
    S[i] = pack2((in && n < p.d) ? own[(size_t)n * p.dv + col] : 0.f, (in && n + 1 < p.d) ? own[(size_t)(n + 1) * p.dv + col] : 0.f);
  }
  // this thread's rows of a vector over the state's rows
  auto rows_at = [&](const float* vec, uint64_t (&v)[PH]) {
#pragma unroll
    for (int i = 0; i < PH / 2; ++i) {
      const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(vec + r0 + 4 * i);
      v[2 * i] = a.x; v[2 * i + 1] = a.y;
    }
  };
  for (int ci = 0; ci < n_chunks; ++ci) {
    if (ci + 1 < n_chunks) {
      issue(ci + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const float* buf = sm + (ci & 1) * kBuf;
    const float* Us = buf + kVecs + KP;                  // [16][kCols] each: U, Y, V
    // the 32 rows of W and X times the state: sums over the thread's rows, then over the warp's two row groups
#pragma unroll 8
    for (int v = 0; v < 2 * kChunk; v += 2) {            // two rows at a time: the two row groups end with one each
      uint64_t w[PH], x[PH];
      rows_at(buf + v * KP, w);
      rows_at(buf + (v + 1) * KP, x);
      uint64_t a = mul2(w[0], S[0]), b = mul2(x[0], S[0]);
#pragma unroll
      for (int i = 1; i < PH; ++i) { a = fma2(w[i], S[i], a); b = fma2(x[i], S[i], b); }
      const float fa = sum2(a), fb = sum2(b);
      const bool upper = lane & 16;
      const float sum = (upper ? fb : fa) + __shfl_xor_sync(0xffffffffu, upper ? fa : fb, 16);
      red[(warp * 2 * kChunk + v + (lane >> 4)) * kCols + cl] = sum;
    }
    __syncthreads();
    {
      const int v = tid >> 3, c2 = (tid & 7) * 2;        // row of W (v < 16) or of X
      float2 s = *reinterpret_cast<const float2*>(Us + v * kCols + c2);       // U's rows, then Y's
#pragma unroll
      for (int w = 0; w < kChunkWarps; ++w) {
        const float2 a = *reinterpret_cast<const float2*>(red + (w * 2 * kChunk + v) * kCols + c2);
        s.x += a.x; s.y += a.y;
      }
      if (v < kChunk) {
        *reinterpret_cast<float2*>(zs + v * kCols + c2) = s;
      } else {
        const int t = ci * kChunk + v - kChunk;
        if (t < q_len) {
          float* dst = p.y + (size_t)(tok0 + t) * inner_v + (size_t)h * p.dv + c0 + c2;
          if (c0 + c2 < p.dv) dst[0] = s.x;
          if (c0 + c2 + 1 < p.dv) dst[1] = s.y;
        }
      }
    }
    __syncthreads();
    {
      uint64_t d[PH];
      rows_at(buf + kVecs, d);
#pragma unroll
      for (int i = 0; i < PH; ++i) S[i] = mul2(d[i], S[i]);
      const float* Qs = buf + 2 * kChunk * KP;           // - D q
      const float* Ms = Qs + kChunk * KP;
      const float* Vs = Us + 2 * kChunk * kCols;
#pragma unroll 8
      for (int t = 0; t < kChunk; ++t) {
        uint64_t q[PH], m[PH];
        rows_at(Qs + t * KP, q);
        rows_at(Ms + t * KP, m);
        const float zf = zs[t * kCols + cl], vf = Vs[t * kCols + cl];
        const uint64_t z = pack2(zf, zf), v = pack2(vf, vf);
#pragma unroll
        for (int i = 0; i < PH; ++i) S[i] = fma2(m[i], v, fma2(q[i], z, S[i]));
      }
    }
    __syncthreads();                                     // everyone is done with this buffer and with zs
  }
  if (own != nullptr && col < p.dv) {
#pragma unroll
    for (int i = 0; i < PH; ++i) {
      const int n = r0 + 2 * i;
      float lo, hi;
      unpack2(S[i], lo, hi);
      if (n < p.d) own[(size_t)n * p.dv + col] = lo;
      if (n + 1 < p.d) own[(size_t)(n + 1) * p.dv + col] = hi;
    }
  }
}

// 16 bytes from global memory, requested where it is written: the request is not moved down to the first use.
__device__ __forceinline__ uint4 load_here(const uint4* p) {
  uint4 v;
  asm volatile("ld.global.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}

// `bytes` (a multiple of 16, both addresses on 16-byte boundaries) from global to this block's shared memory, counted on `bar`.
__device__ __forceinline__ void bulk_load(uint32_t dst, const float* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}

// The same walk on the tensor cores (mma.sync m16n8k16, 32-bit accumulation), for projections stored in bfloat16: every 32-bit
// operand is three exact bfloat16 pieces, and of the nine products of two such operands the six that reach 32-bit precision
// are added, smallest first.  A warp owns 16 rows of the state and the block's 16 columns, transposed in the layout of an
// accumulator, which is the layout of the operand that the two thin products read; the sums over the warps meet in shared
// memory.  What a chunk adds to the state is formed apart and joins it with one rounding.
// RING > 0: the chunks' operands come through a ring of that many stages in shared memory, two bulk copies a chunk (the rows'
// part, which all blocks of the head read, and the block's columns' part); 0: straight into registers, a chunk ahead.
// Waits are bounded; on expiry a flag is raised and the walk goes on without waiting.
template <int KP, int RING>
struct ChunksMma {
  static constexpr int kWarps = KP / 16, kLd = 20, kZ = kCols + 1;      // kLd: floats from one row of a warp's sums to the next
  static constexpr int kStage = row_floats_mma(KP) + kColFloats;        // floats
  static constexpr size_t kSmem = sizeof(float) * ((size_t)RING * kStage + (size_t)kWarps * 2 * kChunk * kLd + kChunk * kZ) + 8 * (RING + 2);
};

template <int KP, int RING>
__global__ void __launch_bounds__(KP * 2, 1)
delta_chunks_mma_kernel(const DeltaParams p, const float* __restrict__ scratch, int* error_flag) {
  ilb::pdl_launch_dependents();
  using C = ChunksMma<KP, RING>;
  constexpr int kWarps = C::kWarps, kLd = C::kLd, kZ = C::kZ, kRow = row_floats_mma(KP);
  extern __shared__ __align__(128) float sm[];
  float* red = sm + RING * C::kStage;                    // [warps][32][kLd]
  const uint32_t bar0 = smem_u32(red + kWarps * 2 * kChunk * kLd);      // one mbarrier a stage
  float* zs = red + kWarps * 2 * kChunk * kLd + 2 * (RING + 1);         // [16][kZ]
  if (RING > 0) {
    if (threadIdx.x == 0) {
      for (int i = 0; i < RING; ++i) mbar_init(bar0 + 8 * i, 1);
      asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
  }
  ilb::pdl_wait();
  const int h = blockIdx.x, cb = blockIdx.y, c0 = cb * kCols, seq = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int DP = padded_cols(p.dv);
  const int tok0 = p.cu_q[seq], q_len = p.cu_q[seq + 1] - tok0, n_chunks = (q_len + kChunk - 1) / kChunk;
  if (n_chunks == 0) return;
  int first = 0;
  for (int i = 0; i < seq; ++i) first += (p.cu_q[i + 1] - p.cu_q[i] + kChunk - 1) / kChunk;
  const int slot = p.slots[seq];
  float* own = slot >= 0 ? p.state + ((size_t)slot * p.heads + h) * p.d * p.dv : nullptr;
  const int inner_v = p.heads * p.dv;
  const size_t per = (size_t)p.heads * chunk_floats_mma(KP, DP);        // from one chunk to the next
  const float* src0 = scratch + ((size_t)first * p.heads + h) * chunk_floats_mma(KP, DP);

  // One thread asks for a chunk's operands; a stage is asked for again once every thread is past the barrier that follows its
  // last read.
  bool ok = true;
  auto ask = [&](int ci) {
    const uint32_t dst = smem_u32(sm) + (uint32_t)(ci % (RING > 0 ? RING : 1)) * C::kStage * 4u, bar = bar0 + 8 * (ci % (RING > 0 ? RING : 1));
    const float* at = src0 + (size_t)ci * per;
    mbar_expect_tx(bar, C::kStage * 4u);
    bulk_load(dst, at, kRow * 4u, bar);
    bulk_load(dst + kRow * 4u, at + kRow + cb * kColFloats, kColFloats * 4u, bar);
  };
  if (RING > 0 && tid == 0)
    for (int i = 0; i < RING && i < n_chunks; ++i) ask(i);

  uint4 A[6], B[6], V;                                   // W hi mid lo, X hi mid lo;  D m hi mid lo, - D q hi mid lo
  float2 D[2];
  constexpr int kAdd = (2 * kChunk * 8 + KP * 2 - 1) / (KP * 2);
  float2 add[kAdd];                                      // this thread's elements of U and Y: pairs of columns, dealt out by number
  auto take = [](const uint4* at) { return RING > 0 ? *at : load_here(at); };
  auto load_a = [&](const float* rows) {
    const uint4* f = reinterpret_cast<const uint4*>(rows) + (size_t)warp * 6 * 32 + lane;
#pragma unroll
    for (int i = 0; i < 6; ++i) A[i] = take(f + 32 * i);
  };
  auto load_b = [&](const float* rows, const float* cols) {
    const uint4* f = reinterpret_cast<const uint4*>(rows) + (size_t)(kWarps * 6 + warp * 6) * 32 + lane;
#pragma unroll
    for (int i = 0; i < 6; ++i) B[i] = take(f + 32 * i);
    const float* d = rows + kWarps * 12 * kFragFloats;
    D[0] = *reinterpret_cast<const float2*>(d + warp * 16 + 2 * t4);
    D[1] = *reinterpret_cast<const float2*>(d + warp * 16 + 8 + 2 * t4);
    V = take(reinterpret_cast<const uint4*>(cols + 2 * kChunk * kCols) + lane);
  };
  auto load_uy = [&](const float* cols) {
#pragma unroll
    for (int i = 0; i < kAdd; ++i) {
      const int e = tid + i * KP * 2;
      if (e < 2 * kChunk * 8) add[i] = *reinterpret_cast<const float2*>(cols + 2 * e);
    }
  };
  if (RING == 0) {
    load_a(src0);
    load_b(src0, src0 + kRow + cb * kColFloats);
    load_uy(src0 + kRow + cb * kColFloats);
  }
  // S[j][0, 1]: rows 16 warp + 8 j + 2 t4 (+ 1), column g; [2, 3]: column g + 8
  float S[2][4];
#pragma unroll
  for (int j = 0; j < 2; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int n = warp * 16 + 8 * j + 2 * t4 + (e & 1), col = c0 + g + 8 * (e >> 1);
      S[j][e] = (own != nullptr && n < p.d && col < p.dv) ? own[(size_t)n * p.dv + col] : 0.f;
    }
  auto mma = [&](float (&c)[4], const uint4& a, uint32_t b0, uint32_t b1) {
    const uint32_t aa[4] = {a.x, a.y, a.z, a.w};
    mma_16816(c, aa, b0, b1);
  };
  for (int ci = 0; ci < n_chunks; ++ci) {
    const float* stage = sm + (ci % (RING > 0 ? RING : 1)) * C::kStage;      // (RING > 0)
    const float* next = src0 + (size_t)(ci + 1) * per;                     // (RING == 0)
    const bool more = ci + 1 < n_chunks;
    if (RING > 0) {
      if (ok && !mbar_wait(bar0 + 8 * (ci % (RING > 0 ? RING : 1)), (ci / (RING > 0 ? RING : 1)) & 1)) {
        ok = false;
        if (error_flag != nullptr) *error_flag = 1;
      }
      load_a(stage);
    }
    {
      uint32_t b[3][2][2];                               // pieces of the state: [piece][columns 8 jj + g][rows 2 t4, 2 t4 + 8]
#pragma unroll
      for (int jj = 0; jj < 2; ++jj)
#pragma unroll
        for (int j = 0; j < 2; ++j) split3(S[j][2 * jj], S[j][2 * jj + 1], b[0][jj][j], b[1][jj][j], b[2][jj][j]);
#pragma unroll
      for (int m = 0; m < 2; ++m)
#pragma unroll
        for (int jj = 0; jj < 2; ++jj) {
          float c[4] = {0.f, 0.f, 0.f, 0.f}, f[4] = {0.f, 0.f, 0.f, 0.f};
          mma(c, A[3 * m + 2], b[0][jj][0], b[0][jj][1]);
          mma(f, A[3 * m], b[1][jj][0], b[1][jj][1]);
          mma(c, A[3 * m], b[2][jj][0], b[2][jj][1]);
          mma(f, A[3 * m], b[0][jj][0], b[0][jj][1]);
          mma(c, A[3 * m + 1], b[1][jj][0], b[1][jj][1]);
          mma(c, A[3 * m + 1], b[0][jj][0], b[0][jj][1]);
#pragma unroll
          for (int e = 0; e < 4; ++e) c[e] += f[e];
          float* r = red + (size_t)(warp * 2 * kChunk + m * kChunk + g) * kLd + 8 * jj + 2 * t4;
          *reinterpret_cast<float2*>(r) = make_float2(c[0], c[1]);
          *reinterpret_cast<float2*>(r + 8 * kLd) = make_float2(c[2], c[3]);
        }
    }
    if (RING > 0) load_uy(stage + kRow);
    else if (more) load_a(next);
    __syncthreads();
    if (RING > 0 && tid == 0 && ci > 0 && ci - 1 + RING < n_chunks) ask(ci - 1 + RING);      // (everyone is done with the chunk before)
#pragma unroll
    for (int i = 0; i < kAdd; ++i) {
      const int e = tid + i * KP * 2;
      if (e < 2 * kChunk * 8) {
        const int v = e >> 3, c2 = (e & 7) * 2;          // row of W (v < 16) or of X
        float2 s = add[i];
#pragma unroll
        for (int w = 0; w < kWarps; ++w) {
          const float2 a = *reinterpret_cast<const float2*>(red + (size_t)(w * 2 * kChunk + v) * kLd + c2);
          s.x += a.x; s.y += a.y;
        }
        if (v < kChunk) {
          zs[v * kZ + c2] = s.x; zs[v * kZ + c2 + 1] = s.y;
        } else {
          const int t = ci * kChunk + v - kChunk;
          if (t < q_len) {
            float* dst = p.y + (size_t)(tok0 + t) * inner_v + (size_t)h * p.dv + c0 + c2;
            if (c0 + c2 < p.dv) dst[0] = s.x;
            if (c0 + c2 + 1 < p.dv) dst[1] = s.y;
          }
        }
      }
    }
    if (RING > 0) load_b(stage, stage + kRow);
    else if (more) load_uy(next + kRow + cb * kColFloats);
    __syncthreads();
    {
      uint4 z[3];                                        // pieces of Z transposed: columns g, g + 8, tokens 2 t4 (+ 1), + 8
      const float* zr = zs + 2 * t4 * kZ + g;
      split3(zr[0], zr[kZ], z[0].x, z[1].x, z[2].x);
      split3(zr[8], zr[kZ + 8], z[0].y, z[1].y, z[2].y);
      split3(zr[8 * kZ], zr[9 * kZ], z[0].z, z[1].z, z[2].z);
      split3(zr[8 * kZ + 8], zr[9 * kZ + 8], z[0].w, z[1].w, z[2].w);
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        auto b0 = [&](int i) { return j == 0 ? B[i].x : B[i].z; };
        auto b1 = [&](int i) { return j == 0 ? B[i].y : B[i].w; };
        float c[4] = {0.f, 0.f, 0.f, 0.f}, e[4] = {0.f, 0.f, 0.f, 0.f}, f[4] = {0.f, 0.f, 0.f, 0.f};
        mma(c, V, b0(2), b1(2));
        mma(e, z[2], b0(3), b1(3));
        mma(f, z[1], b0(3), b1(3));
        mma(c, V, b0(1), b1(1));
        mma(e, z[0], b0(5), b1(5));
        mma(f, z[0], b0(4), b1(4));
        mma(c, V, b0(0), b1(0));
        mma(e, z[1], b0(4), b1(4));
        mma(f, z[0], b0(3), b1(3));
#pragma unroll
        for (int i = 0; i < 4; ++i) c[i] += e[i] + f[i];
        S[j][0] = fmaf(D[j].x, S[j][0], c[0]); S[j][1] = fmaf(D[j].y, S[j][1], c[1]);
        S[j][2] = fmaf(D[j].x, S[j][2], c[2]); S[j][3] = fmaf(D[j].y, S[j][3], c[3]);
      }
    }
    if (RING == 0 && more) load_b(next, next + kRow + cb * kColFloats);
  }
  if (RING > 0 && !ok)                                   // copies that may still be on their way land before the block ends
    for (int i = 0; i < (RING > 0 ? RING : 1); ++i) mbar_wait(bar0 + 8 * i, 0);
  if (own != nullptr) {
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = warp * 16 + 8 * j + 2 * t4 + (e & 1), col = c0 + g + 8 * (e >> 1);
        if (n < p.d && col < p.dv) own[(size_t)n * p.dv + col] = S[j][e];
      }
  }
}

template <int KP, int RING>
static int chunks_mma_launch(const DeltaParams& p, const float* scratch, int* error_flag, cudaStream_t stream) {
  constexpr size_t smem = ChunksMma<KP, RING>::kSmem;
  static_assert(smem <= 227 * 1024, "the ring does not fit shared memory");
  static OncePerDevice once;
  if (smem > 48 * 1024 && once.first() &&
      cudaFuncSetAttribute(delta_chunks_mma_kernel<KP, RING>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
    once.forget();
    return fail("delta_chunks: cannot reserve %zu bytes of shared memory", smem);
  }
  ilb::launch(delta_chunks_mma_kernel<KP, RING>, dim3(p.heads, padded_cols(p.dv) / kCols, p.n_seqs), dim3(KP * 2), smem, stream, p, scratch, error_flag);
  return check_launch("delta_chunks");
}

// Floats of scratch that `n_blocks` chunks need.
ILB_EXPORT long long ilb_delta_chunk_floats(int n_blocks, int heads, int d, int dv, int dtype) {
  const int KP = padded_rows(d), DP = padded_cols(dv);
  return (long long)n_blocks * heads * (dtype == kF32 ? chunk_floats(KP, DP) : chunk_floats_mma(KP, DP));
}

template <int RH>
static int chunks_launch(const DeltaParams& p, const float* scratch, cudaStream_t stream) {
  const size_t smem = sizeof(float) * chunks_smem_floats(16 * RH);
  static OncePerDevice once;
  if (once.first() && cudaFuncSetAttribute(delta_chunks_kernel<RH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
    once.forget();
    return fail("delta_chunks: cannot reserve %zu bytes of shared memory", smem);
  }
  ilb::launch(delta_chunks_kernel<RH>, dim3(p.heads, padded_cols(p.dv) / kCols, p.n_seqs), dim3(kChunkThreads), smem, stream, p, scratch);
  return check_launch("delta_chunks");
}

template <typename TI>
static int prep_launch(const DeltaParams& p, float* scratch, int n_blocks, cudaStream_t stream) {
  const int KP = padded_rows(p.d);
  const size_t smem = sizeof(float) * prep_smem_floats(KP, padded_cols(p.dv));
  ILB_REQUIRE(smem <= 200 * 1024, "delta_prep: states of %d x %d do not fit the block's shared memory", p.d, p.dv);
  static OncePerDevice once;
  if (once.first() && cudaFuncSetAttribute(delta_prep_kernel<TI>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess) {
    once.forget();
    return fail("delta_prep: cannot reserve shared memory");
  }
  ilb::launch(delta_prep_kernel<TI>, dim3(n_blocks, p.heads), dim3(kPrepThreads), smem, stream, p, scratch, KP);
  return check_launch("delta_prep");
}

// As ilb_delta_scan, 16 tokens at a time; n_blocks = the sum over the sequences of ceil(tokens / 16), scratch of
// ilb_delta_chunk_floats(n_blocks, ...) floats on a 16-byte boundary.
ILB_EXPORT int ilb_delta_chunks(const void* proj, int dtype, int ld, int col_r, int col_k, int col_v, int col_a, const float* low,
                                const float* w0, const float* ab, float log_decay, float unit_eps, float* state, float* y,
                                const int* cu_q, const int* slots, int n_seqs, int heads, int d, int dv, float* scratch,
                                long long scratch_floats, int n_blocks, int* error_flag, cudaStream_t stream) {
  const DeltaParams p{proj, ld, col_r, col_k, col_v, col_a, low, w0, ab, state, y, cu_q, slots, n_seqs, heads, d, dv, log_decay, unit_eps};
  if (int rc = check_sizes(p, dtype)) return rc;
  ILB_REQUIRE(log_decay >= 0.f && log_decay * kChunk <= 40.f, "delta_chunks: a decay of exp(-%f) a token leaves a chunk's range", (double)log_decay);
  ILB_REQUIRE(scratch != nullptr && (uintptr_t)scratch % 16 == 0 && ilb_delta_chunk_floats(n_blocks, heads, d, dv, dtype) <= scratch_floats,
              "delta_chunks: scratch too small");
  ILB_REQUIRE(heads <= 65535, "delta_chunks: too many heads");
  if (n_seqs == 0 || n_blocks <= 0) return 0;
  if (int rc = dtype == kF32 ? prep_launch<float>(p, scratch, n_blocks, stream) : prep_launch<__nv_bfloat16>(p, scratch, n_blocks, stream)) return rc;
  const int rows = padded_rows(d);
  if (dtype == kBF16)
    return rows == 64 ? chunks_mma_launch<64, 4>(p, scratch, error_flag, stream)
                      : rows == 128 ? chunks_mma_launch<128, 4>(p, scratch, error_flag, stream) : chunks_mma_launch<256, 0>(p, scratch, error_flag, stream);
  return rows == 64 ? chunks_launch<4>(p, scratch, stream) : rows == 128 ? chunks_launch<8>(p, scratch, stream) : chunks_launch<16>(p, scratch, stream);
}

// ---------------------------------------------------------------- single tokens
struct StepParams {
  DeltaParams a;
  int col_low, rank, ld_w2;          // the low-rank map's inner row in proj, its size, the row stride of w2 [heads * d][ld_w2]
  const void* w2;
  int col_g;                         // the output gate's columns in proj (heads * dv)
  const float* norm_w; float eps;    // [heads * dv]
  void* out; int ld_out;             // [sequences' tokens, heads * dv] of the compute dtype
};

constexpr int kStepThreads = 256;
constexpr int kStepWarps = kStepThreads / 32;
constexpr int kMaxRank = 512;

// A block per (head, sequence): warp w holds rows w, w + 8, ... of the state, lane l columns 4 l .. 4 l + 3 (dv <= 128, a
// multiple of four; d <= 128).
template <typename TI>
__global__ void __launch_bounds__(kStepThreads)
delta_step_kernel(const StepParams q) {
  ilb::pdl_launch_dependents();
  ilb::pdl_wait();
  constexpr bool FAST = sizeof(TI) == 2;
  constexpr int kRows = 128 / kStepWarps;
  const DeltaParams& p = q.a;
  __shared__ float low[kMaxRank];
  __shared__ float Us[128], Ws[128], Gs[128], Ks[128], Rs[128];
  __shared__ float4 red[kStepWarps][32];
  __shared__ float scratch[33];
  const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int t = p.cu_q[seq];
  if (p.cu_q[seq + 1] - t != 1) return;                  // single tokens only
  const int slot = p.slots[seq];
  float* own = slot >= 0 ? p.state + ((size_t)slot * p.heads + h) * p.d * p.dv : nullptr;
  const bool cols = 4 * lane < p.dv;
  float4 S[kRows];
#pragma unroll
  for (int i = 0; i < kRows; ++i) {                      // the whole state's loads go out first
    const int n = warp + kStepWarps * i;
    S[i] = (own != nullptr && cols && n < p.d) ? *reinterpret_cast<const float4*>(own + (size_t)n * p.dv + 4 * lane) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const TI* row = reinterpret_cast<const TI*>(p.proj) + (size_t)t * p.ld;
  for (int i = tid; i < q.rank; i += kStepThreads) low[i] = tanhf(to_float(row[q.col_low + i]));
  float kk = 0.f;
  if (tid < 128) {
    kk = tid < p.d ? to_float(row[p.col_k + h * p.d + tid]) : 0.f;
    Ks[tid] = kk;
    Rs[tid] = tid < p.d ? to_float(row[p.col_r + h * p.d + tid]) : 0.f;
  }
  const float inv = 1.0f / sqrtf(block_sum(kk * kk, scratch) + p.unit_eps);      // (its barriers also publish low, Ks, Rs)
  {   // two threads a channel: the map's row, then decay and removal rate
    const int n = tid >> 1, half = tid & 1;
    const int ch = h * p.d + (n < p.d ? n : 0);
    const TI* w2 = reinterpret_cast<const TI*>(q.w2) + (size_t)ch * q.ld_w2;
    float s = 0.f;
    if constexpr (FAST) {                                // (rows are padded to multiples of eight and start on 16-byte boundaries)
      for (int i = half * 8; i < q.rank; i += 16) {
        const uint4 v = *reinterpret_cast<const uint4*>(w2 + i);
        const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          if (i + 2 * j < q.rank) s = fmaf(__uint_as_float(w[j] << 16), low[i + 2 * j], s);
          if (i + 2 * j + 1 < q.rank) s = fmaf(__uint_as_float(w[j] & 0xFFFF0000u), low[i + 2 * j + 1], s);
        }
      }
    } else {
      for (int i = half; i < q.rank; i += 2) s = fmaf(to_float(w2[i]), low[i], s);
    }
    s += __shfl_xor_sync(0xffffffffu, s, 1);
    if (half == 0) {
      const bool on = n < p.d;
      const float u = Ks[n] * inv;
      Us[n] = u;
      Ws[n] = on ? exp_t<FAST>(-p.log_decay * sigmoid_t<FAST>(s + p.w0[ch])) : 0.f;
      Gs[n] = on ? -sigmoid_t<FAST>(to_float(row[p.col_a + ch]) + p.ab[ch]) * u : 0.f;
    }
  }
  const float4 v = [&]() {
    float e[4];
#pragma unroll
    for (int c = 0; c < 4; ++c) e[c] = cols ? to_float(row[p.col_v + h * p.dv + 4 * lane + c]) : 0.f;
    return make_float4(e[0], e[1], e[2], e[3]);
  }();
  __syncthreads();
  auto total = [&](float4 part) {                        // sum over the warps, the same in every warp
    red[warp][lane] = part;
    __syncthreads();
    float4 s = red[0][lane];
#pragma unroll
    for (int w = 1; w < kStepWarps; ++w) { const float4 a = red[w][lane]; s.x += a.x; s.y += a.y; s.z += a.z; s.w += a.w; }
    __syncthreads();
    return s;
  };
  float4 part = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < kRows; ++i) {
    const float u = Us[warp + kStepWarps * i];
    part.x = fmaf(u, S[i].x, part.x); part.y = fmaf(u, S[i].y, part.y); part.z = fmaf(u, S[i].z, part.z); part.w = fmaf(u, S[i].w, part.w);
  }
  const float4 z = total(part);
  part = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < kRows; ++i) {
    const int n = warp + kStepWarps * i;
    const float w = Ws[n], g = Gs[n], k = Ks[n], r = Rs[n];
    S[i].x = fmaf(w, S[i].x, fmaf(g, z.x, k * v.x)); S[i].y = fmaf(w, S[i].y, fmaf(g, z.y, k * v.y));
    S[i].z = fmaf(w, S[i].z, fmaf(g, z.z, k * v.z)); S[i].w = fmaf(w, S[i].w, fmaf(g, z.w, k * v.w));
    part.x = fmaf(r, S[i].x, part.x); part.y = fmaf(r, S[i].y, part.y); part.z = fmaf(r, S[i].z, part.z); part.w = fmaf(r, S[i].w, part.w);
    if (own != nullptr && cols && n < p.d) *reinterpret_cast<float4*>(own + (size_t)n * p.dv + 4 * lane) = S[i];
  }
  const float4 o = total(part);
  if (warp == 0) {
    const float ss = warp_sum(o.x * o.x + o.y * o.y + o.z * o.z + o.w * o.w);
    const float f = 1.0f / sqrtf(ss / (float)p.dv + q.eps);
    if (cols) {
      const float e[4] = {o.x, o.y, o.z, o.w};
      TI* dst = reinterpret_cast<TI*>(q.out) + (size_t)t * q.ld_out + h * p.dv + 4 * lane;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int at = h * p.dv + 4 * lane + c;
        dst[c] = from_float<TI>(e[c] * f * q.norm_w[at] * sigmoid_t<false>(to_float(row[q.col_g + at])));
      }
    }
  }
}

ILB_EXPORT int ilb_delta_step_supported(int d, int dv, int rank) { return (d <= 128 && dv <= 128 && dv % 4 == 0 && rank <= kMaxRank) ? 1 : 0; }

// Single tokens from the layer's projections to what its output product reads: proj [T, ld] holds r, k, a, v, the gate and the
// map's inner row; w2 [heads * d, ld_w2] of the same dtype; out [T, ld_out].
ILB_EXPORT int ilb_delta_step(const void* proj, int dtype, int ld, int col_r, int col_k, int col_v, int col_a, int col_g, int col_low,
                              int rank, const void* w2, int ld_w2, const float* w0, const float* ab, float log_decay, float unit_eps,
                              const float* norm_w, float eps, float* state, void* out, int ld_out, const int* cu_q, const int* slots,
                              int n_seqs, int heads, int d, int dv, cudaStream_t stream) {
  const DeltaParams p{proj, ld, col_r, col_k, col_v, col_a, w0, w0, ab, state, state, cu_q, slots, n_seqs, heads, d, dv, log_decay, unit_eps};
  if (int rc = check_sizes(p, dtype)) return rc;
  ILB_REQUIRE(ilb_delta_step_supported(d, dv, rank) && rank > 0, "delta_step: states of %d x %d with a map of %d are not built", d, dv, rank);
  ILB_REQUIRE(w2 != nullptr && norm_w != nullptr && out != nullptr && eps > 0.f && col_g >= 0 && col_low >= 0 && ld >= col_g + heads * dv &&
              ld >= col_low + rank && ld_w2 >= (rank + 7) / 8 * 8 && ld_w2 % 8 == 0 && ((uintptr_t)w2 % 16 == 0) && ((uintptr_t)state % 16 == 0) &&
              ld_out >= heads * dv, "delta_step: bad inputs");
  if (n_seqs == 0) return 0;
  const StepParams q{p, col_low, rank, ld_w2, w2, col_g, norm_w, eps, out, ld_out};
  if (dtype == kF32) ilb::launch(delta_step_kernel<float>, dim3(heads, n_seqs), dim3(kStepThreads), 0, stream, q);
  else ilb::launch(delta_step_kernel<__nv_bfloat16>, dim3(heads, n_seqs), dim3(kStepThreads), 0, stream, q);
  return check_launch("delta_step");
}

ILB_DEFINE_LAST_ERROR()
