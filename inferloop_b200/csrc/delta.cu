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
//                memory.
//
// Everything is 32-bit; the projections come in the compute dtype.  A sequence whose slot is negative (a dummy row that
// pads a recorded launch) starts from zero and stores nothing.
#include <math.h>
#include "common.cuh"

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

ILB_DEFINE_LAST_ERROR()
