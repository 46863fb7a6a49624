// Fused per-head q/k RMSNorm + rotary position encoding + paged KV-cache write.
//
// Input is the fused projection output qkv[T, (nq + nkv) * d + nkv * dv].  For every token and
// head this kernel, in 32-bit:
//   q, k heads: optional RMSNorm over the head (weight [d] shared by all heads, or none), and
//               the rotation of the first `rotary_dim` elements (pairs i / i + rd/2, or
//               neighbours 2i / 2i + 1), in either order;
//   v heads:    optionally kept for, or mixed with, the values of the first mixing layer;
//   q -> q_out[T, nq*d];  k, v -> the cache page of the token's position.
// The reference runs these as three launches (norm_rows, prefill_rope, attention::append;
// crates/backend/cuda-kernels/src/tile/state/aux_kernels.rs:104-200 and
// tile/attention/resident_attention_prefill_kernels.rs:170-245).  Formulas: per-head norm
// before the rotation (crates/model/recipes/src/decoder.rs:278-335), rotation
// x[i] = a cos - b sin, x[i + rd/2] = a sin + b cos
// (crates/testing/cpu/reference-ops/src/kernels.rs:217-241).
//
// Cache layout per layer: K [num_pages, nkv, page_size, d], V [num_pages, nkv, page_size, dv]; the page of
// position p of sequence s is block_table[s, p / page_size].
#include "common.cuh"

using namespace ilb;

constexpr int kWarpsPerBlock = 4;

// What a launch may ask for beside the stock order (norm with a weight, then the half-split
// rotation): flag bits of `mode`.
constexpr int kPairsInterleaved = 1;   // rotation pairs are (2i, 2i + 1) instead of (i, i + rd/2)
constexpr int kNormAfterRotation = 2;  // the per-head norm follows the rotation instead of preceding it
constexpr int kNormUnweighted = 4;     // q and k heads are divided by their root mean square, no weight
// Value mixing across layers (`v_mode`): 1 = this layer's values are also kept in `v_first`
// [T, nkv * dv]; 2 = v <- (1 - lambda) v + lambda v_first (lambda a device scalar) before the
// cache write.

template <typename TQ, typename TC>
__global__ void __launch_bounds__(kWarpsPerBlock * 32)
qk_norm_rope_kernel(const TQ* __restrict__ qkv, TQ* __restrict__ q_out,
                    const float* __restrict__ q_weight, const float* __restrict__ k_weight,
                    float eps, const float2* __restrict__ rope_table, int rotary_dim,
                    const int* __restrict__ positions, const int* __restrict__ seq_of_token,
                    const int* __restrict__ block_table, int max_blocks, int page_size,
                    int num_pages, TC* __restrict__ k_cache, TC* __restrict__ v_cache,
                    int n_tokens, int nq, int nkv, int d, int dv, int qkv_stride, int q_out_stride,
                    int mode, int v_mode, const float* __restrict__ v_lambda, TQ* __restrict__ v_first) {
  ilb::pdl_launch_dependents();
  ilb::pdl_wait();
  extern __shared__ float smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x;
  const int head = blockIdx.y * kWarpsPerBlock + warp;
  const int total_heads = nq + 2 * nkv;
  if (head >= total_heads) return;
  const int dmax = d > dv ? d : dv;
  float* vec = smem + warp * dmax;
  const bool is_q = head < nq, is_k = !is_q && head < nq + nkv;
  const int width = (is_q || is_k) ? d : dv;
  const size_t offset = (is_q || is_k) ? (size_t)head * d : (size_t)(nq + nkv) * d + (size_t)(head - nq - nkv) * dv;
  const TQ* src = qkv + (size_t)t * qkv_stride + offset;

  for (int i = lane; i < width; i += 32) vec[i] = to_float(src[i]);
  __syncwarp();
  const float* weight = is_q ? q_weight : (is_k ? k_weight : nullptr);
  const bool normed = (is_q || is_k) && (weight != nullptr || (mode & kNormUnweighted));
  auto norm = [&]() {
    float ss = 0.f;
    for (int i = lane; i < width; i += 32) ss = fmaf(vec[i], vec[i], ss);
    ss = warp_sum(ss);
    const float inv = 1.0f / sqrtf(ss / (float)width + eps);
    for (int i = lane; i < width; i += 32) vec[i] = weight != nullptr ? vec[i] * inv * weight[i] : vec[i] * inv;
    __syncwarp();
  };
  if (normed && !(mode & kNormAfterRotation)) norm();
  if ((is_q || is_k) && rope_table != nullptr) {
    const int half = rotary_dim / 2;
    const float2* cs = rope_table + (size_t)t * half;
    const bool inter = mode & kPairsInterleaved;
    for (int i = lane; i < half; i += 32) {
      const int ia = inter ? 2 * i : i, ib = inter ? 2 * i + 1 : i + half;
      const float a = vec[ia], b = vec[ib];
      const float2 c = cs[i];
      // Products and sums rounded separately, as the reference's scalar code does.
      vec[ia] = __fsub_rn(__fmul_rn(a, c.x), __fmul_rn(b, c.y));
      vec[ib] = __fadd_rn(__fmul_rn(a, c.y), __fmul_rn(b, c.x));
    }
    __syncwarp();
  }
  if (normed && (mode & kNormAfterRotation)) norm();
  if (is_q) {
    TQ* dst = q_out + (size_t)t * q_out_stride + (size_t)head * d;
    for (int i = lane; i < d; i += 32) dst[i] = from_float<TQ>(vec[i]);
    return;
  }
  const int kvh = is_k ? head - nq : head - nq - nkv;
  if (!is_k && v_mode != 0) {
    TQ* keep = v_first + ((size_t)t * nkv + kvh) * dv;
    if (v_mode == 1) {
      for (int i = lane; i < dv; i += 32) keep[i] = from_float<TQ>(vec[i]);
    } else {
      const float lam = *v_lambda;
      for (int i = lane; i < dv; i += 32) vec[i] = fmaf(lam, to_float(keep[i]), (1.0f - lam) * vec[i]);
    }
  }
  if (k_cache == nullptr) return;
  const int pos = positions[t];
  const int seq = seq_of_token[t];
  const int blk = pos / page_size;
  if (blk < 0 || blk >= max_blocks) return;
  const int page = block_table[(size_t)seq * max_blocks + blk];
  if (page < 0 || page >= num_pages) return;   // never write outside the pool
  TC* dst = (is_k ? k_cache : v_cache) +
            (((size_t)page * nkv + kvh) * page_size + (pos % page_size)) * width;
  for (int i = lane; i < width; i += 32) dst[i] = from_float<TC>(vec[i]);
}

// The common geometry, bfloat16 throughout, head size 128, rotation over the whole head: one
// CTA per token; eight lanes take a head, a lane holding elements 8l .. 8l+7 of each half of
// the head (the two members of its eight rotation pairs) in registers: 16-byte accesses, no
// shared memory, a warp works on four heads at a time and has the loads of all its heads in
// flight together (up to kFastUnroll passes).
constexpr int kFastWarps = 4;
constexpr int kFastUnroll = 3;

__device__ __forceinline__ void unpack8(const uint4& r, float* x) {
  const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) { x[2 * i] = __uint_as_float(w[i] << 16); x[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u); }
}
__device__ __forceinline__ uint4 pack8(const float* x) {
  uint32_t w[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    __nv_bfloat162 h = __floats2bfloat162_rn(x[2 * i], x[2 * i + 1]);
    w[i] = *reinterpret_cast<uint32_t*>(&h);
  }
  return make_uint4(w[0], w[1], w[2], w[3]);
}

// kVariant: the modes of the general kernel (pairs of neighbours over the first rotary_dim
// elements, which a lane's eight consecutive elements hold four of; the norm after the rotation;
// no weight) and the kept / mixed values.
template <bool kVariant>
__global__ void __launch_bounds__(kFastWarps * 32)
qk_norm_rope_d128_kernel(const __nv_bfloat16* __restrict__ qkv, __nv_bfloat16* __restrict__ q_out,
                         const float* __restrict__ q_weight, const float* __restrict__ k_weight, float eps,
                         const float2* __restrict__ rope_table, const int* __restrict__ positions,
                         const int* __restrict__ seq_of_token, const int* __restrict__ block_table, int max_blocks,
                         int page_size, int num_pages, __nv_bfloat16* __restrict__ k_cache,
                         __nv_bfloat16* __restrict__ v_cache, int nq, int nkv, int qkv_stride, int q_out_stride,
                         int mode, int rotary_dim, int v_mode, const float* __restrict__ v_lambda,
                         __nv_bfloat16* __restrict__ v_first) {
  ilb::pdl_launch_dependents();
  ilb::pdl_wait();
  constexpr int d = 128;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int slot = lane >> 3, l8 = lane & 7;           // which of the warp's four heads; which eighth of each half
  const int t = blockIdx.x;
  const int total_heads = nq + 2 * nkv;
  const __nv_bfloat16* row = qkv + (size_t)t * qkv_stride;
  // the loads of all this lane's heads first
  const int stride = kFastWarps * 4 * gridDim.y;       // heads between two passes (the CTAs of a token deal its heads out four by four)
  const int h0 = (blockIdx.y * kFastWarps + warp) * 4 + slot;
  uint4 raw[kFastUnroll][2];
#pragma unroll
  for (int u = 0; u < kFastUnroll; ++u) {
    const int head = h0 + u * stride;
    if (head < total_heads) {
      const uint4* src = reinterpret_cast<const uint4*>(row + (size_t)head * d);
      raw[u][0] = __ldg(src + l8);
      raw[u][1] = __ldg(src + 8 + l8);
    } else {
      raw[u][0] = make_uint4(0u, 0u, 0u, 0u);
      raw[u][1] = raw[u][0];
    }
  }
  // where this token's key and value go: looked up by the lanes that hold a k or v head only
  size_t cache_off = 0;
  int cache_state = 0;                                // 0 not looked up, 1 held, -1 no page
  auto cache_row = [&]() {
    if (cache_state == 0) {
      cache_state = -1;
      if (k_cache != nullptr) {
        const int pos = positions[t], seq = seq_of_token[t];
        const int blk = pos / page_size;
        if (blk >= 0 && blk < max_blocks) {
          const int page = block_table[(size_t)seq * max_blocks + blk];
          if (page >= 0 && page < num_pages) {        // never write outside the pool
            cache_off = ((size_t)page * nkv * page_size + (pos % page_size)) * d;
            cache_state = 1;
          }
        }
      }
    }
    return cache_state == 1;
  };
  // cos and sin of this lane's eight pairs (j, j + 64), j = 8 l8 .. 8 l8 + 7; with pairs of
  // neighbours: of the pairs 4 l8 .. 4 l8 + 3 (lower half) and 32 + 4 l8 .. (upper half)
  float2 cs[8];
  if (kVariant && (mode & kPairsInterleaved)) {
    if (rope_table != nullptr) {
#pragma unroll
      for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int pair = 32 * h + 4 * l8 + i;
          cs[4 * h + i] = 2 * pair + 1 < rotary_dim ? __ldg(rope_table + (size_t)t * (rotary_dim / 2) + pair) : make_float2(1.f, 0.f);
        }
    }
  } else if (rope_table != nullptr) {
    const float4* c = reinterpret_cast<const float4*>(rope_table + (size_t)t * (d / 2) + 8 * l8);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float4 v = __ldg(c + i);
      cs[2 * i] = make_float2(v.x, v.y);
      cs[2 * i + 1] = make_float2(v.z, v.w);
    }
  }
  auto weight8 = [&](const float* w, int half, float* out8) {      // weights of elements 64 half + 8 l8 .. + 7
    const float4 a = __ldg(reinterpret_cast<const float4*>(w + 64 * half + 8 * l8));
    const float4 b = __ldg(reinterpret_cast<const float4*>(w + 64 * half + 8 * l8) + 1);
    out8[0] = a.x; out8[1] = a.y; out8[2] = a.z; out8[3] = a.w; out8[4] = b.x; out8[5] = b.y; out8[6] = b.z; out8[7] = b.w;
  };
#pragma unroll
  for (int u = 0; u < kFastUnroll; ++u) {
    const int head = h0 + u * stride;
    const bool valid = head < total_heads;
    const bool is_q = head < nq, is_k = !is_q && head < nq + nkv;
    float x[16];                                       // [0..7]: lower half, [8..15]: upper half
    unpack8(raw[u][0], x);
    unpack8(raw[u][1], x + 8);
    const float* w = is_q ? q_weight : (is_k ? k_weight : nullptr);
    if constexpr (kVariant) {
      const bool turn = (is_q || is_k) && rope_table != nullptr;
      const bool normed = (is_q || is_k) && (w != nullptr || (mode & kNormUnweighted));
      auto rotate = [&]() {
        if (mode & kPairsInterleaved) {
#pragma unroll
          for (int i = 0; i < 8; ++i) {                      // (x[2 i], x[2 i + 1]) is pair i of this lane
            const float a = x[2 * i], b = x[2 * i + 1];
            x[2 * i] = __fsub_rn(__fmul_rn(a, cs[i].x), __fmul_rn(b, cs[i].y));
            x[2 * i + 1] = __fadd_rn(__fmul_rn(a, cs[i].y), __fmul_rn(b, cs[i].x));
          }
        } else {
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            const float a = x[i], b = x[8 + i];
            x[i] = __fsub_rn(__fmul_rn(a, cs[i].x), __fmul_rn(b, cs[i].y));
            x[8 + i] = __fadd_rn(__fmul_rn(a, cs[i].y), __fmul_rn(b, cs[i].x));
          }
        }
      };
      const bool after = mode & kNormAfterRotation;
      if (turn && after) rotate();
      // (every lane takes part in the exchange; a head past the end holds zeros)
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < 16; ++i) ss = fmaf(x[i], x[i], ss);
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
      ss += __shfl_xor_sync(0xffffffffu, ss, 4);
      if (!valid) continue;
      if (normed) {
        const float inv = 1.0f / sqrtf(ss / (float)d + eps);
        if (w != nullptr) {
          float wl[8], wh[8];
          weight8(w, 0, wl);
          weight8(w, 1, wh);
#pragma unroll
          for (int i = 0; i < 8; ++i) { x[i] = x[i] * inv * wl[i]; x[8 + i] = x[8 + i] * inv * wh[i]; }
        } else {
#pragma unroll
          for (int i = 0; i < 16; ++i) x[i] = x[i] * inv;
        }
      }
      if (turn && !after) rotate();
      __nv_bfloat16* dst;
      if (is_q) dst = q_out + (size_t)t * q_out_stride + (size_t)head * d;
      else {
        if (!is_k && v_mode != 0) {                          // this token's values of the first mixing layer
          uint4* keep = reinterpret_cast<uint4*>(v_first + ((size_t)t * nkv + (head - nq - nkv)) * d);
          if (v_mode == 1) {
            keep[l8] = pack8(x);
            keep[8 + l8] = pack8(x + 8);
          } else {
            const float lam = __ldg(v_lambda);
            float f[16];
            unpack8(keep[l8], f);
            unpack8(keep[8 + l8], f + 8);
#pragma unroll
            for (int i = 0; i < 16; ++i) x[i] = fmaf(lam, f[i], (1.0f - lam) * x[i]);
          }
        }
        if (!cache_row()) continue;
        dst = (is_k ? k_cache : v_cache) + cache_off + (size_t)(is_k ? head - nq : head - nq - nkv) * page_size * d;
      }
      reinterpret_cast<uint4*>(dst)[l8] = pack8(x);
      reinterpret_cast<uint4*>(dst)[8 + l8] = pack8(x + 8);
      continue;
    }
    // (every lane takes part in the exchange; a head past the end holds zeros)
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < 16; ++i) ss = fmaf(x[i], x[i], ss);
    ss += __shfl_xor_sync(0xffffffffu, ss, 1);
    ss += __shfl_xor_sync(0xffffffffu, ss, 2);
    ss += __shfl_xor_sync(0xffffffffu, ss, 4);
    if (!valid) continue;
    if (w != nullptr) {
      const float inv = 1.0f / sqrtf(ss / (float)d + eps);
      float wl[8], wh[8];
      weight8(w, 0, wl);
      weight8(w, 1, wh);
#pragma unroll
      for (int i = 0; i < 8; ++i) { x[i] = x[i] * inv * wl[i]; x[8 + i] = x[8 + i] * inv * wh[i]; }
    }
    if ((is_q || is_k) && rope_table != nullptr) {
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float a = x[i], b = x[8 + i];
        // Products and sums rounded separately, as the reference's scalar code does.
        x[i] = __fsub_rn(__fmul_rn(a, cs[i].x), __fmul_rn(b, cs[i].y));
        x[8 + i] = __fadd_rn(__fmul_rn(a, cs[i].y), __fmul_rn(b, cs[i].x));
      }
    }
    __nv_bfloat16* dst;
    if (is_q) dst = q_out + (size_t)t * q_out_stride + (size_t)head * d;
    else {
      if (!cache_row()) continue;
      dst = (is_k ? k_cache : v_cache) + cache_off + (size_t)(is_k ? head - nq : head - nq - nkv) * page_size * d;
    }
    reinterpret_cast<uint4*>(dst)[l8] = pack8(x);
    reinterpret_cast<uint4*>(dst)[8 + l8] = pack8(x + 8);
  }
}

// dtype: element type of qkv and q_out; cache_dtype: element type of the cache.
// q_weight / k_weight may be null (no weighted per-head norm); rope_table may be null (no
// rotation); k_cache / v_cache may be null (this layer does not write a cache).  Keys have
// head size d, values dv (the V cache is [pages, nkv, page_size, dv]); `mode` and `v_mode`
// are described above the kernel.
ILB_EXPORT int ilb_qk_norm_rope_cache(
    const void* qkv, void* q_out, int dtype, const float* q_weight, const float* k_weight,
    float eps, const float* rope_table, int rotary_dim, const int* positions,
    const int* seq_of_token, const int* block_table, int max_blocks, int page_size,
    int num_pages, void* k_cache, void* v_cache, int cache_dtype, int n_tokens, int nq, int nkv,
    int d, int dv, int qkv_stride, int q_out_stride, int mode, int v_mode, const float* v_lambda, void* v_first,
    cudaStream_t stream) {
  ILB_REQUIRE(n_tokens >= 0 && nq > 0 && nkv > 0 && d > 0 && dv > 0, "qk_norm_rope: bad sizes");
  ILB_REQUIRE(d <= 1024 && dv <= 1024, "qk_norm_rope: head size %d / %d exceeds 1024", d, dv);
  ILB_REQUIRE(rope_table == nullptr || (rotary_dim > 0 && rotary_dim % 2 == 0 && rotary_dim <= d),
              "qk_norm_rope: rotary dimension %d must be even and at most the head size %d",
              rotary_dim, d);
  ILB_REQUIRE(qkv_stride >= (nq + nkv) * d + nkv * dv && q_out_stride >= nq * d,
              "qk_norm_rope: strides too small");
  ILB_REQUIRE((k_cache == nullptr) == (v_cache == nullptr), "qk_norm_rope: need both caches or none");
  ILB_REQUIRE(k_cache == nullptr || (page_size > 0 && max_blocks > 0 && num_pages > 0),
              "qk_norm_rope: bad cache geometry");
  ILB_REQUIRE(dtype == cache_dtype || k_cache == nullptr || (dtype == kF32 && cache_dtype == kBF16) ||
              (dtype == kBF16 && cache_dtype == kF32), "qk_norm_rope: unknown dtypes");
  ILB_REQUIRE(mode >= 0 && mode < 8 && v_mode >= 0 && v_mode <= 2, "qk_norm_rope: unknown mode %d / %d", mode, v_mode);
  ILB_REQUIRE(v_mode == 0 || v_first != nullptr, "qk_norm_rope: value mixing needs the buffer of the first values");
  ILB_REQUIRE(v_mode != 2 || v_lambda != nullptr, "qk_norm_rope: value mixing needs its coefficient");
  if (n_tokens == 0) return 0;
  const bool stock = mode == 0 && v_mode == 0;
  if (dtype == kBF16 && (cache_dtype == kBF16 || k_cache == nullptr) && d == 128 && dv == 128 &&
      (rope_table == nullptr || rotary_dim == d || (mode & kPairsInterleaved)) && ((uintptr_t)v_first % 16 == 0) &&
      qkv_stride % 8 == 0 && q_out_stride % 8 == 0 && ((uintptr_t)qkv % 16 == 0) && ((uintptr_t)q_out % 16 == 0) &&
      ((uintptr_t)k_cache % 16 == 0) && ((uintptr_t)v_cache % 16 == 0) && ((uintptr_t)rope_table % 16 == 0) &&
      ((uintptr_t)q_weight % 16 == 0) && ((uintptr_t)k_weight % 16 == 0)) {
    // CTAs per token: one takes kFastWarps x 4 heads per pass and up to kFastUnroll passes; more
    // CTAs when the heads need them, and when the tokens are too few to fill the device
    const int heads = nq + 2 * nkv, per_pass = kFastWarps * 4;
    int ny = (heads + per_pass * kFastUnroll - 1) / (per_pass * kFastUnroll);
    const int most = (heads + per_pass - 1) / per_pass;
    while (ny < most && (long long)n_tokens * ny < 1184) ++ny;
    if (stock)
      ilb::launch(qk_norm_rope_d128_kernel<false>, dim3(n_tokens, ny), dim3(kFastWarps * 32), 0, stream,
                  (const __nv_bfloat16*)qkv, (__nv_bfloat16*)q_out, q_weight, k_weight, eps, (const float2*)rope_table,
                  positions, seq_of_token, block_table, max_blocks, page_size, num_pages, (__nv_bfloat16*)k_cache,
                  (__nv_bfloat16*)v_cache, nq, nkv, qkv_stride, q_out_stride, 0, d, 0, (const float*)nullptr, (__nv_bfloat16*)nullptr);
    else
      ilb::launch(qk_norm_rope_d128_kernel<true>, dim3(n_tokens, ny), dim3(kFastWarps * 32), 0, stream,
                  (const __nv_bfloat16*)qkv, (__nv_bfloat16*)q_out, q_weight, k_weight, eps, (const float2*)rope_table,
                  positions, seq_of_token, block_table, max_blocks, page_size, num_pages, (__nv_bfloat16*)k_cache,
                  (__nv_bfloat16*)v_cache, nq, nkv, qkv_stride, q_out_stride, mode, rope_table ? rotary_dim : 0, v_mode, v_lambda,
                  (__nv_bfloat16*)v_first);
    return check_launch("qk_norm_rope_cache");
  }
  dim3 grid(n_tokens, (nq + 2 * nkv + kWarpsPerBlock - 1) / kWarpsPerBlock);
  const size_t smem = (size_t)kWarpsPerBlock * (d > dv ? d : dv) * sizeof(float);
#define ILB_LAUNCH(TQ, TC)                                                                   \
  ilb::launch(qk_norm_rope_kernel<TQ, TC>, dim3(grid), dim3(kWarpsPerBlock * 32), smem, stream,                    \
      (const TQ*)qkv, (TQ*)q_out, q_weight, k_weight, eps, (const float2*)rope_table,         \
      rotary_dim, positions, seq_of_token, block_table, max_blocks, page_size, num_pages,     \
      (TC*)k_cache, (TC*)v_cache, n_tokens, nq, nkv, d, dv, qkv_stride, q_out_stride, mode, v_mode,     \
      v_lambda, (TQ*)v_first)
  if (dtype == kF32 && cache_dtype == kF32) ILB_LAUNCH(float, float);
  else if (dtype == kBF16 && cache_dtype == kBF16) ILB_LAUNCH(__nv_bfloat16, __nv_bfloat16);
  else if (dtype == kF32 && cache_dtype == kBF16) ILB_LAUNCH(float, __nv_bfloat16);
  else if (dtype == kBF16 && cache_dtype == kF32) ILB_LAUNCH(__nv_bfloat16, float);
  else return fail("qk_norm_rope: unsupported dtypes %d/%d", dtype, cache_dtype);
#undef ILB_LAUNCH
  return check_launch("qk_norm_rope_cache");
}

// ---------------------------------------------------------------- norms over whole rows, turned values
// The input stage of an attention whose query norm is taken over ALL query heads' elements at once and its key norm
// over all key heads' (weights [nq * d] and [nkv * d]), and whose values may be turned too:
//   q <- turn(q / sqrt(mean(q^2) + eps) * wq),  k likewise,  v <- turn_v(v)
// turn: the first `rotary_dim` elements of a head in pairs (i, i + rotary_dim / 2) by `rope`; turn_v: all dv elements
// of a value in pairs (i, i + dv / 2) by `v_rope`.  Either table may be null.
// A row's units of VEC elements are dealt to gridDim.y blocks; every one of them takes the row's sums itself.
// POOL (steps of single tokens only): a token that completes a block of `pool` positions also writes the block's mean key
// and value (its own and the ones before it in the cache) to row pos / pool of the pooled pages; see pool_means below.
template <typename T, int VEC> struct RowUnit;
template <typename T> struct RowUnit<T, 1> {
  __device__ static __forceinline__ void load(const T* p, float* x) { x[0] = to_float(*p); }
  __device__ static __forceinline__ void store(T* p, const float* x) { *p = from_float<T>(x[0]); }
};
template <> struct RowUnit<__nv_bfloat16, 8> {
  __device__ static __forceinline__ void load(const __nv_bfloat16* p, float* x) { unpack8(*reinterpret_cast<const uint4*>(p), x); }
  __device__ static __forceinline__ void store(__nv_bfloat16* p, const float* x) { *reinterpret_cast<uint4*>(p) = pack8(x); }
};

// N consecutive 32-bit numbers; in fours (from a 16-byte boundary) where N is a multiple of eight.
template <int N>
__device__ __forceinline__ void load_f32(const float* p, float* x) {
  if constexpr (N % 8 == 0) {
#pragma unroll
    for (int i = 0; i < N / 4; ++i) {
      const float4 v = __ldg(reinterpret_cast<const float4*>(p) + i);
      x[4 * i] = v.x; x[4 * i + 1] = v.y; x[4 * i + 2] = v.z; x[4 * i + 3] = v.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) x[i] = p[i];
  }
}

struct RowsParams {
  const float* q_weight; const float* k_weight;
  const float2* rope; const float2* v_rope;
  const int* positions; const int* seq_of_token; const int* block_table;
  int max_blocks, page_size, num_pages, nq, nkv, d, dv, rotary_dim, qkv_stride, q_out_stride;
  float eps;
  const int* p_table; int p_num_pages, pool;
};

constexpr int kRowsThreads = 256;

template <typename TQ, typename TC, int VEC, bool POOL>
__global__ void __launch_bounds__(kRowsThreads)
rows_norm_rope_kernel(const TQ* __restrict__ qkv, TQ* __restrict__ q_out, TC* k_cache, TC* v_cache, TC* pk_cache, TC* pv_cache,
                      const RowsParams p) {
  ilb::pdl_launch_dependents();
  ilb::pdl_wait();
  __shared__ float scratch[33];
  const int t = blockIdx.x;
  const TQ* row = qkv + (size_t)t * p.qkv_stride;
  const int nqd = p.nq * p.d, nkd = p.nkv * p.d, nvd = p.nkv * p.dv;
  float x[VEC], y[VEC];
  float sum_q = 0.f, sum_k = 0.f;
  constexpr int kFlight = 4;                               // units whose loads are in flight together
  for (int e0 = threadIdx.x * VEC; e0 < nqd + nkd; e0 += kFlight * kRowsThreads * VEC) {
    float v[kFlight][VEC];
#pragma unroll
    for (int f = 0; f < kFlight; ++f) {
      const int e = e0 + f * kRowsThreads * VEC;
      if (e < nqd + nkd) RowUnit<TQ, VEC>::load(row + e, v[f]);
      else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[f][i] = 0.f;
      }
    }
#pragma unroll
    for (int f = 0; f < kFlight; ++f) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss = fmaf(v[f][i], v[f][i], ss);
      if (e0 + f * kRowsThreads * VEC < nqd) sum_q += ss; else sum_k += ss;
    }
  }
  // both sums over the block in one exchange
  sum_q = warp_sum(sum_q);
  sum_k = warp_sum(sum_k);
  if ((threadIdx.x & 31) == 0) { scratch[threadIdx.x >> 5] = sum_q; scratch[16 + (threadIdx.x >> 5)] = sum_k; }
  __syncthreads();
  sum_q = 0.f; sum_k = 0.f;
#pragma unroll
  for (int w = 0; w < kRowsThreads / 32; ++w) { sum_q += scratch[w]; sum_k += scratch[16 + w]; }
  const float inv_q = 1.0f / sqrtf(sum_q / (float)nqd + p.eps);
  const float inv_k = 1.0f / sqrtf(sum_k / (float)nkd + p.eps);
  // where this token's key and value go
  long long place = -1;
  if (k_cache != nullptr) {
    const int pos = p.positions[t], blk = pos / p.page_size;
    if (blk >= 0 && blk < p.max_blocks) {
      const int page = p.block_table[(size_t)p.seq_of_token[t] * p.max_blocks + blk];
      if (page >= 0 && page < p.num_pages) place = (long long)page * p.nkv * p.page_size + pos % p.page_size;      // never write outside the pool
    }
  }
  long long pooled_place = -1;                             // where the block's mean goes, if this token completes one
  int first = 0, pos = 0;
  if constexpr (POOL) {
    pos = p.positions[t];
    if (place >= 0 && (pos + 1) % p.pool == 0) {
      const int b = pos / p.pool;
      first = b * p.pool;
      if (b / p.page_size < p.max_blocks) {
        const int page = p.p_table[(size_t)p.seq_of_token[t] * p.max_blocks + b / p.page_size];
        if (page >= 0 && page < p.p_num_pages) pooled_place = (long long)page * p.nkv * p.page_size + b % p.page_size;
      }
    }
  }
  const int units = (nqd + nkd + nvd) / VEC;
  for (int u = blockIdx.y * kRowsThreads + threadIdx.x; u < units; u += gridDim.y * kRowsThreads) {
    int e = u * VEC;
    const int kind = e < nqd ? 0 : (e < nqd + nkd ? 1 : 2);
    if (kind != 0 && place < 0) continue;
    e -= kind == 0 ? 0 : (kind == 1 ? nqd : nqd + nkd);
    const int width = kind == 2 ? p.dv : p.d;
    const int h = e / width, c = e % width;
    const float2* table = kind == 2 ? p.v_rope : p.rope;
    const int half = kind == 2 ? p.dv / 2 : p.rotary_dim / 2;
    const bool pair = table != nullptr && c < 2 * half;
    if (pair && c >= half) continue;                       // the pair's first member writes both
    const TQ* src = row + u * VEC;
    RowUnit<TQ, VEC>::load(src, x);
    if (pair) RowUnit<TQ, VEC>::load(src + half, y);
    if (kind != 2) {
      const float inv = kind == 0 ? inv_q : inv_k;
      const float* w = (kind == 0 ? p.q_weight : p.k_weight) + e;
      float wv[VEC];
      load_f32<VEC>(w, wv);
#pragma unroll
      for (int i = 0; i < VEC; ++i) x[i] = x[i] * inv * wv[i];
      if (pair) {
        load_f32<VEC>(w + half, wv);
#pragma unroll
        for (int i = 0; i < VEC; ++i) y[i] = y[i] * inv * wv[i];
      }
    }
    if (pair) {
      float cs[2 * VEC];
      load_f32<2 * VEC>(reinterpret_cast<const float*>(table + (size_t)t * half + c), cs);
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        const float a = x[i], b = y[i];
        const float2 w = make_float2(cs[2 * i], cs[2 * i + 1]);
        x[i] = __fsub_rn(__fmul_rn(a, w.x), __fmul_rn(b, w.y));
        y[i] = __fadd_rn(__fmul_rn(a, w.y), __fmul_rn(b, w.x));
      }
    }
    if (kind == 0) {
      TQ* dst = q_out + (size_t)t * p.q_out_stride + e;
      RowUnit<TQ, VEC>::store(dst, x);
      if (pair) RowUnit<TQ, VEC>::store(dst + half, y);
    } else {
      TC* cache = kind == 1 ? k_cache : v_cache;
      TC* dst = cache + ((size_t)place + (size_t)h * p.page_size) * width + c;
      RowUnit<TC, VEC>::store(dst, x);
      if (pair) RowUnit<TC, VEC>::store(dst + half, y);
      if constexpr (POOL) {
        if (pooled_place >= 0) {
          const int* table = p.block_table + (size_t)p.seq_of_token[t] * p.max_blocks;
          TC* mean = (kind == 1 ? pk_cache : pv_cache) + ((size_t)pooled_place + (size_t)h * p.page_size) * width + c;
          for (int member = 0; member < (pair ? 2 : 1); ++member) {
            const int off = member * half;
            float sum[VEC], own[VEC];
#pragma unroll
            for (int i = 0; i < VEC; ++i) { sum[i] = 0.f; own[i] = to_float(from_float<TC>(member ? y[i] : x[i])); }
            constexpr int kFlight = 4;                     // rows whose loads are in flight together
            for (int j0 = first; j0 < pos; j0 += kFlight) {
              float r[kFlight][VEC];
#pragma unroll
              for (int f = 0; f < kFlight; ++f) {
                const int j = j0 + f;
                const int page = j < pos ? table[j / p.page_size] : -1;
                if (page >= 0 && page < p.num_pages)
                  RowUnit<TC, VEC>::load(cache + (((size_t)page * p.nkv + h) * p.page_size + j % p.page_size) * width + c + off, r[f]);
                else {
#pragma unroll
                  for (int i = 0; i < VEC; ++i) r[f][i] = 0.f;
                }
              }
#pragma unroll
              for (int f = 0; f < kFlight; ++f)
#pragma unroll
                for (int i = 0; i < VEC; ++i) sum[i] += r[f][i];
            }
#pragma unroll
            for (int i = 0; i < VEC; ++i) sum[i] = (sum[i] + own[i]) / (float)p.pool;
            RowUnit<TC, VEC>::store(mean + off, sum);
          }
        }
      }
    }
  }
}

ILB_EXPORT int ilb_rows_norm_rope_cache(
    const void* qkv, void* q_out, int dtype, const float* q_weight, const float* k_weight, float eps, const float* rope,
    int rotary_dim, const float* v_rope, const int* positions, const int* seq_of_token, const int* block_table, int max_blocks,
    int page_size, int num_pages, void* k_cache, void* v_cache, int n_tokens, int nq, int nkv, int d, int dv, int qkv_stride,
    int q_out_stride, void* pk_cache, void* pv_cache, const int* p_table, int p_num_pages, int pool, cudaStream_t stream) {
  ILB_REQUIRE(n_tokens >= 0 && nq > 0 && nkv > 0 && d > 0 && dv > 0 && eps > 0.f, "rows_norm_rope: bad sizes");
  ILB_REQUIRE(q_weight != nullptr && k_weight != nullptr, "rows_norm_rope: the norms' weights are missing");
  ILB_REQUIRE(rope == nullptr || (rotary_dim > 0 && rotary_dim % 2 == 0 && rotary_dim <= d),
              "rows_norm_rope: rotary dimension %d must be even and at most the head size %d", rotary_dim, d);
  ILB_REQUIRE(v_rope == nullptr || dv % 2 == 0, "rows_norm_rope: values of %d elements cannot be turned in pairs", dv);
  ILB_REQUIRE(qkv_stride >= (nq + nkv) * d + nkv * dv && q_out_stride >= nq * d, "rows_norm_rope: strides too small");
  ILB_REQUIRE((k_cache == nullptr) == (v_cache == nullptr), "rows_norm_rope: need both caches or none");
  ILB_REQUIRE(k_cache == nullptr || (page_size > 0 && max_blocks > 0 && num_pages > 0), "rows_norm_rope: bad cache geometry");
  ILB_REQUIRE(dtype == kF32 || dtype == kBF16, "rows_norm_rope: unknown dtype %d", dtype);
  ILB_REQUIRE(pool == 0 || (pool > 0 && k_cache != nullptr && pk_cache != nullptr && pv_cache != nullptr && p_table != nullptr && p_num_pages > 0),
              "rows_norm_rope: pooled rows need both sets of pages");
  if (n_tokens == 0) return 0;
  const RowsParams p{q_weight, k_weight, (const float2*)rope, (const float2*)v_rope, positions, seq_of_token, block_table, max_blocks,
                     page_size, num_pages, nq, nkv, d, dv, rope != nullptr ? rotary_dim : 0, qkv_stride, q_out_stride, eps, p_table, p_num_pages, pool};
  auto a16 = [](const void* x) { return (uintptr_t)x % 16 == 0; };
  const bool vec = dtype == kBF16 && d % 8 == 0 && dv % 8 == 0 && (rope == nullptr || rotary_dim % 16 == 0) && (v_rope == nullptr || dv % 16 == 0) &&
                   qkv_stride % 8 == 0 && q_out_stride % 8 == 0 && a16(qkv) && a16(q_out) && a16(k_cache) && a16(v_cache) && a16(pk_cache) && a16(pv_cache) && a16(q_weight) && a16(k_weight) && a16(rope) && a16(v_rope);
  const int units = ((nq + nkv) * d + nkv * dv) / (vec ? 8 : 1);
  int ny = 1;
  while (n_tokens * ny < 296 && ny * kRowsThreads < units) ++ny;
  const dim3 grid(n_tokens, ny);
#define ILB_ROWS(T, V, POOL) ilb::launch(rows_norm_rope_kernel<T, T, V, POOL>, grid, dim3(kRowsThreads), 0, stream, (const T*)qkv, (T*)q_out, \
                                         (T*)k_cache, (T*)v_cache, (T*)pk_cache, (T*)pv_cache, p)
  if (vec) { if (pool) ILB_ROWS(__nv_bfloat16, 8, true); else ILB_ROWS(__nv_bfloat16, 8, false); }
  else if (dtype == kBF16) { if (pool) ILB_ROWS(__nv_bfloat16, 1, true); else ILB_ROWS(__nv_bfloat16, 1, false); }
  else { if (pool) ILB_ROWS(float, 1, true); else ILB_ROWS(float, 1, false); }
#undef ILB_ROWS
  return check_launch("rows_norm_rope_cache");
}

// ---------------------------------------------------------------- short convolutions, then norms over whole rows
// The same input stage for queries and keys that pass a causal convolution per channel first:
//   u_t = sum_j w[j, c] raw_{t - (taps - 1) + j},   q <- turn(u_q / sqrt(mean(u_q^2) + eps) * wq),   k likewise
// and values that are either columns of their own behind q | k, as they are, or (values_are_keys) u_k before its norm.
// The raw inputs ahead of the step come from state [slots, taps - 1, (nq + nkv) d] 32-bit; zeros before the sequence's start.
// A block takes up to TT consecutive tokens of a sequence: a thread owns units of VEC channels, has the raw inputs of all its
// taps and tokens in flight together, and the convolved rows wait in shared memory for their sums.  A sequence of one token is
// one block, which also moves the state on; the state of the others is moved on by a second launch, when nobody reads the old
// one any more.
constexpr int kMostTaps = 16;
constexpr int kConvTile = 4;                             // tokens of a sequence per block (1 for rows that would not fit shared memory so often)

struct ConvRowsParams {
  RowsParams r;
  const float* conv_w;               // [taps, (nq + nkv) d]
  float* state;
  const int* cu_q; const int* slots;
  int n_seqs, taps, values_are_keys;
};

// VEC raw inputs as they are stored.  (The state keeps them widened: a bfloat16 input comes back from there without loss.)
template <typename T, int VEC> struct RawUnit;
template <typename T> struct RawUnit<T, 1> {
  float v;
  __device__ __forceinline__ void zero() { v = 0.f; }
  __device__ __forceinline__ void load(const T* p) { v = to_float(*p); }
  __device__ __forceinline__ void load_state(const float* p) { v = *p; }
  __device__ __forceinline__ void get(float* x) const { x[0] = v; }
  __device__ __forceinline__ void store_state(float* p) const { *p = v; }
};
template <> struct RawUnit<__nv_bfloat16, 8> {
  uint4 v;
  __device__ __forceinline__ void zero() { v = make_uint4(0u, 0u, 0u, 0u); }
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { v = *reinterpret_cast<const uint4*>(p); }
  __device__ __forceinline__ void load_state(const float* p) {      // (plain loads: this launch may write the slot)
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    const float x[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
    v = pack8(x);
  }
  __device__ __forceinline__ void get(float* x) const { unpack8(v, x); }
  __device__ __forceinline__ void store_state(float* p) const {
    float x[8];
    unpack8(v, x);
    reinterpret_cast<float4*>(p)[0] = make_float4(x[0], x[1], x[2], x[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(x[4], x[5], x[6], x[7]);
  }
};

// MT: the most taps (taps <= MT; the taps are aligned to its end).
template <typename T, int VEC, int MT, int TT>
__global__ void __launch_bounds__(512)
conv_rows_norm_kernel(const T* __restrict__ qkv, T* __restrict__ q_out, T* k_cache, T* v_cache, const ConvRowsParams c) {
  ilb::pdl_launch_dependents();
  ilb::pdl_wait();
  const RowsParams& p = c.r;
  extern __shared__ __align__(16) float u[];             // [TT][(nq + nkv) d]
  __shared__ float scratch[2 * TT * 16];
  __shared__ long long places[TT];
  __shared__ float inv[2 * TT];
  int seq = 0, tile = blockIdx.x;
  for (; seq < c.n_seqs; ++seq) {
    const int n = (c.cu_q[seq + 1] - c.cu_q[seq] + TT - 1) / TT;
    if (tile < n) break;
    tile -= n;
  }
  if (seq >= c.n_seqs) return;
  const int tok0 = c.cu_q[seq], q_len = c.cu_q[seq + 1] - tok0, slot = c.slots[seq];
  const int lt0 = tile * TT, ts = min(TT, q_len - lt0), t0 = tok0 + lt0;
  const int nqd = p.nq * p.d, nkd = p.nkv * p.d, width = nqd + nkd, before = c.taps - 1, skip = MT - c.taps;
  float* own = slot >= 0 ? c.state + (size_t)slot * before * width : nullptr;
  const int warps = blockDim.x / 32, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x < ts) {                                // where each token's key and value go
    long long place = -1;
    if (k_cache != nullptr) {
      const int pos = p.positions[t0 + threadIdx.x], blk = pos / p.page_size;
      if (blk >= 0 && blk < p.max_blocks) {
        const int page = p.block_table[(size_t)seq * p.max_blocks + blk];
        if (page >= 0 && page < p.num_pages) place = (long long)page * p.nkv * p.page_size + pos % p.page_size;      // never write outside the pool
      }
    }
    places[threadIdx.x] = place;
  }
  float sum_q[TT], sum_k[TT];
#pragma unroll
  for (int tt = 0; tt < TT; ++tt) { sum_q[tt] = 0.f; sum_k[tt] = 0.f; }
  for (int e = threadIdx.x * VEC; e < width; e += blockDim.x * VEC) {
    RawUnit<T, VEC> raw[MT + TT - 1];                    // row r: the token r - (MT - 1) places from the tile's first
#pragma unroll
    for (int r = 0; r < MT + TT - 1; ++r) {
      const int lt = lt0 + r - (MT - 1);
      raw[r].zero();
      if (r >= skip && lt < q_len) {
        if (lt >= 0) raw[r].load(qkv + (size_t)(tok0 + lt) * p.qkv_stride + e);
        else if (own != nullptr) raw[r].load_state(own + (size_t)(before + lt) * width + e);
      }
    }
    float acc[TT][VEC];
#pragma unroll
    for (int tt = 0; tt < TT; ++tt)
#pragma unroll
      for (int i = 0; i < VEC; ++i) acc[tt][i] = 0.f;
#pragma unroll
    for (int j = 0; j < MT; ++j) {
      if (j >= skip) {
        float w[VEC];
        load_f32<VEC>(c.conv_w + (size_t)(j - skip) * width + e, w);
#pragma unroll
        for (int tt = 0; tt < TT; ++tt) {
          float x[VEC];
          raw[j + tt].get(x);
#pragma unroll
          for (int i = 0; i < VEC; ++i) acc[tt][i] = fmaf(w[i], x[i], acc[tt][i]);
        }
      }
    }
    if (q_len == 1 && own != nullptr) {
#pragma unroll
      for (int r = 1; r < MT; ++r)
        if (r > skip) raw[r].store_state(own + (size_t)(r - skip - 1) * width + e);
    }
#pragma unroll
    for (int tt = 0; tt < TT; ++tt) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < VEC; ++i) { u[(size_t)tt * width + e + i] = acc[tt][i]; ss = fmaf(acc[tt][i], acc[tt][i], ss); }
      if (e < nqd) sum_q[tt] += ss; else sum_k[tt] += ss;
    }
  }
#pragma unroll
  for (int tt = 0; tt < TT; ++tt) {
    const float a = warp_sum(sum_q[tt]), b = warp_sum(sum_k[tt]);
    if (lane == 0) { scratch[(2 * tt) * 16 + warp] = a; scratch[(2 * tt + 1) * 16 + warp] = b; }
  }
  __syncthreads();
  if (threadIdx.x < 2 * TT) {
    float a = 0.f;
    for (int w = 0; w < warps; ++w) a += scratch[threadIdx.x * 16 + w];
    inv[threadIdx.x] = 1.0f / sqrtf(a / (float)((threadIdx.x & 1) ? nkd : nqd) + p.eps);
  }
  __syncthreads();
  const int half = p.rotary_dim / 2;
  for (int e = threadIdx.x * VEC; e < width; e += blockDim.x * VEC) {
    const bool is_q = e < nqd;
    const int r = is_q ? e : e - nqd, h = r / p.d, ch = r % p.d;
    const bool turned = p.rope != nullptr && ch < 2 * half;
    const int o = ch < half ? half : -half;              // the pair's other member
    float w[VEC], w2[VEC];
    load_f32<VEC>((is_q ? p.q_weight : p.k_weight) + r, w);
    if (turned) load_f32<VEC>((is_q ? p.q_weight : p.k_weight) + r + o, w2);
#pragma unroll
    for (int tt = 0; tt < TT; ++tt) {
      if (tt >= ts) break;
      const long long place = places[tt];
      if (!is_q && place < 0) continue;
      const float f = inv[2 * tt + (is_q ? 0 : 1)];
      const float* ut = u + (size_t)tt * width + e;
      float x[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) x[i] = ut[i];
      if (!is_q && c.values_are_keys) RowUnit<T, VEC>::store(v_cache + ((size_t)place + (size_t)h * p.page_size) * p.dv + ch, x);
#pragma unroll
      for (int i = 0; i < VEC; ++i) x[i] = x[i] * f * w[i];
      if (turned) {
        float cs[2 * VEC];
        load_f32<2 * VEC>(reinterpret_cast<const float*>(p.rope + (size_t)(t0 + tt) * half + (ch < half ? ch : ch - half)), cs);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          const float y = ut[o + i] * f * w2[i];
          x[i] = __fadd_rn(__fmul_rn(x[i], cs[2 * i]), __fmul_rn(y, ch < half ? -cs[2 * i + 1] : cs[2 * i + 1]));
        }
      }
      if (is_q) RowUnit<T, VEC>::store(q_out + (size_t)(t0 + tt) * p.q_out_stride + r, x);
      else RowUnit<T, VEC>::store(k_cache + ((size_t)place + (size_t)h * p.page_size) * p.d + ch, x);
    }
  }
  if (c.values_are_keys) return;
  for (int e = threadIdx.x * VEC; e < p.nkv * p.dv * ts; e += blockDim.x * VEC) {
    const int tt = e / (p.nkv * p.dv), r = e % (p.nkv * p.dv);
    if (places[tt] < 0) continue;
    float x[VEC];
    RowUnit<T, VEC>::load(qkv + (size_t)(t0 + tt) * p.qkv_stride + width + r, x);
    RowUnit<T, VEC>::store(v_cache + ((size_t)places[tt] + (size_t)(r / p.dv) * p.page_size) * p.dv + r % p.dv, x);
  }
}

// The sequences that bring several tokens: state <- their last taps - 1 raw inputs.
template <typename T>
__global__ void __launch_bounds__(256)
conv_rows_state_kernel(const T* __restrict__ qkv, int ld, int width, int before, float* __restrict__ state, const int* __restrict__ cu_q,
                       const int* __restrict__ slots) {
  ilb::pdl_launch_dependents();
  ilb::pdl_wait();
  const int seq = blockIdx.y, e = blockIdx.x * 256 + threadIdx.x;
  const int tok0 = cu_q[seq], n = cu_q[seq + 1] - tok0, slot = slots[seq];
  if (e >= width || n <= 1 || slot < 0) return;
  float* own = state + (size_t)slot * before * width + e;
  for (int j = 0; j < before; ++j) {                     // (rows behind j are still the old ones)
    const int at = n - before + j;
    own[(size_t)j * width] = at >= 0 ? to_float(qkv[(size_t)(tok0 + at) * ld + e]) : own[(size_t)(j + n) * width];
  }
}

// qkv [T, qkv_stride] of `dtype`: raw q | k (| v); n_tiles: the sum over the sequences of ceil(tokens / 4); several: whether a
// sequence of the step brings more than one token.
ILB_EXPORT int ilb_conv_rows_norm_cache(
    const void* qkv, void* q_out, int dtype, const float* conv_w, int taps, float* state, const float* q_weight, const float* k_weight,
    float eps, const float* rope, int rotary_dim, const int* positions, const int* seq_of_token, const int* cu_q, const int* slots,
    int n_seqs, int n_tiles, int several, const int* block_table, int max_blocks, int page_size, int num_pages, void* k_cache, void* v_cache,
    int n_tokens, int nq, int nkv, int d, int dv, int qkv_stride, int q_out_stride, int values_are_keys, cudaStream_t stream) {
  ILB_REQUIRE(n_tokens >= 0 && nq > 0 && nkv > 0 && d > 0 && dv > 0 && eps > 0.f && n_seqs >= 0 && n_seqs <= 65535, "conv_rows_norm: bad sizes");
  ILB_REQUIRE(conv_w != nullptr && taps >= 1 && taps <= kMostTaps && (taps == 1 || state != nullptr), "conv_rows_norm: %d taps (at most %d) need weights and a state", taps, kMostTaps);
  ILB_REQUIRE(q_weight != nullptr && k_weight != nullptr, "conv_rows_norm: the norms' weights are missing");
  ILB_REQUIRE(rope == nullptr || (rotary_dim > 0 && rotary_dim % 2 == 0 && rotary_dim <= d),
              "conv_rows_norm: rotary dimension %d must be even and at most the head size %d", rotary_dim, d);
  ILB_REQUIRE(!values_are_keys || dv == d, "conv_rows_norm: values that are keys have the keys' head size, found %d and %d", dv, d);
  const int width = (nq + nkv) * d;
  ILB_REQUIRE(qkv_stride >= width + (values_are_keys ? 0 : nkv * dv) && q_out_stride >= nq * d, "conv_rows_norm: strides too small");
  ILB_REQUIRE((k_cache == nullptr) == (v_cache == nullptr), "conv_rows_norm: need both caches or none");
  ILB_REQUIRE(k_cache == nullptr || (page_size > 0 && max_blocks > 0 && num_pages > 0), "conv_rows_norm: bad cache geometry");
  ILB_REQUIRE(dtype == kF32 || dtype == kBF16, "conv_rows_norm: unknown dtype %d", dtype);
  constexpr int kMost = 200 * 1024;
  // (single tokens, and rows of many channels, go a token a block)
  const int tile = several && (size_t)kConvTile * width * sizeof(float) <= 100 * 1024 ? kConvTile : 1;
  const size_t smem = sizeof(float) * width * tile;
  ILB_REQUIRE(smem <= kMost, "conv_rows_norm: rows of %d channels do not fit shared memory", width);
  if (n_tokens == 0) return 0;
  ConvRowsParams c{};
  c.r.q_weight = q_weight; c.r.k_weight = k_weight; c.r.rope = (const float2*)rope; c.r.positions = positions; c.r.seq_of_token = seq_of_token;
  c.r.block_table = block_table; c.r.max_blocks = max_blocks; c.r.page_size = page_size; c.r.num_pages = num_pages; c.r.nq = nq; c.r.nkv = nkv;
  c.r.d = d; c.r.dv = dv; c.r.rotary_dim = rope != nullptr ? rotary_dim : 0; c.r.qkv_stride = qkv_stride; c.r.q_out_stride = q_out_stride; c.r.eps = eps;
  c.conv_w = conv_w; c.state = state; c.cu_q = cu_q; c.slots = slots; c.n_seqs = n_seqs; c.taps = taps; c.values_are_keys = values_are_keys;
  auto a16 = [](const void* x) { return (uintptr_t)x % 16 == 0; };
  const bool vec = dtype == kBF16 && d % 8 == 0 && dv % 8 == 0 && (rope == nullptr || rotary_dim % 16 == 0) && qkv_stride % 8 == 0 && q_out_stride % 8 == 0 &&
                   a16(qkv) && a16(q_out) && a16(k_cache) && a16(v_cache) && a16(q_weight) && a16(k_weight) && a16(conv_w) && a16(state) && a16(rope);
  // (tiles of several tokens: small blocks, of which enough fit a multiprocessor to hide each other's loads)
  const int units = width / (vec ? 8 : 1), most = tile == kConvTile ? 128 : 512, threads = units >= most ? most : (units + 31) / 32 * 32;
  const int blocks = tile == kConvTile ? n_tiles : n_tokens;
#define ILB_CR(T, V, MT, TT)                                                                                                        \
  do {                                                                                                                              \
    static OncePerDevice once;                                                                                                      \
    if (smem > 48 * 1024 && once.first() &&                                                                                         \
        cudaFuncSetAttribute(conv_rows_norm_kernel<T, V, MT, TT>, cudaFuncAttributeMaxDynamicSharedMemorySize, kMost) != cudaSuccess) { \
      once.forget();                                                                                                                \
      return fail("conv_rows_norm: cannot reserve %d bytes of shared memory", kMost);                                               \
    }                                                                                                                               \
    ilb::launch(conv_rows_norm_kernel<T, V, MT, TT>, dim3(blocks), dim3(threads), smem, stream, (const T*)qkv, (T*)q_out, (T*)k_cache, \
                (T*)v_cache, c);                                                                                                    \
  } while (0)
#define ILB_CRT(T, V, MT) do { if (tile == kConvTile) ILB_CR(T, V, MT, kConvTile); else ILB_CR(T, V, MT, 1); } while (0)
  if (vec && taps <= 4) ILB_CRT(__nv_bfloat16, 8, 4);
  else if (dtype == kBF16) ILB_CRT(__nv_bfloat16, 1, kMostTaps);
  else ILB_CRT(float, 1, kMostTaps);
#undef ILB_CRT
#undef ILB_CR
  if (int rc = check_launch("conv_rows_norm")) return rc;
  if (!several || taps == 1 || n_seqs == 0) return 0;
  const dim3 grid((width + 255) / 256, n_seqs);
  if (dtype == kF32) ilb::launch(conv_rows_state_kernel<float>, grid, dim3(256), 0, stream, (const float*)qkv, qkv_stride, width, taps - 1, state, cu_q, slots);
  else ilb::launch(conv_rows_state_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, (const __nv_bfloat16*)qkv, qkv_stride, width, taps - 1, state, cu_q, slots);
  return check_launch("conv_rows_state");
}

// ---------------------------------------------------------------- means of blocks of cached rows
// The token at position p completes block b = p / pool if (p + 1) % pool == 0: row b of the second set of pages becomes the
// mean (32-bit sum) of the block's `pool` keys and of its values as the cache holds them.  One block of threads per block of
// positions that the step completes (and slice of the channels); eight groups of threads share a block's rows.
constexpr int kMeanRows = 8, kMeanCols = 32;

template <typename T, int VEC>
__global__ void __launch_bounds__(kMeanRows * kMeanCols)
pool_means_kernel(const T* __restrict__ k_cache, const T* __restrict__ v_cache, T* __restrict__ pk_cache, T* __restrict__ pv_cache,
                  const int* __restrict__ positions, const int* __restrict__ cu_q, int n_seqs, const int* __restrict__ block_table,
                  const int* __restrict__ p_table, int max_blocks, int page_size, int num_pages, int p_num_pages, int pool, int nkv,
                  int d, int dv) {
  ilb::pdl_launch_dependents();
  ilb::pdl_wait();
  __shared__ float part[kMeanRows][kMeanCols * VEC];
  int seq = 0, left = blockIdx.x, b = -1;
  for (; seq < n_seqs; ++seq) {
    const int n = cu_q[seq + 1] - cu_q[seq];
    if (n <= 0) continue;
    const int p0 = positions[cu_q[seq]], done = (p0 + n) / pool - p0 / pool;      // blocks whose last position lies in this step
    if (left < done) { b = p0 / pool + left; break; }
    left -= done;
  }
  if (b < 0 || b / page_size >= max_blocks) return;
  const int* table = block_table + (size_t)seq * max_blocks;
  const int p_page = p_table[(size_t)seq * max_blocks + b / page_size];
  if (p_page < 0 || p_page >= p_num_pages) return;          // never write outside the pool
  const int col = threadIdx.x % kMeanCols, grp = threadIdx.x / kMeanCols;
  const int e = (blockIdx.y * kMeanCols + col) * VEC;
  const bool live = e < nkv * (d + dv), is_k = e < nkv * d;
  const int width = is_k ? d : dv, h = (is_k ? e : e - nkv * d) / width, c = (is_k ? e : e - nkv * d) % width;
  const T* src = is_k ? k_cache : v_cache;
  float sum[VEC];
#pragma unroll
  for (int i = 0; i < VEC; ++i) sum[i] = 0.f;
  if (live) {
    for (int j0 = grp; j0 < pool; j0 += 4 * kMeanRows) {    // four rows in flight
      float x[4][VEC];
#pragma unroll
      for (int f = 0; f < 4; ++f) {
        const int j = j0 + f * kMeanRows, pj = b * pool + j;
        const int page = j < pool ? table[pj / page_size] : -1;
        if (page >= 0 && page < num_pages) RowUnit<T, VEC>::load(src + (((size_t)page * nkv + h) * page_size + pj % page_size) * width + c, x[f]);
        else {
#pragma unroll
          for (int i = 0; i < VEC; ++i) x[f][i] = 0.f;
        }
      }
#pragma unroll
      for (int f = 0; f < 4; ++f)
#pragma unroll
        for (int i = 0; i < VEC; ++i) sum[i] += x[f][i];
    }
  }
#pragma unroll
  for (int i = 0; i < VEC; ++i) part[grp][col * VEC + i] = sum[i];
  __syncthreads();
  if (grp != 0 || !live) return;
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    float s = 0.f;
#pragma unroll
    for (int g = 0; g < kMeanRows; ++g) s += part[g][col * VEC + i];
    sum[i] = s / (float)pool;
  }
  RowUnit<T, VEC>::store((is_k ? pk_cache : pv_cache) + (((size_t)p_page * nkv + h) * page_size + b % page_size) * width + c, sum);
}

// n_done: blocks of positions that the step's tokens complete, over all sequences.
ILB_EXPORT int ilb_pool_means(const void* k_cache, const void* v_cache, void* pk_cache, void* pv_cache, int dtype, const int* positions,
                              const int* cu_q, int n_seqs, const int* block_table, const int* p_table, int max_blocks, int page_size,
                              int num_pages, int p_num_pages, int pool, int n_done, int nkv, int d, int dv, cudaStream_t stream) {
  ILB_REQUIRE(n_done >= 0 && n_seqs > 0 && nkv > 0 && d > 0 && dv > 0 && pool > 0, "pool_means: bad sizes");
  ILB_REQUIRE(page_size > 0 && max_blocks > 0 && num_pages > 0 && p_num_pages > 0, "pool_means: bad cache geometry");
  ILB_REQUIRE(k_cache != nullptr && v_cache != nullptr && pk_cache != nullptr && pv_cache != nullptr, "pool_means: a cache is missing");
  if (n_done == 0) return 0;
  auto a16 = [](const void* x) { return (uintptr_t)x % 16 == 0; };
  const bool vec = dtype == kBF16 && d % 8 == 0 && dv % 8 == 0 && a16(k_cache) && a16(v_cache) && a16(pk_cache) && a16(pv_cache);
  const int per = kMeanCols * (vec ? 8 : 1);
  const dim3 grid(n_done, (nkv * (d + dv) + per - 1) / per);
#define ILB_PM(T, V) ilb::launch(pool_means_kernel<T, V>, grid, dim3(kMeanRows * kMeanCols), 0, stream, (const T*)k_cache, (const T*)v_cache, \
                                 (T*)pk_cache, (T*)pv_cache, positions, cu_q, n_seqs, block_table, p_table, max_blocks, page_size, num_pages, \
                                 p_num_pages, pool, nkv, d, dv)
  if (dtype == kF32) ILB_PM(float, 1);
  else if (dtype == kBF16) { if (vec) ILB_PM(__nv_bfloat16, 8); else ILB_PM(__nv_bfloat16, 1); }
  else return fail("pool_means: unknown dtype %d", dtype);
#undef ILB_PM
  return check_launch("pool_means");
}

// ---------------------------------------------------------------- heads turned back, in place
// o[t, h, :] of `dv` elements in pairs (i, i + dv / 2), turned by minus the angle whose (cos, sin) is table[t, i].
template <typename T>
__global__ void __launch_bounds__(256)
turn_back_kernel(T* __restrict__ o, const float2* __restrict__ table, int n_tokens, int heads, int dv) {
  ilb::pdl_launch_dependents();
  ilb::pdl_wait();
  const int half = dv / 2;
  const size_t n = (size_t)n_tokens * heads * half;
  for (size_t i = (size_t)blockIdx.x * 256 + threadIdx.x; i < n; i += (size_t)gridDim.x * 256) {
    const int m = (int)(i % half);
    const size_t th = i / half, t = th / heads;
    T* p = o + th * dv + m;
    const float a = to_float(p[0]), b = to_float(p[half]);
    const float2 w = table[t * half + m];
    p[0] = from_float<T>(__fadd_rn(__fmul_rn(a, w.x), __fmul_rn(b, w.y)));
    p[half] = from_float<T>(__fsub_rn(__fmul_rn(b, w.x), __fmul_rn(a, w.y)));
  }
}

ILB_EXPORT int ilb_turn_back(void* o, int dtype, const float* table, int n_tokens, int heads, int dv, cudaStream_t stream) {
  ILB_REQUIRE(n_tokens >= 0 && heads > 0 && dv > 0 && dv % 2 == 0 && table != nullptr, "turn_back: bad sizes");
  if (n_tokens == 0) return 0;
  const size_t n = (size_t)n_tokens * heads * (dv / 2);
  const int blocks = (int)((n + 255) / 256 < 148 * 16 ? (n + 255) / 256 : 148 * 16);
  if (dtype == kF32) ilb::launch(turn_back_kernel<float>, dim3(blocks), dim3(256), 0, stream, (float*)o, (const float2*)table, n_tokens, heads, dv);
  else if (dtype == kBF16)
    ilb::launch(turn_back_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, (__nv_bfloat16*)o, (const float2*)table, n_tokens, heads, dv);
  else return fail("turn_back: unknown dtype %d", dtype);
  return check_launch("turn_back");
}

ILB_DEFINE_LAST_ERROR()
