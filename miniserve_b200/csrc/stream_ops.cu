// Kernels at the two ends of the residual stream's layers that go beyond one table and one norm:
//
//   * an embedding that is a sum: the token's row (times a constant), a row of a second table chosen by a hash of the previous and the
//     current token (a bigram table; a sequence's first token takes the table's last row), and a sinusoidal vector of
//     the position. The token before a portion's first one comes from the request's state slot (int32), which the CTA of
//     that first token, the only one that reads it, leaves holding the portion's last token;
//   * RMS norm of the stream after an addend that is normed itself: h = residual + norm_b(delta), out = norm(h). Either
//     norm's weight is a vector or one number for all coordinates;
//   * several residual streams (hyper-connections): a sublayer's output y changes all streams at once, x_t <- sum_s mix[s, t] x_s +
//     out[t] y, and the next sublayer reads the norm of sum_s in[s] x_s: both in one pass over the streams.
//
// Angles, statistics, norms and the sums are float32; each output is rounded once.
#include "common.cuh"

namespace ms {

struct PairTable {
  const void* table;  // [buckets + 1, hidden] or null
  long long buckets, mul_prev, mul_cur;
};

// The row of the pair table for flat token t, or -1 without a table. Every thread of the CTA calls it (there is a barrier
// between the read of the slot and its update).
__device__ __forceinline__ long long pair_row(const PairTable& pt, int t, const int* __restrict__ ids, const int* __restrict__ positions,
                                              const int* __restrict__ row_of_token, const int* __restrict__ cu_q,
                                              const int* __restrict__ state_slot, int* __restrict__ prev_token) {
  if (!pt.table) return -1;
  const int row = row_of_token[t];
  const int first = cu_q[row];
  long long out = pt.buckets;
  if (t == first) {
    int* slot = prev_token + state_slot[row];
    const int prev = *slot;
    __syncthreads();
    if (threadIdx.x == 0) *slot = ids[cu_q[row + 1] - 1];
    if (positions[t] > 0) out = ((long long)prev * pt.mul_prev + (long long)ids[t] * pt.mul_cur) % pt.buckets;
  } else {
    out = ((long long)ids[t - 1] * pt.mul_prev + (long long)ids[t] * pt.mul_cur) % pt.buckets;
  }
  // (the host takes no negative factors and ids are valid; stay inside the table anyway)
  return out < 0 ? 0 : out;
}

// inv_freq [(hidden + 1) / 2] float32 or null: entry 2i gets sin(position * inv_freq[i]), entry 2i + 1 the cosine. One CTA per token.
template <typename T>
__global__ void embed_sum_kernel(float* __restrict__ residual, const T* __restrict__ table, PairTable pt, const float* __restrict__ inv_freq,
                                 const int* __restrict__ ids, const int* __restrict__ positions, const int* __restrict__ row_of_token,
                                 const int* __restrict__ cu_q, const int* __restrict__ state_slot, int* __restrict__ prev_token,
                                 int hidden, int vocab, float scale) {
  pdl_prologue();
  const int t = blockIdx.x;
  int id = ids[t];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const long long pr = pair_row(pt, t, ids, positions, row_of_token, cu_q, state_slot, prev_token);
  const T* src = table + (size_t)id * hidden;
  const T* pair = pr < 0 ? nullptr : reinterpret_cast<const T*>(pt.table) + (size_t)pr * hidden;
  float* dst = residual + (size_t)t * hidden;
  const float pos = (float)positions[t];
  for (int i = threadIdx.x; 2 * i < hidden; i += blockDim.x) {
    float sn = 0.f, cs = 0.f;
    if (inv_freq) sincosf(pos * inv_freq[i], &sn, &cs);
    const int c = 2 * i;
    float a = Elem<T>::load(src + c) * scale;
    if (pair) a += Elem<T>::load(pair + c);
    dst[c] = a + sn;
    if (c + 1 < hidden) {
      float b = Elem<T>::load(src + c + 1) * scale;
      if (pair) b += Elem<T>::load(pair + c + 1);
      dst[c + 1] = b + cs;
    }
  }
}

// bfloat16 rows that are a multiple of 8 wide and start on 16 bytes: eight elements per thread and trip
__global__ void embed_sum_bf16x8_kernel(float* __restrict__ residual, const __nv_bfloat16* __restrict__ table, PairTable pt,
                                        const float* __restrict__ inv_freq, const int* __restrict__ ids, const int* __restrict__ positions,
                                        const int* __restrict__ row_of_token, const int* __restrict__ cu_q,
                                        const int* __restrict__ state_slot, int* __restrict__ prev_token, int hidden, int vocab, float scale) {
  pdl_prologue();
  const int t = blockIdx.x;
  int id = ids[t];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const long long pr = pair_row(pt, t, ids, positions, row_of_token, cu_q, state_slot, prev_token);
  const uint4* src = reinterpret_cast<const uint4*>(table + (size_t)id * hidden);
  const uint4* pair = pr < 0 ? nullptr : reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(pt.table) + (size_t)pr * hidden);
  float4* dst = reinterpret_cast<float4*>(residual + (size_t)t * hidden);
  const float pos = (float)positions[t];
  for (int c = threadIdx.x; c < hidden >> 3; c += blockDim.x) {
    float v[8];
    bf16x8_to_float(src[c], v);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] *= scale;
    if (pair) {
      float p[8];
      bf16x8_to_float(pair[c], p);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] += p[e];
    }
    if (inv_freq) {
      const float4 f = reinterpret_cast<const float4*>(inv_freq)[c];
      const float fr[4] = {f.x, f.y, f.z, f.w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float sn, cs;
        sincosf(pos * fr[e], &sn, &cs);
        v[2 * e] += sn;
        v[2 * e + 1] += cs;
      }
    }
    dst[2 * c] = make_float4(v[0], v[1], v[2], v[3]);
    dst[2 * c + 1] = make_float4(v[4], v[5], v[6], v[7]);
  }
}

// One norm's weight: a vector, or one number (stride 0).
struct NormWeight {
  const float* w;  // null: no norm
  int stride;
  float eps;
};

// h = residual[r] + norm_b(delta[r]) (or + delta[r] where norm_b has no weight; or residual[r] without delta), written back to
// residual[r] without a gather; out[i] = norm(h). r = rows ? rows[i] : i. One CTA per row.
template <typename T, int THREADS>
__global__ void __launch_bounds__(THREADS)
add_normed_rmsnorm_kernel(T* __restrict__ out, float* __restrict__ residual, const T* __restrict__ delta, NormWeight nb, NormWeight n,
                          const int* __restrict__ rows, int hidden, int write_residual) {
  extern __shared__ float row_h[];  // hidden floats
  __shared__ float red[32];
  pdl_prologue();
  const int i = blockIdx.x;
  const int r = rows ? rows[i] : i;
  float* res = residual + (size_t)r * hidden;
  const T* dl = delta ? delta + (size_t)r * hidden : nullptr;
  float inv_b = 1.f;
  if (dl && nb.w) {
    float ss = 0.f;
    for (int c = threadIdx.x; c < hidden; c += THREADS) {
      const float d = Elem<T>::load(dl + c);
      ss += d * d;
    }
    inv_b = 1.0f / sqrtf(block_sum(ss, red) / (float)hidden + nb.eps);
  }
  float ss = 0.f;
  for (int c = threadIdx.x; c < hidden; c += THREADS) {
    float h = res[c];
    if (dl) {
      const float d = Elem<T>::load(dl + c);
      h += nb.w ? (d * inv_b) * nb.w[c * nb.stride] : d;
    }
    row_h[c] = h;
    ss += h * h;
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)hidden + n.eps);
  for (int c = threadIdx.x; c < hidden; c += THREADS) {
    const float h = row_h[c];
    if (write_residual && dl) res[c] = h;
    Elem<T>::store(out + (size_t)i * hidden + c, (h * inv) * n.w[c * n.stride]);
  }
}

__device__ __forceinline__ void weights8(const NormWeight& n, int c, float (&w)[8]) {
  if (n.stride == 0) {
    const float g = n.w[0];
#pragma unroll
    for (int e = 0; e < 8; ++e) w[e] = g;
  } else {
    const float4 a = *reinterpret_cast<const float4*>(n.w + c), b = *reinterpret_cast<const float4*>(n.w + c + 4);
    w[0] = a.x; w[1] = a.y; w[2] = a.z; w[3] = a.w; w[4] = b.x; w[5] = b.y; w[6] = b.z; w[7] = b.w;
  }
}

// bfloat16 rows that are a multiple of 8 wide and at most 8 * THREADS: eight elements per thread, kept in registers
template <int THREADS>
__global__ void __launch_bounds__(THREADS)
add_normed_rmsnorm_bf16x8_kernel(__nv_bfloat16* __restrict__ out, float* __restrict__ residual, const __nv_bfloat16* __restrict__ delta,
                                 NormWeight nb, NormWeight n, const int* __restrict__ rows, int hidden, int write_residual) {
  __shared__ float red[32];
  pdl_prologue();
  const int i = blockIdx.x;
  const int r = rows ? rows[i] : i;
  float* res = residual + (size_t)r * hidden;
  const int c = threadIdx.x * 8;
  const bool mine = c < hidden;
  float h[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f}, d[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
  if (mine) {
    const float4 a = *reinterpret_cast<const float4*>(res + c), b4 = *reinterpret_cast<const float4*>(res + c + 4);
    h[0] = a.x; h[1] = a.y; h[2] = a.z; h[3] = a.w; h[4] = b4.x; h[5] = b4.y; h[6] = b4.z; h[7] = b4.w;
    if (delta) bf16x8_to_float(*reinterpret_cast<const uint4*>(delta + (size_t)r * hidden + c), d);
  }
  if (delta) {
    if (nb.w) {
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += d[e] * d[e];
      const float inv_b = 1.0f / sqrtf(block_sum(ss, red) / (float)hidden + nb.eps);
      if (mine) {
        float w[8];
        weights8(nb, c, w);
#pragma unroll
        for (int e = 0; e < 8; ++e) h[e] += (d[e] * inv_b) * w[e];
      }
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) h[e] += d[e];
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int e = 0; e < 8; ++e) ss += h[e] * h[e];
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)hidden + n.eps);
  if (!mine) return;
  if (write_residual && delta) {
    *reinterpret_cast<float4*>(res + c) = make_float4(h[0], h[1], h[2], h[3]);
    *reinterpret_cast<float4*>(res + c + 4) = make_float4(h[4], h[5], h[6], h[7]);
  }
  float w[8], y[8];
  weights8(n, c, w);
#pragma unroll
  for (int e = 0; e < 8; ++e) y[e] = (h[e] * inv) * w[e];
  *reinterpret_cast<uint4*>(out + (size_t)i * hidden + c) = float_to_bf16x8(y);
}

// ---------------------------------------------------------------- several residual streams
// What a sublayer's output does to the streams: mix [S, S] (from, to) and out [S], float32 (null: nothing, the streams stay); and what
// the next sublayer reads: into [S] (null: the sum of the streams).
struct StreamLinks {
  const float* mix;
  const float* out;
  const float* into;
};

constexpr int HC_MAX_STREAMS = 16;

// src [T, src_streams, hidden] (one stream: all streams are equal to it), dst [T, S, hidden] (may be src). With y: the new streams go to
// dst unless rows are gathered. out[i] = rmsnorm(sum_s into[s] x_s) * w over the new streams. One CTA per row.
template <typename T, int THREADS>
__global__ void __launch_bounds__(THREADS)
stream_norm_kernel(T* __restrict__ out, float* dst, const float* src, int src_streams, int S, const T* __restrict__ y, StreamLinks links,
                   const float* __restrict__ w, float eps, const int* __restrict__ rows, int hidden, int write) {
  extern __shared__ float row_u[];  // hidden floats
  __shared__ float red[32];
  pdl_prologue();
  const int i = blockIdx.x;
  const int r = rows ? rows[i] : i;
  const float* xs = src + (size_t)r * src_streams * hidden;
  float* xd = dst + (size_t)r * S * hidden;
  float ss = 0.f;
  for (int c = threadIdx.x; c < hidden; c += THREADS) {
    float x[HC_MAX_STREAMS];
    for (int s = 0; s < S; ++s) x[s] = xs[(size_t)(src_streams == 1 ? 0 : s) * hidden + c];
    float u = 0.f;
    if (y) {
      const float d = Elem<T>::load(y + (size_t)r * hidden + c);
      for (int t = 0; t < S; ++t) {
        float n = links.out[t] * d;
        for (int s = 0; s < S; ++s) n = fmaf(links.mix[s * S + t], x[s], n);
        if (write) xd[(size_t)t * hidden + c] = n;
        u = fmaf(links.into ? links.into[t] : 1.f, n, u);
      }
    } else {
      for (int s = 0; s < S; ++s) u = fmaf(links.into ? links.into[s] : 1.f, x[s], u);
    }
    row_u[c] = u;
    ss += u * u;
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)hidden + eps);
  for (int c = threadIdx.x; c < hidden; c += THREADS) Elem<T>::store(out + (size_t)i * hidden + c, (row_u[c] * inv) * w[c]);
}

// bfloat16 rows that are a multiple of 8 wide and at most 8 * THREADS, up to four streams: eight elements of every stream per thread, in
// registers from the read to the norm
template <int THREADS, int S>
__global__ void __launch_bounds__(THREADS)
stream_norm_bf16x8_kernel(__nv_bfloat16* __restrict__ out, float* dst, const float* src, int src_streams, const __nv_bfloat16* __restrict__ y,
                          StreamLinks links, const float* __restrict__ w, float eps, const int* __restrict__ rows, int hidden, int write) {
  __shared__ float red[32];
  // (weights: none of an earlier kernel's output)
  float mix[S][S], into[S], outw[S];
#pragma unroll
  for (int s = 0; s < S; ++s) {
    into[s] = links.into ? links.into[s] : 1.f;
    outw[s] = y ? links.out[s] : 0.f;
#pragma unroll
    for (int t = 0; t < S; ++t) mix[s][t] = y ? links.mix[s * S + t] : 0.f;
  }
  pdl_prologue();
  const int i = blockIdx.x;
  const int r = rows ? rows[i] : i;
  const int c = threadIdx.x * 8;
  const bool mine = c < hidden;
  float x[S][8], u[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
  if (mine) {
    const float* xs = src + (size_t)r * src_streams * hidden + c;
    float d[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int s = 0; s < S; ++s) {
      if (s > 0 && src_streams == 1) {
#pragma unroll
        for (int e = 0; e < 8; ++e) x[s][e] = x[0][e];
      } else {
        const float4 a = *reinterpret_cast<const float4*>(xs + (size_t)s * hidden), b = *reinterpret_cast<const float4*>(xs + (size_t)s * hidden + 4);
        x[s][0] = a.x; x[s][1] = a.y; x[s][2] = a.z; x[s][3] = a.w; x[s][4] = b.x; x[s][5] = b.y; x[s][6] = b.z; x[s][7] = b.w;
      }
    }
    if (y) {
      bf16x8_to_float(*reinterpret_cast<const uint4*>(y + (size_t)r * hidden + c), d);
      float* xd = dst + (size_t)r * S * hidden + c;
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        float n[S];
#pragma unroll
        for (int t = 0; t < S; ++t) {
          n[t] = outw[t] * d[e];
#pragma unroll
          for (int s = 0; s < S; ++s) n[t] = fmaf(mix[s][t], x[s][e], n[t]);
        }
#pragma unroll
        for (int t = 0; t < S; ++t) x[t][e] = n[t];
      }
      if (write) {
#pragma unroll
        for (int t = 0; t < S; ++t) {
          *reinterpret_cast<float4*>(xd + (size_t)t * hidden) = make_float4(x[t][0], x[t][1], x[t][2], x[t][3]);
          *reinterpret_cast<float4*>(xd + (size_t)t * hidden + 4) = make_float4(x[t][4], x[t][5], x[t][6], x[t][7]);
        }
      }
    }
#pragma unroll
    for (int s = 0; s < S; ++s)
#pragma unroll
      for (int e = 0; e < 8; ++e) u[e] = fmaf(into[s], x[s][e], u[e]);
  }
  float ss = 0.f;
#pragma unroll
  for (int e = 0; e < 8; ++e) ss += u[e] * u[e];
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)hidden + eps);
  if (!mine) return;
  const float4 wa = *reinterpret_cast<const float4*>(w + c), wb = *reinterpret_cast<const float4*>(w + c + 4);
  const float wv[8] = {wa.x, wa.y, wa.z, wa.w, wb.x, wb.y, wb.z, wb.w};
#pragma unroll
  for (int e = 0; e < 8; ++e) u[e] = (u[e] * inv) * wv[e];
  *reinterpret_cast<uint4*>(out + (size_t)i * hidden + c) = float_to_bf16x8(u);
}

}  // namespace ms

using namespace ms;

// residual [T, hidden] float32; the table's rows count times `scale`. pair_table null: no second table (the arguments about rows and slots are not read then).
MS_EXPORT int ms_embed_sum(float* residual, const void* table, const void* pair_table, long long buckets, long long mul_prev,
                           long long mul_cur, const float* inv_freq, const int* ids, const int* positions, const int* row_of_token,
                           const int* cu_q, const int* state_slot, int* prev_token, int tokens, int hidden, int vocab, float scale, int dtype,
                           cudaStream_t stream) {
  if (tokens == 0) return 0;
  MS_CHECK_ARG(hidden > 0 && vocab > 0, "embed_sum: hidden=%d vocab=%d", hidden, vocab);
  MS_CHECK_ARG(!pair_table || (buckets > 0 && mul_prev >= 0 && mul_cur >= 0 && prev_token), "embed_sum: a pair table needs buckets (%lld), factors that are not negative and a state", buckets);
  const PairTable pt{pair_table, buckets, mul_prev, mul_cur};
  if (dtype == MS_F32) {
    MS_LAUNCH(embed_sum_kernel<float>, tokens, hidden >= 1024 ? 256 : 128, 0, stream, residual, (const float*)table, pt, inv_freq, ids, positions,
              row_of_token, cu_q, state_slot, prev_token, hidden, vocab, scale);
  } else if (hidden % 8 == 0 && ((uintptr_t)table % 16 == 0) && ((uintptr_t)pair_table % 16 == 0) && ((uintptr_t)inv_freq % 16 == 0) &&
             ((uintptr_t)residual % 16 == 0)) {
    MS_LAUNCH(embed_sum_bf16x8_kernel, tokens, hidden >= 1024 ? 128 : 64, 0, stream, residual, (const __nv_bfloat16*)table, pt, inv_freq, ids,
              positions, row_of_token, cu_q, state_slot, prev_token, hidden, vocab, scale);
  } else {
    MS_LAUNCH(embed_sum_kernel<__nv_bfloat16>, tokens, hidden >= 1024 ? 256 : 128, 0, stream, residual, (const __nv_bfloat16*)table, pt,
              inv_freq, ids, positions, row_of_token, cu_q, state_slot, prev_token, hidden, vocab, scale);
  }
  return 0;
}

// w_b null: the addend is added as it is. w_n / w_b_n: elements of the weights (hidden, or 1: one number for all coordinates).
MS_EXPORT int ms_add_normed_rmsnorm(void* out, float* residual, const void* delta, const float* w_b, int w_b_n, float eps_b, const float* w,
                                    int w_n, float eps, const int* rows, int n, int hidden, int write_residual, int dtype,
                                    cudaStream_t stream) {
  if (n == 0) return 0;
  MS_CHECK_ARG(hidden > 0 && (w_n == 1 || w_n == hidden) && (!w_b || w_b_n == 1 || w_b_n == hidden),
               "add_normed_rmsnorm: a weight has one element or hidden=%d, not %d / %d", hidden, w_n, w_b_n);
  const NormWeight nb{w_b, w_b_n == 1 ? 0 : 1, eps_b}, nn{w, w_n == 1 ? 0 : 1, eps};
  if (dtype == MS_BF16 && hidden % 8 == 0 && hidden <= 8192 && (uintptr_t)out % 16 == 0 && (uintptr_t)residual % 16 == 0 &&
      (uintptr_t)delta % 16 == 0 && (w_n == 1 || (uintptr_t)w % 16 == 0) && (w_b_n == 1 || (uintptr_t)w_b % 16 == 0)) {
    __nv_bfloat16* o = (__nv_bfloat16*)out;
    const __nv_bfloat16* d = (const __nv_bfloat16*)delta;
    if (hidden <= 1024) MS_LAUNCH(add_normed_rmsnorm_bf16x8_kernel<128>, n, 128, 0, stream, o, residual, d, nb, nn, rows, hidden, write_residual);
    else if (hidden <= 2048) MS_LAUNCH(add_normed_rmsnorm_bf16x8_kernel<256>, n, 256, 0, stream, o, residual, d, nb, nn, rows, hidden, write_residual);
    else if (hidden <= 4096) MS_LAUNCH(add_normed_rmsnorm_bf16x8_kernel<512>, n, 512, 0, stream, o, residual, d, nb, nn, rows, hidden, write_residual);
    else MS_LAUNCH(add_normed_rmsnorm_bf16x8_kernel<1024>, n, 1024, 0, stream, o, residual, d, nb, nn, rows, hidden, write_residual);
    return 0;
  }
  const size_t smem = (size_t)hidden * sizeof(float);
  MS_CHECK_ARG(smem <= 48 * 1024, "add_normed_rmsnorm: rows of %d do not fit shared memory", hidden);
  if (dtype == MS_F32)
    MS_LAUNCH((add_normed_rmsnorm_kernel<float, 256>), n, 256, smem, stream, (float*)out, residual, (const float*)delta, nb, nn, rows, hidden,
              write_residual);
  else
    MS_LAUNCH((add_normed_rmsnorm_kernel<__nv_bfloat16, 256>), n, 256, smem, stream, (__nv_bfloat16*)out, residual,
              (const __nv_bfloat16*)delta, nb, nn, rows, hidden, write_residual);
  return 0;
}

// dst [T, S, hidden] float32, src [T, src_streams, hidden] (src_streams 1 or S; dst may be src where it is S). y null: the streams stay as
// they are and nothing is written to dst. rows: only those rows' norms, without writing the streams.
MS_EXPORT int ms_stream_norm(void* out, float* dst, const float* src, int src_streams, int streams, const void* y, const float* mix,
                             const float* out_w, const float* into, const float* w, float eps, const int* rows, int n, int hidden, int write,
                             int dtype, cudaStream_t stream) {
  if (n == 0) return 0;
  MS_CHECK_ARG(hidden > 0 && streams >= 1 && streams <= HC_MAX_STREAMS && (src_streams == 1 || src_streams == streams),
               "stream_norm: %d streams (%d stored) of %d; at most %d are taken", streams, src_streams, hidden, HC_MAX_STREAMS);
  MS_CHECK_ARG(!y || (mix && out_w), "stream_norm: a sublayer's output needs the weights that it enters the streams with");
  MS_CHECK_ARG(!(y && write) || (dst && (dst != src || src_streams == streams)), "stream_norm: nowhere to write %d streams", streams);
  const StreamLinks links{mix, out_w, into};
  if (dtype == MS_BF16 && hidden % 8 == 0 && hidden <= 8192 && streams <= 4 && (uintptr_t)out % 16 == 0 && (uintptr_t)src % 16 == 0 &&
      (uintptr_t)dst % 16 == 0 && (uintptr_t)y % 16 == 0 && (uintptr_t)w % 16 == 0) {
    __nv_bfloat16* o = (__nv_bfloat16*)out;
    const __nv_bfloat16* d = (const __nv_bfloat16*)y;
#define MS_STREAM_NORM(TH)                                                                                                               \
  do {                                                                                                                                   \
    if (streams == 1) MS_LAUNCH((stream_norm_bf16x8_kernel<TH, 1>), n, TH, 0, stream, o, dst, src, src_streams, d, links, w, eps, rows, hidden, write);      \
    else if (streams == 2) MS_LAUNCH((stream_norm_bf16x8_kernel<TH, 2>), n, TH, 0, stream, o, dst, src, src_streams, d, links, w, eps, rows, hidden, write); \
    else if (streams == 3) MS_LAUNCH((stream_norm_bf16x8_kernel<TH, 3>), n, TH, 0, stream, o, dst, src, src_streams, d, links, w, eps, rows, hidden, write); \
    else MS_LAUNCH((stream_norm_bf16x8_kernel<TH, 4>), n, TH, 0, stream, o, dst, src, src_streams, d, links, w, eps, rows, hidden, write); \
  } while (0)
    if (hidden <= 1024) MS_STREAM_NORM(128);
    else if (hidden <= 2048) MS_STREAM_NORM(256);
    else if (hidden <= 4096) MS_STREAM_NORM(512);
    else MS_STREAM_NORM(1024);
#undef MS_STREAM_NORM
    return 0;
  }
  const size_t smem = (size_t)hidden * sizeof(float);
  MS_CHECK_ARG(smem <= 48 * 1024, "stream_norm: rows of %d do not fit shared memory", hidden);
  if (dtype == MS_F32)
    MS_LAUNCH((stream_norm_kernel<float, 256>), n, 256, smem, stream, (float*)out, dst, src, src_streams, streams, (const float*)y, links, w, eps,
              rows, hidden, write);
  else
    MS_LAUNCH((stream_norm_kernel<__nv_bfloat16, 256>), n, 256, smem, stream, (__nv_bfloat16*)out, dst, src, src_streams, streams,
              (const __nv_bfloat16*)y, links, w, eps, rows, hidden, write);
  return 0;
}
