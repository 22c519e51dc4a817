// Recurrences whose gates are worked out per token before the walk:
//
// A matrix memory with exponential gates (mLSTM). Per head, log input gate i_t = cap tanh((.)/cap) and log forget gate
// f_t = logsigmoid(cap tanh((.)/cap)), a running maximum m_t = max(f_t + m_(t-1), i_t) from m_0 = 0, and
//   S_t = exp(f_t + m_(t-1) - m_t) S_(t-1) + exp(i_t - m_t) k_t v_t^T,  n_t likewise with k_t alone,
//   o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6).
// With m known, this is the decay rule of recurrence.cu with one decay for the head and a factor on the token's write; n is
// one more column of S whose value is 1. So three kernels surround that walk: the gates (m is a scan of the pairs
// (f, i) under (F1, M1) o (F2, M2) = (F1 + F2, max(M1 + F2, M2))), the walk (recurrence.cu, or chunk_scan.cu for prompts in
// bfloat16), and the division with the norm and the gate.
//
// A gated linear recurrence per channel (the real-gated linear recurrent unit):
//   r_t, g_t = sigmoid of two products of u_t, log a_t = -c r_t, S_t = a_t S_(t-1) + sqrt(1 - a_t^2) g_t u_t,
// read out as S_t times a GELU-gated branch. u is a short causal convolution (no activation) of a biased projection.
//
// State, gates, decays and everything else that enters a recurrence are float32.
#include <cooperative_groups.h>

#include "common.cuh"

namespace ms {

namespace cg = cooperative_groups;

__device__ __forceinline__ float softplus_of(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float sigmoid_of(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float gelu_tanh_of(float z) { return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }

// ---------------------------------------------------------------- matrix memory: gates
// raw [T, .]: columns 0..H-1 the input gate's product, H..2H-1 the forget gate's; bias [2 H]. decay, write, floor_ [T, H].
// One CTA per (row, head); a thread takes a run of the row's tokens. m_state [slots, H]: the running maximum (0 before a sequence).
template <typename T, int THREADS>
__global__ void __launch_bounds__(THREADS)
mlstm_gates_kernel(float* __restrict__ decay, float* __restrict__ write, float* __restrict__ floor_, const T* __restrict__ raw, int ld,
                   const float* __restrict__ bias, float* __restrict__ m_state, const int* __restrict__ cu_q, const int* __restrict__ q_start,
                   const int* __restrict__ state_slot, int H, float cap) {
  __shared__ float wf[THREADS / 32], wm[THREADS / 32];
  pdl_prologue();
  const int r = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int t0 = cu_q[r], len = cu_q[r + 1] - t0;
  if (len <= 0) return;
  const float bi = bias[h], bf = bias[H + h], inv_cap = 1.0f / cap;
  float* slot = m_state + (size_t)state_slot[r] * H + h;
  const float m0 = q_start[r] == 0 ? 0.f : *slot;
  const int per = (len + THREADS - 1) / THREADS;
  const int a = min(len, tid * per), b = min(len, a + per);
  auto gates = [&](int t, float& i, float& f) {
    const T* p = raw + (size_t)(t0 + t) * ld;
    i = cap * tanhf((Elem<T>::load(p + h) + bi) * inv_cap);
    f = -softplus_of(-cap * tanhf((Elem<T>::load(p + H + h) + bf) * inv_cap));
  };
  float F = 0.f, M = -INFINITY;
  for (int t = a; t < b; ++t) {
    float i, f;
    gates(t, i, f);
    F += f;
    M = fmaxf(M + f, i);
  }
  // inclusive scan over the threads, then the exclusive prefix of this one
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float pf = __shfl_up_sync(0xffffffffu, F, o), pm = __shfl_up_sync(0xffffffffu, M, o);
    if (lane >= o) {
      M = fmaxf(pm + F, M);
      F += pf;
    }
  }
  if (lane == 31) {
    wf[warp] = F;
    wm[warp] = M;
  }
  __syncthreads();  // (also: every thread has read the slot)
  float ef = __shfl_up_sync(0xffffffffu, F, 1), em = __shfl_up_sync(0xffffffffu, M, 1);
  if (lane == 0) {
    ef = 0.f;
    em = -INFINITY;
  }
  float pf = 0.f, pm = -INFINITY;
  for (int w = 0; w < warp; ++w) {
    pm = fmaxf(pm + wf[w], wm[w]);
    pf += wf[w];
  }
  em = fmaxf(pm + ef, em);
  ef += pf;
  float m = fmaxf(m0 + ef, em);
  for (int t = a; t < b; ++t) {
    float i, f;
    gates(t, i, f);
    const float next = fmaxf(f + m, i);
    const size_t at = (size_t)(t0 + t) * H + h;
    decay[at] = expf(f + m - next);
    write[at] = expf(i - next);
    floor_[at] = expf(-next);
    m = next;
  }
  if (b == len && a < b) *slot = m;
}

// out[t, h * dv + c] = (o[t, h, c] / (max(|o[t, h, dv]|, floor[t, h]) + den_eps)), divided by its root mean square over c, times
// w[h * dv + c], times sigmoid(gate[t, h * dv + c]). o [T, H, ld_o] float32, its first dv + 1 columns. One warp per (token, head).
template <typename T>
__global__ void mlstm_output_kernel(T* __restrict__ out, int ld_out, const float* __restrict__ o, int ld_o, const float* __restrict__ floor_,
                                    const float* __restrict__ w, const T* __restrict__ gate, int ld_gate, long long items, int H, int dv,
                                    float eps, float den_eps) {
  pdl_prologue();
  const int lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (item >= items) return;
  const long long t = item / H;
  const int h = (int)(item - t * H);
  const float* src = o + item * ld_o;
  const float inv_den = 1.0f / (fmaxf(fabsf(src[dv]), floor_[item]) + den_eps);
  float ss = 0.f;
  for (int c = lane; c < dv; c += 32) {
    const float x = src[c] * inv_den;
    ss += x * x;
  }
  ss = warp_sum(ss);
  const float inv = 1.0f / sqrtf(ss / (float)dv + eps);
  for (int c = lane; c < dv; c += 32) {
    const float g = Elem<T>::load(gate + t * ld_gate + (size_t)h * dv + c);
    Elem<T>::store(out + t * ld_out + (size_t)h * dv + c, (((src[c] * inv_den) * inv) * w[(size_t)h * dv + c]) * sigmoid_of(g));
  }
}

// The same for bfloat16 rows on 16 bytes and value sizes that are multiples of 8: eight channels per lane and trip.
__global__ void mlstm_output_bf16x8_kernel(__nv_bfloat16* __restrict__ out, int ld_out, const float* __restrict__ o, int ld_o,
                                           const float* __restrict__ floor_, const float* __restrict__ w, const __nv_bfloat16* __restrict__ gate,
                                           int ld_gate, long long items, int H, int dv, float eps, float den_eps) {
  pdl_prologue();
  const int lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (item >= items) return;
  const long long t = item / H;
  const int h = (int)(item - t * H);
  const float* src = o + item * ld_o;
  const float inv_den = 1.0f / (fmaxf(fabsf(src[dv]), floor_[item]) + den_eps);
  float ss = 0.f;
  for (int c = lane * 8; c < dv; c += 256) {
    const float4 a = *reinterpret_cast<const float4*>(src + c), b = *reinterpret_cast<const float4*>(src + c + 4);
    const float x[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
#pragma unroll
    for (int e = 0; e < 8; ++e) ss += (x[e] * inv_den) * (x[e] * inv_den);
  }
  ss = warp_sum(ss);
  const float inv = 1.0f / sqrtf(ss / (float)dv + eps);
  for (int c = lane * 8; c < dv; c += 256) {
    const float4 a = *reinterpret_cast<const float4*>(src + c), b = *reinterpret_cast<const float4*>(src + c + 4);
    const float4 wa = *reinterpret_cast<const float4*>(w + (size_t)h * dv + c), wb = *reinterpret_cast<const float4*>(w + (size_t)h * dv + c + 4);
    const float x[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w}, wv[8] = {wa.x, wa.y, wa.z, wa.w, wb.x, wb.y, wb.z, wb.w};
    float g[8], r[8];
    bf16x8_to_float(*reinterpret_cast<const uint4*>(gate + t * ld_gate + (size_t)h * dv + c), g);
    // (fast exponential and division: relative error about 1e-6, far below the bfloat16 rounding of the result)
#pragma unroll
    for (int e = 0; e < 8; ++e) r[e] = (((x[e] * inv_den) * inv) * wv[e]) * __fdividef(1.0f, 1.0f + __expf(-g[e]));
    *reinterpret_cast<uint4*>(out + t * ld_out + (size_t)h * dv + c) = float_to_bf16x8(r);
  }
}

// ---------------------------------------------------------------- a short causal convolution of a biased projection, no activation
// u[t, c] = bias[c] + sum_j w[j, c] x'(t - (taps - 1) + j), x'(s) = x[s, c] + in_bias[c] at positions from 0 on and 0 before the
// start. w [taps, C] (tap-major). Inputs before a portion's first token come from the request's slot (the raw x, without in_bias).
// `single`: every row of the step brings one token; then the thread that read the slot's column also moves it up and appends
// the token's x (otherwise conv_state_update_kernel does that). V channels per thread.
template <typename T, int V>
__global__ void conv_bias_kernel(T* __restrict__ u, const T* __restrict__ x, int ld, T* __restrict__ conv_state, const float* __restrict__ w,
                                 const float* __restrict__ bias, const float* __restrict__ in_bias, const int* __restrict__ row_of_token,
                                 const int* __restrict__ cu_q, const int* __restrict__ q_start, const int* __restrict__ state_slot,
                                 long long items, int C, int taps, int single) {
  pdl_prologue();
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= items) return;
  const int groups = C / V;
  const int t = (int)(idx / groups), c = (int)(idx - (long long)t * groups) * V;
  const int row = row_of_token[t];
  const int local = t - cu_q[row], start = q_start[row];
  T* st = conv_state + (size_t)state_slot[row] * (taps - 1) * C + c;
  auto load = [&](const T* p, float (&f)[V]) {
    if constexpr (V == 8) bf16x8_to_float(*reinterpret_cast<const uint4*>(p), f);
    else f[0] = Elem<T>::load(p);
  };
  float acc[V], ib[V];
#pragma unroll
  for (int e = 0; e < V; ++e) {
    acc[e] = bias[c + e];
    ib[e] = in_bias[c + e];
  }
  for (int j = 0; j < taps; ++j) {
    const int at = local - (taps - 1) + j;  // place within the portion; negative: from the slot
    if (start + at < 0) continue;           // before the sequence's start
    float f[V];
    load(at >= 0 ? x + (size_t)(t - local + at) * ld + c : st + (size_t)(taps - 1 + at) * C, f);
#pragma unroll
    for (int e = 0; e < V; ++e) acc[e] = fmaf(w[(size_t)j * C + c + e], f[e] + ib[e], acc[e]);
  }
  if constexpr (V == 8) *reinterpret_cast<uint4*>(u + (size_t)t * C + c) = float_to_bf16x8(acc);
  else Elem<T>::store(u + (size_t)t * C + c, acc[0]);
  if (single) {
    for (int s = 0; s < taps - 1; ++s) {
      const bool last = s == taps - 2;
#pragma unroll
      for (int e = 0; e < V; ++e) st[(size_t)s * C + e] = last ? x[(size_t)t * ld + c + e] : st[(size_t)(s + 1) * C + e];
    }
  }
}

// The same for prompts in bfloat16 with TAPS taps: a thread takes eight channels over a run of CONV_RUN consecutive tokens of the step,
// its taps in registers and the last inputs in a window that moves along (and starts anew where a row does).
constexpr int CONV_RUN = 8;
template <int TAPS>
__global__ void conv_bias_run_kernel(__nv_bfloat16* __restrict__ u, const __nv_bfloat16* __restrict__ x, int ld,
                                     const __nv_bfloat16* __restrict__ conv_state, const float* __restrict__ w, const float* __restrict__ bias,
                                     const float* __restrict__ in_bias, const int* __restrict__ row_of_token, const int* __restrict__ cu_q,
                                     const int* __restrict__ q_start, const int* __restrict__ state_slot, int tokens, int C) {
  pdl_prologue();
  const int groups = C >> 3;
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  const int run = (int)(idx / groups), c = (int)(idx - (long long)run * groups) * 8;
  const int t0 = run * CONV_RUN, t1 = min(tokens, t0 + CONV_RUN);
  if (t0 >= tokens) return;
  float wt[TAPS][8], bs[8], ib[8];
#pragma unroll
  for (int e = 0; e < 8; e += 4) {
    *reinterpret_cast<float4*>(bs + e) = *reinterpret_cast<const float4*>(bias + c + e);
    *reinterpret_cast<float4*>(ib + e) = *reinterpret_cast<const float4*>(in_bias + c + e);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) *reinterpret_cast<float4*>(wt[j] + e) = *reinterpret_cast<const float4*>(w + (size_t)j * C + c + e);
  }
  uint4 raw[CONV_RUN];  // the run's own inputs, all in flight at once
#pragma unroll
  for (int s = 0; s < CONV_RUN; ++s) raw[s] = *reinterpret_cast<const uint4*>(x + (size_t)min(t0 + s, t1 - 1) * ld + c);
  float win[TAPS - 1][8];
  int row = -1, end = t0;
#pragma unroll
  for (int s = 0; s < CONV_RUN; ++s) {
    const int t = t0 + s;
    if (t >= t1) break;
    if (t >= end) {  // the first token of the run, or of a row: what lies before it comes from the step, the slot, or is nothing
      row = row_of_token[t];
      const int first = cu_q[row], start = q_start[row];
      end = cu_q[row + 1];
      const __nv_bfloat16* st = conv_state + (size_t)state_slot[row] * (TAPS - 1) * C + c;
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) {
        const int at = t - first - (TAPS - 1) + j;
        float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        if (start + at >= 0) {
          bf16x8_to_float(*reinterpret_cast<const uint4*>(at >= 0 ? x + (size_t)(first + at) * ld + c : st + (size_t)(TAPS - 1 + at) * C), f);
#pragma unroll
          for (int e = 0; e < 8; ++e) f[e] += ib[e];
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) win[j][e] = f[e];
      }
    }
    float now[8], acc[8];
    bf16x8_to_float(raw[s], now);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      now[e] += ib[e];
      acc[e] = bs[e];
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) acc[e] = fmaf(wt[j][e], win[j][e], acc[e]);
      acc[e] = fmaf(wt[TAPS - 1][e], now[e], acc[e]);
#pragma unroll
      for (int j = 0; j < TAPS - 2; ++j) win[j][e] = win[j + 1][e];
      win[TAPS - 2][e] = now[e];
    }
    *reinterpret_cast<uint4*>(u + (size_t)t * C + c) = float_to_bf16x8(acc);
  }
}

// ---------------------------------------------------------------- the gated linear recurrence
// One token's decay and write from the two gates' products (biases not yet added). With e = exp(log a) - 1: a = 1 + e and
// 1 - a^2 = -e (2 + e), exact where a is near one. FAST: the gates' exponential and division with relative errors of about 1e-6.
template <bool FAST>
__device__ __forceinline__ float gate_of(float x) {
  return FAST ? __fdividef(1.0f, 1.0f + __expf(-x)) : sigmoid_of(x);
}
template <bool FAST>
__device__ __forceinline__ void rglru_coefs(float zr, float zi, float u, float coef, float& a, float& b) {
  const float e = expm1f(-coef * gate_of<FAST>(zr));
  a = 1.f + e;
  b = sqrtf(-e * (2.f + e)) * (gate_of<FAST>(zi) * u);
}
// gelu_tanh(z) = z sigmoid(2 sqrt(2/pi) (z + 0.044715 z^3)), since (1 + tanh x) / 2 = sigmoid(2 x)
template <bool FAST>
__device__ __forceinline__ float gelu_gate(float z) {
  return FAST ? z * gate_of<true>(1.5957691216057308f * (z + 0.044715f * z * z * z)) : gelu_tanh_of(z);
}

// z [T, blocks, 2, bs] float32: the recurrence gate's and the input gate's products of each part; u [T, C]; y [T, .] the gated
// branch's product (y_bias added here). CTA: 32 channels (a lane each), LRU_WARPS warps, each with a run of LRU_RUN tokens; a
// cluster of `ctas` CTAs takes consecutive runs of the row, so a pass covers ctas * LRU_WARPS * LRU_RUN tokens. Within a pass: every
// warp composes its run's (a, b) pairs, the pairs of warps and CTAs are composed in order, then every warp walks its run from
// the state it found. state [slots, C] float32.
constexpr int LRU_WARPS = 16, LRU_RUN = 8, LRU_MAX_CTAS = 8;

template <typename T>
__global__ void __launch_bounds__(LRU_WARPS * 32)
rglru_scan_kernel(T* __restrict__ out, float* __restrict__ state, const float* __restrict__ z, const T* __restrict__ u,
                  const T* __restrict__ y, int ld_y, const float* __restrict__ bias_r, const float* __restrict__ bias_i,
                  const float* __restrict__ coef, const float* __restrict__ y_bias, const int* __restrict__ cu_q,
                  const int* __restrict__ q_start, const int* __restrict__ state_slot, int C, int bs, int ctas) {
  constexpr bool FAST = sizeof(T) == 2;
  __shared__ float wa[LRU_WARPS][32], wb[LRU_WARPS][32];
  __shared__ float ta[2][32], tb[2][32];  // this CTA's composed pair of the pass, in two buffers in turn
  pdl_prologue();
  cg::cluster_group cluster = cg::this_cluster();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int rank = blockIdx.x % ctas, c = (blockIdx.x / ctas) * 32 + lane, r = blockIdx.y;
  const bool active = c < C;
  const int cc = active ? c : 0;
  const int t0 = cu_q[r], len = cu_q[r + 1] - t0;
  const float br = bias_r[cc], bi = bias_i[cc], cf = coef[cc], yb = y_bias[cc];
  const int blk = cc / bs, in_blk = cc - blk * bs;
  const size_t z_row = 2 * (size_t)C, z_at = (size_t)blk * 2 * bs + in_blk;
  float* slot = state + (size_t)state_slot[r] * C + cc;
  float carry = q_start[r] == 0 ? 0.f : *slot;
  const int pass = ctas * LRU_WARPS * LRU_RUN;
  int buf = 0;
  for (int p0 = 0; p0 < len; p0 += pass, buf ^= 1) {
    const int first = p0 + (rank * LRU_WARPS + warp) * LRU_RUN;
    const int n = max(0, min(LRU_RUN, len - first));
    float a[LRU_RUN], b[LRU_RUN], yv[LRU_RUN];
    {
      float zr[LRU_RUN], zi[LRU_RUN], uv[LRU_RUN];
#pragma unroll
      for (int s = 0; s < LRU_RUN; ++s) {  // the run's loads in flight together (tokens beyond the row read its last one)
        const size_t t = (size_t)(t0 + min(first + s, len - 1));
        const float* zt = z + t * z_row + z_at;
        zr[s] = zt[0];
        zi[s] = zt[bs];
        uv[s] = Elem<T>::load(u + t * C + cc);
        yv[s] = Elem<T>::load(y + t * ld_y + cc);
      }
#pragma unroll
      for (int s = 0; s < LRU_RUN; ++s) {
        rglru_coefs<FAST>(zr[s] + br, zi[s] + bi, uv[s], cf, a[s], b[s]);
        if (s >= n) {
          a[s] = 1.f;
          b[s] = 0.f;
        }
      }
    }
    float A = 1.f, B = 0.f;
#pragma unroll
    for (int s = 0; s < LRU_RUN; ++s) {
      B = fmaf(a[s], B, b[s]);
      A *= a[s];
    }
    wa[warp][lane] = A;
    wb[warp][lane] = B;
    __syncthreads();
    // what comes before this warp inside the CTA, and the CTA's own pair
    float pa = 1.f, pb = 0.f, qa = 1.f, qb = 0.f;
#pragma unroll
    for (int w = 0; w < LRU_WARPS; ++w) {
      const float xa = wa[w][lane], xb = wb[w][lane];
      qb = fmaf(xa, qb, xb);
      qa *= xa;
      if (w < warp) {
        pa = qa;
        pb = qb;
      }
    }
    if (ctas > 1) {
      if (warp == 0) {
        ta[buf][lane] = qa;
        tb[buf][lane] = qb;
      }
      cluster.sync();  // (a buffer is written again two passes on, behind a barrier that every CTA reaches after its reads)
      float xa[LRU_MAX_CTAS], xb[LRU_MAX_CTAS];
#pragma unroll
      for (int k = 0; k < LRU_MAX_CTAS; ++k) {
        xa[k] = k < ctas ? cluster.map_shared_rank(&ta[buf][0], k)[lane] : 1.f;
        xb[k] = k < ctas ? cluster.map_shared_rank(&tb[buf][0], k)[lane] : 0.f;
      }
      float before = carry;
#pragma unroll
      for (int k = 0; k < LRU_MAX_CTAS; ++k) {
        if (k == rank) before = carry;
        carry = fmaf(xa[k], carry, xb[k]);
      }
      pb = fmaf(pa, before, pb);
    } else {
      pb = fmaf(pa, carry, pb);
      carry = fmaf(qa, carry, qb);
      __syncthreads();  // wa and wb are written again in the next pass
    }
    float S = pb;
#pragma unroll
    for (int s = 0; s < LRU_RUN; ++s) {
      S = fmaf(a[s], S, b[s]);
      if (s < n && active) Elem<T>::store(out + (size_t)(t0 + first + s) * C + c, S * gelu_gate<FAST>(yv[s] + yb));
    }
  }
  if (ctas > 1) cluster.sync();  // no CTA leaves while another may still read its shared memory
  if (rank == 0 && warp == 0 && active && len > 0) *slot = carry;
}

// One token per row (decode steps): one thread per (row, channel).
template <typename T>
__global__ void rglru_step_kernel(T* __restrict__ out, float* __restrict__ state, const float* __restrict__ z, const T* __restrict__ u,
                                  const T* __restrict__ y, int ld_y, const float* __restrict__ bias_r, const float* __restrict__ bias_i,
                                  const float* __restrict__ coef, const float* __restrict__ y_bias, const int* __restrict__ q_start,
                                  const int* __restrict__ state_slot, long long items, int C, int bs) {
  pdl_prologue();
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= items) return;
  const int r = (int)(idx / C), c = (int)(idx - (long long)r * C);
  const int blk = c / bs;
  const float* zt = z + (size_t)r * 2 * C + (size_t)blk * 2 * bs + (c - blk * bs);
  float a, b;
  constexpr bool FAST = sizeof(T) == 2;
  rglru_coefs<FAST>(zt[0] + bias_r[c], zt[bs] + bias_i[c], Elem<T>::load(u + idx), coef[c], a, b);
  float* slot = state + (size_t)state_slot[r] * C + c;
  const float S = fmaf(a, q_start[r] == 0 ? 0.f : *slot, b);
  *slot = S;
  Elem<T>::store(out + idx, S * gelu_gate<FAST>(Elem<T>::load(y + (size_t)r * ld_y + c) + y_bias[c]));
}

}  // namespace ms

using namespace ms;

MS_EXPORT int ms_mlstm_gates(float* decay, float* write, float* floor_, const void* raw, int ld, const float* bias, float* m_state,
                             const int* cu_q, const int* q_start, const int* state_slot, int num_rows, int tokens, int H, float cap, int single,
                             int dtype, cudaStream_t stream) {
  if (num_rows == 0) return 0;
  MS_CHECK_ARG(H > 0 && H <= 65535 && cap > 0.f, "mlstm_gates: %d heads, cap %g", H, (double)cap);
  const dim3 grid(num_rows, H);
#define MS_GATES(T, N) MS_LAUNCH((mlstm_gates_kernel<T, N>), grid, N, 0, stream, decay, write, floor_, (const T*)raw, ld, bias, m_state, cu_q, q_start, state_slot, H, cap)
  if (dtype == MS_F32) {
    if (single) MS_GATES(float, 32);
    else if (tokens < 512) MS_GATES(float, 256);
    else MS_GATES(float, 1024);
  } else {
    if (single) MS_GATES(__nv_bfloat16, 32);
    else if (tokens < 512) MS_GATES(__nv_bfloat16, 256);
    else MS_GATES(__nv_bfloat16, 1024);
  }
#undef MS_GATES
  return 0;
}

MS_EXPORT int ms_mlstm_output(void* out, int ld_out, const float* o, int ld_o, const float* floor_, const float* w, const void* gate, int ld_gate,
                              int tokens, int H, int dv, float eps, float den_eps, int dtype, cudaStream_t stream) {
  if (tokens == 0) return 0;
  const long long items = (long long)tokens * H;
  const unsigned blocks = (unsigned)((items + 7) / 8);
  if (dtype == MS_F32)
    MS_LAUNCH(mlstm_output_kernel<float>, blocks, 256, 0, stream, (float*)out, ld_out, o, ld_o, floor_, w, (const float*)gate, ld_gate, items, H, dv,
              eps, den_eps);
  else if (dv % 8 == 0 && ld_o % 4 == 0 && ld_out % 8 == 0 && ld_gate % 8 == 0 && (uintptr_t)out % 16 == 0 && (uintptr_t)o % 16 == 0 &&
           (uintptr_t)gate % 16 == 0 && (uintptr_t)w % 16 == 0)
    MS_LAUNCH(mlstm_output_bf16x8_kernel, blocks, 256, 0, stream, (__nv_bfloat16*)out, ld_out, o, ld_o, floor_, w, (const __nv_bfloat16*)gate,
              ld_gate, items, H, dv, eps, den_eps);
  else
    MS_LAUNCH(mlstm_output_kernel<__nv_bfloat16>, blocks, 256, 0, stream, (__nv_bfloat16*)out, ld_out, o, ld_o, floor_, w,
              (const __nv_bfloat16*)gate, ld_gate, items, H, dv, eps, den_eps);
  return 0;
}

MS_EXPORT int ms_conv_bias(void* u, const void* x, int ld, void* conv_state, const float* w, const float* bias, const float* in_bias,
                           const int* row_of_token, const int* cu_q, const int* q_start, const int* state_slot, int tokens, int C, int taps,
                           int single, int dtype, cudaStream_t stream) {
  if (tokens == 0) return 0;
  MS_CHECK_ARG(taps >= 1 && C >= 1, "conv_bias: %d taps over %d channels", taps, C);
  if (dtype == MS_BF16 && C % 8 == 0 && ld % 8 == 0 && (uintptr_t)u % 16 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)conv_state % 16 == 0) {
    if (!single && taps == 4 && (uintptr_t)w % 16 == 0 && (uintptr_t)bias % 16 == 0 && (uintptr_t)in_bias % 16 == 0) {
      const long long threads = (long long)ceil_div(tokens, CONV_RUN) * (C / 8);
      MS_LAUNCH(conv_bias_run_kernel<4>, (unsigned)((threads + 127) / 128), 128, 0, stream, (__nv_bfloat16*)u, (const __nv_bfloat16*)x, ld,
                (const __nv_bfloat16*)conv_state, w, bias, in_bias, row_of_token, cu_q, q_start, state_slot, tokens, C);
      return 0;
    }
    const long long items = (long long)tokens * (C / 8);
    MS_LAUNCH((conv_bias_kernel<__nv_bfloat16, 8>), (unsigned)((items + 127) / 128), 128, 0, stream, (__nv_bfloat16*)u, (const __nv_bfloat16*)x,
              ld, (__nv_bfloat16*)conv_state, w, bias, in_bias, row_of_token, cu_q, q_start, state_slot, items, C, taps, single);
    return 0;
  }
  const long long items = (long long)tokens * C;
  const unsigned blocks = (unsigned)((items + 255) / 256);
  if (dtype == MS_F32)
    MS_LAUNCH((conv_bias_kernel<float, 1>), blocks, 256, 0, stream, (float*)u, (const float*)x, ld, (float*)conv_state, w, bias, in_bias,
              row_of_token, cu_q, q_start, state_slot, items, C, taps, single);
  else
    MS_LAUNCH((conv_bias_kernel<__nv_bfloat16, 1>), blocks, 256, 0, stream, (__nv_bfloat16*)u, (const __nv_bfloat16*)x, ld,
              (__nv_bfloat16*)conv_state, w, bias, in_bias, row_of_token, cu_q, q_start, state_slot, items, C, taps, single);
  return 0;
}

MS_EXPORT int ms_rglru_scan(void* out, float* state, const float* z, const void* u, const void* y, int ld_y, const float* bias_r,
                            const float* bias_i, const float* coef, const float* y_bias, const int* cu_q, const int* q_start,
                            const int* state_slot, int num_rows, int tokens, int C, int bs, int single, int dtype, cudaStream_t stream) {
  if (num_rows == 0 || tokens == 0) return 0;
  MS_CHECK_ARG(C >= 1 && bs >= 1 && C % bs == 0, "rglru_scan: %d channels in parts of %d", C, bs);
  if (single) {
    const long long items = (long long)num_rows * C;
    const unsigned blocks = (unsigned)((items + 127) / 128);
    if (dtype == MS_F32)
      MS_LAUNCH(rglru_step_kernel<float>, blocks, 128, 0, stream, (float*)out, state, z, (const float*)u, (const float*)y, ld_y, bias_r,
                bias_i, coef, y_bias, q_start, state_slot, items, C, bs);
    else
      MS_LAUNCH(rglru_step_kernel<__nv_bfloat16>, blocks, 128, 0, stream, (__nv_bfloat16*)out, state, z, (const __nv_bfloat16*)u,
                (const __nv_bfloat16*)y, ld_y, bias_r, bias_i, coef, y_bias, q_start, state_slot, items, C, bs);
    return 0;
  }
  MS_CHECK_ARG(num_rows <= 65535, "rglru_scan: %d rows", num_rows);
  // a step of few tokens has nothing to share out between CTAs
  const int ctas = tokens >= 4 * LRU_WARPS * LRU_RUN ? LRU_MAX_CTAS : tokens >= 2 * LRU_WARPS * LRU_RUN ? 2 : 1;
  const dim3 grid((unsigned)(ctas * ceil_div(C, 32)), num_rows);
  if (dtype == MS_F32)
    MS_LAUNCH_CLUSTERED(rglru_scan_kernel<float>, grid, LRU_WARPS * 32, 0, stream, ctas, (float*)out, state, z, (const float*)u,
                        (const float*)y, ld_y, bias_r, bias_i, coef, y_bias, cu_q, q_start, state_slot, C, bs, ctas);
  else
    MS_LAUNCH_CLUSTERED(rglru_scan_kernel<__nv_bfloat16>, grid, LRU_WARPS * 32, 0, stream, ctas, (__nv_bfloat16*)out, state, z,
                        (const __nv_bfloat16*)u, (const __nv_bfloat16*)y, ld_y, bias_r, bias_i, coef, y_bias, cu_q, q_start, state_slot, C,
                        bs, ctas);
  return 0;
}
