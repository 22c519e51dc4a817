// Time mixing with a decay per key channel and token and a bonus for the token's own write (RWKV-style):
//
//   o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t,   S_t = diag(d_t) S_(t-1) + k_t v_t^T,   d_t = exp(-exp(z_t + w0))
//
// per head, S [dk, dv] kept as [dv, dk] in float32; z is the output of a low-rank product, z = W2 low. Three forms:
//   * one token per row (decode steps): one CTA per (row, head) works out z and the decays, reads and writes the state once, and
//     goes on to the head's norm and gate;
//   * prompts in bfloat16, by chunks of 64 tokens on the tensor cores (below);
//   * everything else: decays by channel_decay_kernel, then the token-by-token walk of recurrence.cu (the bonus rule).
//
// Chunks. With P(a..b)[c] the product of channel c's decays over tokens a..b (1 where a > b),
//   o_i = sum_(j < i) (sum_c r_i k_j P(j+1..i-1)) v_j + (sum_c r_i u k_i) v_i + S_before^T (r_i P(first..i-1)),
//   S_after = P(first..last) S_before + sum_j (k_j P(j+1..last)) v_j^T.
// A decay may be as small as zero, so nothing is divided by a product of decays: a chunk is cut into blocks of 16 tokens. Between
// two blocks the product splits at the later block's first token, and r (times the product from there) meets k (times the product up
// to there) in a matrix product; inside a block the 120 pairs are summed channel by channel with a running product. What goes to the
// tensor cores and is not exact in bfloat16 (r and k times products, the weights, the state) goes as two bfloat16 numbers. Launches:
//   states (what every chunk adds), carry (the states before every chunk, and the row's last one), outputs (for heads of one value tile with
//   the norm and the gate behind them).
#include "chunk_mma.cuh"

namespace ms {

__device__ __forceinline__ float channel_decay_of(float z) { return expf(-expf(z)); }

// out[t, c] = exp(-exp(z[t, c] + w0[c])), float32
template <typename T>
__global__ void channel_decay_kernel(float* __restrict__ out, const T* __restrict__ z, int ld_z, const float* __restrict__ w0, long long items,
                                     int width) {
  pdl_prologue();
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= items) return;
  const long long t = idx / width;
  const int c = (int)(idx - t * width);
  out[idx] = channel_decay_of(Elem<T>::load(z + t * ld_z + c) + w0[c]);
}

// ---------------------------------------------------------------- one token per row
constexpr int TS_THREADS = 256, TS_WARPS = TS_THREADS / 32, TS_COLS = 4;

// a 2-d operand: rows ld apart
template <typename T>
struct Rows {
  const T* p;
  int ld;
};

__device__ __forceinline__ void step_load8(const __nv_bfloat16* p, float (&f)[8]) { bf16x8_to_float(*reinterpret_cast<const uint4*>(p), f); }
__device__ __forceinline__ void step_load8(const float* p, float (&f)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}

// grid (H, rows). LPC lanes take a column's key channels, four at a time; a warp 32 / LPC columns at once, TS_COLS of them in turn with
// their loads in flight together; the first ones are asked for before the decays are worked out. out [T, H * dv] = o / sqrt(mean o^2 + eps) *
// norm_w * silu(gate).
template <typename T, int LPC>
__global__ void __launch_bounds__(TS_THREADS)
time_step_kernel(T* __restrict__ out, float* __restrict__ state, Rows<T> r, Rows<T> k, Rows<T> v, Rows<T> gate, Rows<T> low,
                 const T* __restrict__ w2, int rank, const float* __restrict__ w0, const float* __restrict__ u,
                 const float* __restrict__ norm_w, float eps, const int* __restrict__ cu_q, const int* __restrict__ q_start,
                 const int* __restrict__ state_slot, int H, int dk, int dv, int vec) {
  extern __shared__ __align__(16) float ts_smem[];
  __shared__ float red[32];
  float* rs = ts_smem;       // [dk]
  float* ks = rs + dk;       // [dk]
  float* ds = ks + dk;       // [dk]
  float* uk = ds + dk;       // [dk] bonus times key
  float* os = uk + dk;       // [dv]
  const int h = blockIdx.x, row = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  {  // weights: asked for before the wait
    const char* w = reinterpret_cast<const char*>(w2 + (size_t)h * dk * rank);
    for (size_t at = (size_t)tid * 128; at < (size_t)dk * rank * sizeof(T); at += TS_THREADS * 128) asm volatile("prefetch.global.L2 [%0];\n" ::"l"(w + at));
  }
  pdl_prologue();
  const int t = cu_q[row];
  const bool fresh = q_start[row] == 0;
  constexpr int CPW = 32 / LPC;
  const int l = lane % LPC, sub = lane / LPC;
  float* head = state + ((size_t)state_slot[row] * H + h) * (size_t)dv * dk;
  auto load = [&](float4 (&S)[TS_COLS], int j0, int i) {
#pragma unroll
    for (int s = 0; s < TS_COLS; ++s) {
      const int j = j0 + s * TS_WARPS * CPW;
      S[s] = fresh || j >= dv || i >= dk ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(head + (size_t)j * dk + i);
    }
  };
  float4 S[TS_COLS];
  load(S, warp * CPW + sub, l * 4);
  float vj[TS_COLS], gate0 = 0.f, nw0 = 0.f;
  auto load_v = [&](int j0) {
#pragma unroll
    for (int s = 0; s < TS_COLS; ++s) {
      const int j = j0 + s * TS_WARPS * CPW;
      vj[s] = j < dv ? Elem<T>::load(v.p + (size_t)t * v.ld + (size_t)h * dv + j) : 0.f;
    }
  };
  load_v(warp * CPW + sub);
  if (tid < dv) {
    gate0 = Elem<T>::load(gate.p + (size_t)t * gate.ld + (size_t)h * dv + tid);
    nw0 = norm_w[(size_t)h * dv + tid];
  }
  for (int c = tid; c < dk; c += TS_THREADS) {
    const size_t at = (size_t)h * dk + c;
    const float kk = Elem<T>::load(k.p + (size_t)t * k.ld + at);
    rs[c] = Elem<T>::load(r.p + (size_t)t * r.ld + at);
    ks[c] = kk;
    uk[c] = u[at] * kk;
  }
  // z of the head's channels: eight lanes a channel
  {
    const int zl = tid & 7;
    for (int c0 = 0; c0 < dk; c0 += TS_THREADS / 8) {
      const int c = c0 + (tid >> 3);
      float acc = 0.f;
      if (c < dk) {
        const T *w = w2 + ((size_t)h * dk + c) * rank, *lo = low.p + (size_t)t * low.ld;
        if (vec) {  // rows of whole eights that start on 16 bytes
          for (int i = zl * 8; i < rank; i += 64) {
            float a[8], b[8];
            step_load8(lo + i, a);
            step_load8(w + i, b);
#pragma unroll
            for (int e = 0; e < 8; ++e) acc = fmaf(a[e], b[e], acc);
          }
        } else {
          for (int i = zl; i < rank; i += 8) acc = fmaf(Elem<T>::load(lo + i), Elem<T>::load(w + i), acc);
        }
      }
#pragma unroll
      for (int o = 4; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
      if (zl == 0 && c < dk) ds[c] = channel_decay_of(acc + w0[(size_t)h * dk + c]);
    }
  }
  __syncthreads();
  bool loaded = true;  // the first group is
  for (int j0 = warp * CPW + sub; j0 - sub < dv; j0 += TS_WARPS * CPW * TS_COLS) {
    float acc[TS_COLS] = {};
    if (j0 != warp * CPW + sub) load_v(j0);
    for (int i = l * 4; i < dk; i += LPC * 4) {
      if (!loaded) load(S, j0, i);
      loaded = false;
      const float4 r4 = *reinterpret_cast<const float4*>(rs + i), k4 = *reinterpret_cast<const float4*>(ks + i);
      const float4 d4 = *reinterpret_cast<const float4*>(ds + i), u4 = *reinterpret_cast<const float4*>(uk + i);
#pragma unroll
      for (int s = 0; s < TS_COLS; ++s) {
        const int j = j0 + s * TS_WARPS * CPW;
        acc[s] += (r4.x * fmaf(u4.x, vj[s], S[s].x) + r4.y * fmaf(u4.y, vj[s], S[s].y)) +
                  (r4.z * fmaf(u4.z, vj[s], S[s].z) + r4.w * fmaf(u4.w, vj[s], S[s].w));
        S[s] = make_float4(fmaf(d4.x, S[s].x, k4.x * vj[s]), fmaf(d4.y, S[s].y, k4.y * vj[s]), fmaf(d4.z, S[s].z, k4.z * vj[s]),
                           fmaf(d4.w, S[s].w, k4.w * vj[s]));
        if (j < dv) *reinterpret_cast<float4*>(head + (size_t)j * dk + i) = S[s];
      }
    }
    loaded = false;  // (a lane beyond the key channels has used none)
#pragma unroll
    for (int s = 0; s < TS_COLS; ++s) {
      float x = acc[s];
#pragma unroll
      for (int o = LPC >> 1; o > 0; o >>= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
      const int j = j0 + s * TS_WARPS * CPW;
      if (l == 0 && j < dv) os[j] = x;
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < dv; c += TS_THREADS) ss += os[c] * os[c];
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)dv + eps);
  for (int c = tid; c < dv; c += TS_THREADS) {
    const size_t at = (size_t)h * dv + c;
    const float g = c == tid ? gate0 : Elem<T>::load(gate.p + (size_t)t * gate.ld + at);
    Elem<T>::store(out + (size_t)t * H * dv + at, ((os[c] * inv) * (c == tid ? nw0 : norm_w[at])) * (g / (1.0f + expf(-g))));
  }
}

// ---------------------------------------------------------------- chunks: what every chunk adds to the state
constexpr int TC_DV = 64;  // value columns per CTA
constexpr int TC_BLK = 16, TC_BLOCKS = CS_TOK / TC_BLK;

struct ChunkPlace {
  const int2* tab;       // (row, first flat token) of a chunk
  const int* row_first;  // a row's first chunk; [num_rows]: how many chunks there are
  const int* cu_q;
  const int* q_start;
  const int* state_slot;
  int num_rows;
};

// Two float32 in a register pair, one instruction for both.
__device__ __forceinline__ uint64_t pack2(float a, float b) {
  uint64_t v;
  asm("mov.b64 %0, {%1, %2};" : "=l"(v) : "f"(a), "f"(b));
  return v;
}
__device__ __forceinline__ float2 unpack2(uint64_t v) {
  float2 f;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(v));
  return f;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t v;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(v) : "l"(a), "l"(b), "l"(c));
  return v;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t v;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(v) : "l"(a), "l"(b));
  return v;
}
__device__ __forceinline__ float sum2(uint64_t v) {
  const float2 f = unpack2(v);
  return f.x + f.y;
}
__device__ __forceinline__ uint64_t widen2(__nv_bfloat162 v) {
  const float2 f = __bfloat1622float2(v);
  return pack2(f.x, f.y);
}
// Two neighbours as two bfloat16 each.
__device__ __forceinline__ void split2(uint64_t v, __nv_bfloat16* hi, __nv_bfloat16* lo) {
  const float2 x = unpack2(v);
  const __nv_bfloat162 h = __floats2bfloat162_rn(x.x, x.y);
  const float2 f = __bfloat1622float2(h);
  *reinterpret_cast<__nv_bfloat162*>(hi) = h;
  *reinterpret_cast<__nv_bfloat162*>(lo) = __floats2bfloat162_rn(x.x - f.x, x.y - f.y);
}

// A warp takes half a block (eight tokens) of 64 key channels at a time, a lane two neighbouring channels: their decays, and another operand
// or two of the same shape. FULL: a whole chunk of heads as wide as the tile; otherwise tokens from n on have a decay of one and operands
// of zero, and so have channels from dk on. (The hardware's exponential: relative error about 1e-6 of an exponent.)
constexpr int TC_HALF = 8;
template <bool FULL>
__device__ __forceinline__ void half_decays(uint64_t (&d)[TC_HALF], const float* __restrict__ z, int ld_z, const float* __restrict__ w0, int row0, int n,
                                            bool in) {
  float2 v[TC_HALF];
#pragma unroll
  for (int i = 0; i < TC_HALF; ++i)
    v[i] = FULL || (in && row0 + i < n) ? *reinterpret_cast<const float2*>(z + (size_t)(row0 + i) * ld_z) : make_float2(0.f, 0.f);
  const float2 w = FULL || in ? *reinterpret_cast<const float2*>(w0) : make_float2(0.f, 0.f);
#pragma unroll
  for (int i = 0; i < TC_HALF; ++i) {
    const float a = __expf(-__expf(v[i].x + w.x)), b = __expf(-__expf(v[i].y + w.y));
    d[i] = FULL || (in && row0 + i < n) ? pack2(a, b) : pack2(1.f, 1.f);
  }
}
template <bool FULL>
__device__ __forceinline__ void half_rows(__nv_bfloat162 (&x)[TC_HALF], const __nv_bfloat16* __restrict__ src, int ld, int row0, int n, bool in) {
#pragma unroll
  for (int i = 0; i < TC_HALF; ++i)
    x[i] = FULL || (in && row0 + i < n) ? *reinterpret_cast<const __nv_bfloat162*>(src + (size_t)(row0 + i) * ld) : __floats2bfloat162_rn(0.f, 0.f);
}

template <int DKT>
struct TmStatesSmem {
  __nv_bfloat16 v[CS_TOK][TC_DV + 8], khi[CS_TOK][DKT + 8], klo[CS_TOK][DKT + 8];
  float half[2 * TC_BLOCKS][DKT];  // the products of half blocks
};

// What the chunk's keys are multiplied by on their way into the state; this warp's share.
template <int DKT, bool FULL>
__device__ __forceinline__ void state_keys(TmStatesSmem<DKT>& sm, float* __restrict__ passed, const __nv_bfloat16* __restrict__ k, int ld_k,
                                           const float* __restrict__ z, int ld_z, const float* __restrict__ w0, int n, int dk) {
  constexpr int TRIPS = DKT / 64;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, row0 = warp * TC_HALF;
  uint64_t x[TRIPS][TC_HALF];
#pragma unroll
  for (int tr = 0; tr < TRIPS; ++tr) {
    const int c = tr * 64 + lane * 2;
    const bool in = c < dk;
    __nv_bfloat162 kk[TC_HALF];
    half_rows<FULL>(kk, k + c, ld_k, row0, n, in);
    uint64_t d[TC_HALF];
    half_decays<FULL>(d, z + c, ld_z, w0 + c, row0, n, in);
    uint64_t suf = pack2(1.f, 1.f);
#pragma unroll
    for (int i = TC_HALF - 1; i >= 0; --i) {
      x[tr][i] = mul2(widen2(kk[i]), suf);
      suf = mul2(suf, d[i]);
    }
    *reinterpret_cast<uint64_t*>(&sm.half[warp][c]) = suf;
  }
  __syncthreads();
#pragma unroll
  for (int tr = 0; tr < TRIPS; ++tr) {
    const int c = tr * 64 + lane * 2;
    uint64_t behind = pack2(1.f, 1.f);
#pragma unroll
    for (int q = 1; q < 2 * TC_BLOCKS; ++q)
      if (q > warp) behind = mul2(behind, *reinterpret_cast<const uint64_t*>(&sm.half[q][c]));
#pragma unroll
    for (int i = 0; i < TC_HALF; ++i) split2(mul2(x[tr][i], behind), &sm.khi[row0 + i][c], &sm.klo[row0 + i][c]);
    if (passed && warp == 0 && c < dk) *reinterpret_cast<uint64_t*>(passed + c) = mul2(behind, *reinterpret_cast<const uint64_t*>(&sm.half[0][c]));
  }
}

// added [chunks, H, dv, dk] float32, passed [chunks, H, dk]: the product of the chunk's decays. grid (chunks, H, dv tiles).
template <int DKT>
__global__ void __launch_bounds__(CS_THREADS)
tm_states_kernel(float* __restrict__ added, float* __restrict__ passed, const __nv_bfloat16* __restrict__ k, int ld_k,
                 const __nv_bfloat16* __restrict__ v, int ld_v, const float* __restrict__ z, int ld_z, const float* __restrict__ w0,
                 const ChunkPlace pl, int H, int dk, int dv) {
  extern __shared__ __align__(16) unsigned char cs_raw[];
  TmStatesSmem<DKT>& sm = *reinterpret_cast<TmStatesSmem<DKT>*>(cs_raw);
  pdl_prologue();
  const int chunk = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * TC_DV;
  if (chunk >= pl.row_first[pl.num_rows]) return;
  const int2 at = pl.tab[chunk];
  const int t0 = at.y, n = min(CS_TOK, pl.cu_q[at.x + 1] - t0);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  for (int idx = tid; idx < CS_TOK * (TC_DV / 8); idx += CS_THREADS) {
    const int tt = idx / (TC_DV / 8), c = (idx - tt * (TC_DV / 8)) * 8;
    const bool in = tt < n && v0 + c < dv;
    cs_cp16(&sm.v[tt][c], in ? (const void*)(v + (size_t)(t0 + tt) * ld_v + (size_t)h * dv + v0 + c) : (const void*)v, in);
  }
  cs_commit();
  {
    float* all = blockIdx.z == 0 ? passed + ((size_t)chunk * H + h) * dk : nullptr;
    const __nv_bfloat16* kh = k + (size_t)t0 * ld_k + (size_t)h * dk;
    const float* zh = z + (size_t)t0 * ld_z + (size_t)h * dk;
    if (n == CS_TOK && dk == DKT) state_keys<DKT, true>(sm, all, kh, ld_k, zh, ld_z, w0 + (size_t)h * dk, n, dk);
    else state_keys<DKT, false>(sm, all, kh, ld_k, zh, ld_z, w0 + (size_t)h * dk, n, dk);
  }
  cs_wait<0>();
  __syncthreads();
  constexpr int NC = DKT / 2;  // key columns per warp
  const int wm = (warp >> 1) * 16, wn = (warp & 1) * NC;  // 4 x 2 warps of 16 value rows x NC key columns
  float acc[NC / 8][4] = {};
  const int i8 = lane & 7, mat = lane >> 3;
#pragma unroll
  for (int kk = 0; kk < CS_TOK; kk += 16) {
    uint32_t a[4];
    cs_ldsm_t(a, &sm.v[kk + i8 + (mat >= 2 ? 8 : 0)][wm + (mat & 1 ? 8 : 0)]);
#pragma unroll
    for (int nj = 0; nj < NC / 16; ++nj) {
      uint32_t bh[4], bl[4];
      const int row = kk + i8 + (mat & 1 ? 8 : 0), col = wn + nj * 16 + (mat >= 2 ? 8 : 0);
      cs_ldsm_t(bh, &sm.khi[row][col]);
      cs_ldsm_t(bl, &sm.klo[row][col]);
      cs_mma(acc[2 * nj], a, bh[0], bh[1]);
      cs_mma(acc[2 * nj], a, bl[0], bl[1]);
      cs_mma(acc[2 * nj + 1], a, bh[2], bh[3]);
      cs_mma(acc[2 * nj + 1], a, bl[2], bl[3]);
    }
  }
  float* out = added + ((size_t)chunk * H + h) * (size_t)dv * dk;
  const int g = lane >> 2, tg = (lane & 3) * 2;
#pragma unroll
  for (int ni = 0; ni < NC / 8; ++ni)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int row = v0 + wm + g + half * 8, col = wn + ni * 8 + tg;  // (dk is even: a pair is inside or outside)
      if (row < dv && col < dk) *reinterpret_cast<float2*>(out + (size_t)row * dk + col) = make_float2(acc[ni][2 * half], acc[ni][2 * half + 1]);
    }
}

// ---------------------------------------------------------------- chunks: the states before every chunk
// before_hi / before_lo [chunks, H, dv, dk]: the state before every chunk as two bfloat16; the row's slot of state [slots, H, dv, dk] gets
// the state behind its last chunk. One element per thread, the reads of sixteen chunks in flight; grid (elements of a row's state, rows).
__global__ void __launch_bounds__(CS_THREADS)
tm_carry_kernel(float* __restrict__ state, __nv_bfloat16* __restrict__ before_hi, __nv_bfloat16* __restrict__ before_lo,
                const float* __restrict__ added, const float* __restrict__ passed, const ChunkPlace pl, int H, int dk, int dv) {
  pdl_prologue();
  const int total = H * dv * dk;
  const int i = blockIdx.x * CS_THREADS + threadIdx.x, r = blockIdx.y;
  if (i >= total) return;
  const int h = i / (dv * dk), c = i % dk;
  const int c0 = pl.row_first[r], c1 = pl.row_first[r + 1];
  if (c1 <= c0) return;
  float* slot = state + (size_t)pl.state_slot[r] * total + i;
  float S = pl.q_start[r] == 0 ? 0.f : *slot;
  constexpr int AHEAD = 16;
  for (int ch0 = c0; ch0 < c1; ch0 += AHEAD) {
    float d[AHEAD], a[AHEAD];
#pragma unroll
    for (int q = 0; q < AHEAD; ++q) {
      if (ch0 + q < c1) {
        d[q] = added[(size_t)(ch0 + q) * total + i];
        a[q] = passed[((size_t)(ch0 + q) * H + h) * dk + c];
      }
    }
#pragma unroll
    for (int q = 0; q < AHEAD; ++q) {
      if (ch0 + q < c1) {
        const size_t at = (size_t)(ch0 + q) * total + i;
        cs_split(S, before_hi[at], before_lo[at]);
        S = fmaf(a[q], S, d[q]);
      }
    }
  }
  *slot = S;
}

// ---------------------------------------------------------------- chunks: the outputs
template <int DKT>
struct TmOutputsSmem {
  static constexpr int LDK = DKT + 8, LDP = CS_TOK + 8;
  union {
    struct {
      float d[CS_TOK][DKT + 4], r[CS_TOK][DKT + 4];  // decays, and r as it is
    };
    struct {
      __nv_bfloat16 shi[TC_DV][LDK], slo[TC_DV][LDK];  // the state before the chunk, once the pairs inside the blocks are done
    };
  };
  float half[2 * TC_BLOCKS][DKT];                   // the products of half blocks
  float dsum[2][TC_BLOCKS][TC_BLK][TC_BLK + 1];     // [channel half][block][j][i]: sums of the pairs inside a block
  float squares[2][CS_TOK];                         // [column half][token]
  __nv_bfloat16 k[CS_TOK][LDK];
  __nv_bfloat16 rhi[CS_TOK][LDK], rlo[CS_TOK][LDK];  // r times the product from its block's (then: the chunk's) first token on
  union {
    struct {
      __nv_bfloat16 hi[96][LDK], lo[96][LDK];  // k times the product up to block 1 (rows 0..15), 2 (16..47), 3 (48..95)
    } kb;
    struct {
      __nv_bfloat16 hi[CS_TOK][LDP], lo[CS_TOK][LDP];  // the weights of v
    } p;
  };
  __nv_bfloat16 v[CS_TOK][TC_DV + 8];
};

// A warp's half block: r and k with the products of decays that they meet in; pr keeps r times the product from its block's first token on.
template <int DKT, bool FULL>
__device__ __forceinline__ void output_operands(TmOutputsSmem<DKT>& sm, uint64_t (&pr)[DKT / 64][TC_HALF], const __nv_bfloat16* __restrict__ r, int ld_r,
                                                const __nv_bfloat16* __restrict__ k, int ld_k, const float* __restrict__ z, int ld_z,
                                                const float* __restrict__ w0, int n, int dk) {
  constexpr int TRIPS = DKT / 64;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, blk = warp >> 1, upper = warp & 1, row0 = warp * TC_HALF;
  uint64_t kx[TRIPS][TC_HALF];
#pragma unroll
  for (int tr = 0; tr < TRIPS; ++tr) {
    const int c = tr * 64 + lane * 2;
    const bool in = c < dk;
    __nv_bfloat162 rr[TC_HALF], kk[TC_HALF];
    half_rows<FULL>(rr, r + c, ld_r, row0, n, in);
    half_rows<FULL>(kk, k + c, ld_k, row0, n, in);
    uint64_t d[TC_HALF];
    half_decays<FULL>(d, z + c, ld_z, w0 + c, row0, n, in);
    uint64_t run = pack2(1.f, 1.f), suf = pack2(1.f, 1.f);
#pragma unroll
    for (int i = 0; i < TC_HALF; ++i) {
      const uint64_t x = widen2(rr[i]);
      *reinterpret_cast<uint64_t*>(&sm.r[row0 + i][c]) = x;
      *reinterpret_cast<uint64_t*>(&sm.d[row0 + i][c]) = d[i];
      *reinterpret_cast<__nv_bfloat162*>(&sm.k[row0 + i][c]) = kk[i];
      pr[tr][i] = mul2(run, x);  // times the product up to the token before
      run = mul2(run, d[i]);
    }
#pragma unroll
    for (int i = TC_HALF - 1; i >= 0; --i) {
      kx[tr][i] = mul2(widen2(kk[i]), suf);
      suf = mul2(suf, d[i]);
    }
    *reinterpret_cast<uint64_t*>(&sm.half[warp][c]) = run;
  }
  __syncthreads();
#pragma unroll
  for (int tr = 0; tr < TRIPS; ++tr) {
    const int c = tr * 64 + lane * 2;
    const auto half = [&](int q) { return *reinterpret_cast<const uint64_t*>(&sm.half[q][c]); };
    if (upper) {
      const uint64_t a = half(warp - 1);
#pragma unroll
      for (int i = 0; i < TC_HALF; ++i) pr[tr][i] = mul2(pr[tr][i], a);
    } else {
      const uint64_t b = half(warp + 1);
#pragma unroll
      for (int i = 0; i < TC_HALF; ++i) kx[tr][i] = mul2(kx[tr][i], b);
    }
#pragma unroll
    for (int i = 0; i < TC_HALF; ++i) split2(pr[tr][i], &sm.rhi[row0 + i][c], &sm.rlo[row0 + i][c]);
    if (blk == TC_BLOCKS - 1) continue;
    // k for the next block, and times the products of the blocks between for those behind it
    const int base = (blk == 0 ? 0 : blk == 1 ? 32 : 80) + upper * TC_HALF;
#pragma unroll
    for (int i = 0; i < TC_HALF; ++i) split2(kx[tr][i], &sm.kb.hi[base + i][c], &sm.kb.lo[base + i][c]);
    if (blk == 2) continue;
    const uint64_t w2 = mul2(half(4), half(5));
    if (blk == 0) {
      const uint64_t w1 = mul2(half(2), half(3));
#pragma unroll
      for (int i = 0; i < TC_HALF; ++i) {
        kx[tr][i] = mul2(kx[tr][i], w1);
        split2(kx[tr][i], &sm.kb.hi[16 + upper * TC_HALF + i][c], &sm.kb.lo[16 + upper * TC_HALF + i][c]);
      }
    }
    const int last = (blk == 0 ? 48 : 64) + upper * TC_HALF;
#pragma unroll
    for (int i = 0; i < TC_HALF; ++i) split2(mul2(kx[tr][i], w2), &sm.kb.hi[last + i][c], &sm.kb.lo[last + i][c]);
  }
}

// What follows the recurrence: out [T, H * dv] bfloat16 = o / sqrt(mean o^2 + eps) * norm_w * silu(gate) (heads of one value tile).
struct HeadGate {
  __nv_bfloat16* out;  // null: o is written as it is
  const __nv_bfloat16* gate;
  int ld_gate;
  const float* norm_w;
  float eps;
};

// o [T, H, dv] float32 (or hg.out). grid (chunks, H, dv tiles).
template <int DKT>
__global__ void __launch_bounds__(CS_THREADS, DKT <= 64 ? 2 : 1)
tm_outputs_kernel(float* __restrict__ o, const HeadGate hg, const __nv_bfloat16* __restrict__ r, int ld_r, const __nv_bfloat16* __restrict__ k,
                  int ld_k, const __nv_bfloat16* __restrict__ v, int ld_v, const float* __restrict__ z, int ld_z, const float* __restrict__ w0,
                  const float* __restrict__ u, const __nv_bfloat16* __restrict__ before_hi, const __nv_bfloat16* __restrict__ before_lo,
                  const ChunkPlace pl, int H, int dk, int dv) {
  extern __shared__ __align__(16) unsigned char cs_raw[];
  TmOutputsSmem<DKT>& sm = *reinterpret_cast<TmOutputsSmem<DKT>*>(cs_raw);
  pdl_prologue();
  const int chunk = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * TC_DV;
  if (chunk >= pl.row_first[pl.num_rows]) return;
  const int2 at = pl.tab[chunk];
  const int t0 = at.y, n = min(CS_TOK, pl.cu_q[at.x + 1] - t0);
  const bool has_state = !(pl.q_start[at.x] == 0 && chunk == pl.row_first[at.x]);  // else nothing came before
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int i8 = lane & 7, mat = lane >> 3, g = lane >> 2, tg = (lane & 3) * 2;
  for (int idx = tid; idx < CS_TOK * (TC_DV / 8); idx += CS_THREADS) {
    const int tt = idx / (TC_DV / 8), c = (idx - tt * (TC_DV / 8)) * 8;
    const bool in = tt < n && v0 + c < dv;
    cs_cp16(&sm.v[tt][c], in ? (const void*)(v + (size_t)(t0 + tt) * ld_v + (size_t)h * dv + v0 + c) : (const void*)v, in);
  }
  cs_commit();

  constexpr int TRIPS = DKT / 64;
  uint64_t pr[TRIPS][TC_HALF];
  {
    const __nv_bfloat16 *rh = r + (size_t)t0 * ld_r + (size_t)h * dk, *kh = k + (size_t)t0 * ld_k + (size_t)h * dk;
    const float* zh = z + (size_t)t0 * ld_z + (size_t)h * dk;
    if (n == CS_TOK && dk == DKT) output_operands<DKT, true>(sm, pr, rh, ld_r, kh, ld_k, zh, ld_z, w0 + (size_t)h * dk, n, dk);
    else output_operands<DKT, false>(sm, pr, rh, ld_r, kh, ld_k, zh, ld_z, w0 + (size_t)h * dk, n, dk);
  }
  const int bi = warp >> 1, half_w = warp & 1, wm = bi * TC_BLK;
  // pairs inside a block: a lane takes j and 15 - j (15 pairs together) over DKT / 8 channels; two warps make up a block's channels
  {
    const int j = lane & 7;
    constexpr int QC = DKT / 8;
    const int cbeg = (half_w * 4 + (lane >> 3)) * QC;
    uint64_t acc2[TC_BLK - 1] = {}, own2[2] = {};  // pairs of sums: even and odd channels
    constexpr int STRIDE = DKT + 4;
    const float* r0 = &sm.r[wm][0];
    const float* d0 = &sm.d[wm][0];
#pragma unroll 1
    for (int c = cbeg; c < cbeg + QC; c += 4) {
      uint64_t x[2], y[2];
      {
        const float4 u4 = c < dk ? *reinterpret_cast<const float4*>(u + (size_t)h * dk + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        const uint64_t u01 = pack2(u4.x, u4.y), u23 = pack2(u4.z, u4.w);
#pragma unroll
        for (int q = 0; q < 2; ++q) {
          const int jj = q == 0 ? j : 15 - j;
          const __nv_bfloat162* kp = reinterpret_cast<const __nv_bfloat162*>(&sm.k[wm + jj][c]);
          uint64_t(&w)[2] = q == 0 ? x : y;
          w[0] = widen2(kp[0]);
          w[1] = widen2(kp[1]);
          const ulonglong2 rr = *reinterpret_cast<const ulonglong2*>(r0 + jj * STRIDE + c);
          own2[q] = fma2(mul2(rr.x, u01), w[0], fma2(mul2(rr.y, u23), w[1], own2[q]));
        }
      }
#pragma unroll
      for (int s = 0; s < TC_BLK - 1; ++s) {
        // (15 - j is 8 at least: the first eight steps are j's for every lane)
        if (s >= 8 && s == 15 - j) {
          x[0] = y[0];
          x[1] = y[1];
        }
        const int at = (s < 8 || s < 15 - j ? j * STRIDE : 0) + (s + 1) * STRIDE + c;
        const ulonglong2 rr = *reinterpret_cast<const ulonglong2*>(r0 + at), dd = *reinterpret_cast<const ulonglong2*>(d0 + at);
        acc2[s] = fma2(rr.x, x[0], fma2(rr.y, x[1], acc2[s]));
        x[0] = mul2(x[0], dd.x);
        x[1] = mul2(x[1], dd.y);
      }
    }
    float acc[TC_BLK - 1], own[2];
#pragma unroll
    for (int s = 0; s < TC_BLK - 1; ++s) acc[s] = sum2(acc2[s]);
    own[0] = sum2(own2[0]);
    own[1] = sum2(own2[1]);
#pragma unroll
    for (int s = 0; s < TC_BLK - 1; ++s) {
      acc[s] += __shfl_xor_sync(0xffffffffu, acc[s], 8);
      acc[s] += __shfl_xor_sync(0xffffffffu, acc[s], 16);
    }
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      own[q] += __shfl_xor_sync(0xffffffffu, own[q], 8);
      own[q] += __shfl_xor_sync(0xffffffffu, own[q], 16);
    }
    if (lane < 8) {
#pragma unroll
      for (int s = 0; s < TC_BLK - 1; ++s) sm.dsum[half_w][bi][s < 15 - j ? j : 15 - j][s + 1 + (s < 15 - j ? j : 0)] = acc[s];
      sm.dsum[half_w][bi][j][j] = own[0];
      sm.dsum[half_w][bi][15 - j][15 - j] = own[1];
    }
  }
  __syncthreads();  // kb is whole, d and r have been read
  if (has_state) {
    const size_t st = ((size_t)chunk * H + h) * (size_t)dv * dk;
    for (int idx = tid; idx < TC_DV * (DKT / 8); idx += CS_THREADS) {
      const int row = idx / (DKT / 8), c = (idx - row * (DKT / 8)) * 8;
      const bool in = v0 + row < dv && c < dk;
      const size_t src = in ? st + (size_t)(v0 + row) * dk + c : 0;
      cs_cp16(&sm.shi[row][c], before_hi + src, in);
      cs_cp16(&sm.slo[row][c], before_lo + src, in);
    }
  }
  cs_commit();
  // pairs of blocks: weights of the tokens of block jt < bi for those of block bi
  float s[2][2][4] = {};  // [this warp's tiles: jt = half_w, half_w + 2][n8][..]
  {
    const int base = bi == 1 ? 0 : bi == 2 ? 16 : 48;
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      const int jt = half_w + 2 * q;
      if (jt >= bi) continue;
#pragma unroll
      for (int kk = 0; kk < DKT; kk += 16) {
        uint32_t ah[4], al[4], bh[4], bl[4];
        const int ra = wm + i8 + (mat & 1 ? 8 : 0), ca = kk + (mat >= 2 ? 8 : 0);
        cs_ldsm(ah, &sm.rhi[ra][ca]);
        cs_ldsm(al, &sm.rlo[ra][ca]);
        const int rb = base + jt * TC_BLK + i8 + (mat >= 2 ? 8 : 0), cb = kk + (mat & 1 ? 8 : 0);
        cs_ldsm(bh, &sm.kb.hi[rb][cb]);
        cs_ldsm(bl, &sm.kb.lo[rb][cb]);
        cs_mma(s[q][0], ah, bh[0], bh[1]);
        cs_mma(s[q][0], ah, bl[0], bl[1]);
        cs_mma(s[q][0], al, bh[0], bh[1]);
        cs_mma(s[q][1], ah, bh[2], bh[3]);
        cs_mma(s[q][1], ah, bl[2], bl[3]);
        cs_mma(s[q][1], al, bh[2], bh[3]);
      }
    }
  }
  __syncthreads();  // kb and r's products have been read
#pragma unroll
  for (int q = 0; q < 2; ++q) {
    const int jt = half_w + 2 * q;
    if (jt >= bi) continue;
#pragma unroll
    for (int nj = 0; nj < 2; ++nj)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int i = wm + g + half * 8, j = jt * TC_BLK + nj * 8 + tg;
        __align__(4) __nv_bfloat16 hi[2];
        __align__(4) __nv_bfloat16 lo[2];
        cs_split(s[q][nj][2 * half], hi[0], lo[0]);
        cs_split(s[q][nj][2 * half + 1], hi[1], lo[1]);
        *reinterpret_cast<uint32_t*>(&sm.p.hi[i][j]) = *reinterpret_cast<const uint32_t*>(hi);
        *reinterpret_cast<uint32_t*>(&sm.p.lo[i][j]) = *reinterpret_cast<const uint32_t*>(lo);
      }
  }
  for (int idx = tid; idx < TC_BLOCKS * TC_BLK * TC_BLK; idx += CS_THREADS) {
    const int b = idx >> 8, i = (idx >> 4) & 15, j = idx & 15;
    const float x = j <= i ? sm.dsum[0][b][j][i] + sm.dsum[1][b][j][i] : 0.f;
    cs_split(x, sm.p.hi[b * TC_BLK + i][b * TC_BLK + j], sm.p.lo[b * TC_BLK + i][b * TC_BLK + j]);
  }
  if (has_state && bi > 0) {  // r times the product from the chunk's first token on (block 0 has it already)
#pragma unroll
    for (int tr = 0; tr < TRIPS; ++tr) {
      const int c = tr * 64 + lane * 2;
      uint64_t ahead = pack2(1.f, 1.f);
#pragma unroll
      for (int q = 0; q < 2 * (TC_BLOCKS - 1); ++q)
        if (q < 2 * bi) ahead = mul2(ahead, *reinterpret_cast<const uint64_t*>(&sm.half[q][c]));
#pragma unroll
      for (int i = 0; i < TC_HALF; ++i) split2(mul2(pr[tr][i], ahead), &sm.rhi[warp * TC_HALF + i][c], &sm.rlo[warp * TC_HALF + i][c]);
    }
  }
  cs_wait<0>();
  __syncthreads();

  // 4 x 2 warps of 16 tokens x 32 value columns
  const int wn = half_w * 32;
  float acc[4][4] = {};
  if (has_state) {
#pragma unroll
    for (int kk = 0; kk < DKT; kk += 16) {
      uint32_t ah[4], al[4];
      const int ra = wm + i8 + (mat & 1 ? 8 : 0), ca = kk + (mat >= 2 ? 8 : 0);
      cs_ldsm(ah, &sm.rhi[ra][ca]);
      cs_ldsm(al, &sm.rlo[ra][ca]);
#pragma unroll
      for (int nj = 0; nj < 2; ++nj) {
        uint32_t bh[4], bl[4];
        const int rb = wn + nj * 16 + i8 + (mat >= 2 ? 8 : 0), cb = kk + (mat & 1 ? 8 : 0);
        cs_ldsm(bh, &sm.shi[rb][cb]);
        cs_ldsm(bl, &sm.slo[rb][cb]);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          cs_mma(acc[2 * nj + e], ah, bh[2 * e], bh[2 * e + 1]);
          cs_mma(acc[2 * nj + e], ah, bl[2 * e], bl[2 * e + 1]);
          cs_mma(acc[2 * nj + e], al, bh[2 * e], bh[2 * e + 1]);
        }
      }
    }
  }
  for (int kk = 0; kk <= wm; kk += 16) {  // (later tokens have no weight)
    uint32_t ah[4], al[4];
    const int ra = wm + i8 + (mat & 1 ? 8 : 0), ca = kk + (mat >= 2 ? 8 : 0);
    cs_ldsm(ah, &sm.p.hi[ra][ca]);
    cs_ldsm(al, &sm.p.lo[ra][ca]);
#pragma unroll
    for (int nj = 0; nj < 2; ++nj) {
      uint32_t b[4];
      cs_ldsm_t(b, &sm.v[kk + i8 + (mat & 1 ? 8 : 0)][wn + nj * 16 + (mat >= 2 ? 8 : 0)]);
      cs_mma(acc[2 * nj], ah, b[0], b[1]);
      cs_mma(acc[2 * nj], al, b[0], b[1]);
      cs_mma(acc[2 * nj + 1], ah, b[2], b[3]);
      cs_mma(acc[2 * nj + 1], al, b[2], b[3]);
    }
  }
  if (hg.out) {  // the head's norm and its gate (columns beyond dv are zero: their V is)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      float ss = 0.f;
#pragma unroll
      for (int ni = 0; ni < 4; ++ni) ss += acc[ni][2 * half] * acc[ni][2 * half] + acc[ni][2 * half + 1] * acc[ni][2 * half + 1];
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
      if ((lane & 3) == 0) sm.squares[half_w][wm + g + half * 8] = ss;
    }
    __syncthreads();
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int i = wm + g + half * 8;
      if (i >= n) continue;
      const float inv = 1.0f / sqrtf((sm.squares[0][i] + sm.squares[1][i]) / (float)dv + hg.eps);
#pragma unroll
      for (int ni = 0; ni < 4; ++ni) {
        const int col = wn + ni * 8 + tg;
        if (col >= dv) continue;
        const size_t hc = (size_t)h * dv + col;
        const float2 gt = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(hg.gate + (size_t)(t0 + i) * hg.ld_gate + hc));
        const float2 nw = *reinterpret_cast<const float2*>(hg.norm_w + hc);
        const float a = (acc[ni][2 * half] * inv) * nw.x * __fdividef(gt.x, 1.0f + __expf(-gt.x));
        const float b = (acc[ni][2 * half + 1] * inv) * nw.y * __fdividef(gt.y, 1.0f + __expf(-gt.y));
        *reinterpret_cast<__nv_bfloat162*>(hg.out + (size_t)(t0 + i) * H * dv + hc) = __floats2bfloat162_rn(a, b);
      }
    }
    return;
  }
#pragma unroll
  for (int ni = 0; ni < 4; ++ni)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int i = wm + g + half * 8, col = v0 + wn + ni * 8 + tg;
      if (i < n && col < dv) *reinterpret_cast<float2*>(o + ((size_t)(t0 + i) * H + h) * dv + col) = make_float2(acc[ni][2 * half], acc[ni][2 * half + 1]);
    }
}

template <int DKT>
static int launch_chunks(float* o, const HeadGate& hg, float* state, const __nv_bfloat16* r, int ld_r, const __nv_bfloat16* k, int ld_k, const __nv_bfloat16* v, int ld_v,
                         const float* z, int ld_z, const float* w0, const float* u, float* added, __nv_bfloat16* before_hi,
                         __nv_bfloat16* before_lo, float* passed, const ChunkPlace& pl, int max_chunks, int H, int dk, int dv, cudaStream_t stream) {
  static bool configured = false;
  if (!configured) {
    MS_CHECK_CUDA(cudaFuncSetAttribute(tm_states_kernel<DKT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(TmStatesSmem<DKT>)));
    MS_CHECK_CUDA(cudaFuncSetAttribute(tm_outputs_kernel<DKT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(TmOutputsSmem<DKT>)));
    configured = true;
  }
  const int v_tiles = ceil_div(dv, TC_DV);
  MS_LAUNCH(tm_states_kernel<DKT>, dim3(max_chunks, H, v_tiles), CS_THREADS, sizeof(TmStatesSmem<DKT>), stream, added, passed, k, ld_k, v, ld_v, z, ld_z,
            w0, pl, H, dk, dv);
  MS_LAUNCH(tm_carry_kernel, dim3(ceil_div(H * dv * dk, CS_THREADS), pl.num_rows), CS_THREADS, 0, stream, state, before_hi, before_lo, added, passed,
            pl, H, dk, dv);
  MS_LAUNCH(tm_outputs_kernel<DKT>, dim3(max_chunks, H, v_tiles), CS_THREADS, sizeof(TmOutputsSmem<DKT>), stream, o, hg, r, ld_r, k, ld_k, v, ld_v, z, ld_z,
            w0, u, before_hi, before_lo, pl, H, dk, dv);
  return 0;
}

}  // namespace ms

using namespace ms;

MS_EXPORT int ms_channel_decay(float* out, const void* z, int ld_z, const float* w0, int tokens, int width, int dtype, cudaStream_t stream) {
  if (tokens == 0) return 0;
  const long long items = (long long)tokens * width;
  const unsigned blocks = (unsigned)((items + 255) / 256);
  if (dtype == MS_F32) MS_LAUNCH(channel_decay_kernel<float>, blocks, 256, 0, stream, out, (const float*)z, ld_z, w0, items, width);
  else MS_LAUNCH(channel_decay_kernel<__nv_bfloat16>, blocks, 256, 0, stream, out, (const __nv_bfloat16*)z, ld_z, w0, items, width);
  return 0;
}

// One token per row; dk a multiple of 4. r, k, v, gate and low are rows of one run dtype; w2 [H * dk, rank] in that dtype.
MS_EXPORT int ms_time_step(void* out, float* state, const void* r, const void* k, const void* v, const void* gate, int ld, const void* low,
                           int ld_low, const void* w2, int rank, const float* w0, const float* u, const float* norm_w, float eps,
                           const int* cu_q, const int* q_start, const int* state_slot, int num_rows, int H, int dk, int dv, int dtype,
                           cudaStream_t stream) {
  if (num_rows == 0) return 0;
  const size_t smem = ((size_t)4 * dk + dv) * sizeof(float);
  const int per16 = 16 / (dtype == MS_F32 ? 4 : 2);
  const int vec = rank % 8 == 0 && ld_low % per16 == 0 && (uintptr_t)low % 16 == 0 && (uintptr_t)w2 % 16 == 0;
  MS_CHECK_ARG(H > 0 && dk > 0 && dk % 4 == 0 && dv > 0 && rank > 0 && (uintptr_t)state % 16 == 0 && num_rows <= 65535 && smem <= 48 * 1024,
               "time_step: %d rows, heads of %d x %d, rank %d", num_rows, dk, dv, rank);
#define MS_STEP(T, LPC)                                                                                                                        \
  MS_LAUNCH((time_step_kernel<T, LPC>), dim3(H, num_rows), TS_THREADS, smem, stream, (T*)out, state, Rows<T>{(const T*)r, ld},                \
            Rows<T>{(const T*)k, ld}, Rows<T>{(const T*)v, ld}, Rows<T>{(const T*)gate, ld}, Rows<T>{(const T*)low, ld_low}, (const T*)w2, rank, w0, u, \
            norm_w, eps, cu_q, q_start, state_slot, H, dk, dv, vec)
  if (dtype == MS_F32) {
    if (dk > 64) MS_STEP(float, 32);
    else if (dk > 32) MS_STEP(float, 16);
    else MS_STEP(float, 8);
  } else {
    if (dk > 64) MS_STEP(__nv_bfloat16, 32);
    else if (dk > 32) MS_STEP(__nv_bfloat16, 16);
    else MS_STEP(__nv_bfloat16, 8);
  }
#undef MS_STEP
  return 0;
}

// 1 if the chunk kernels take these sizes.
MS_EXPORT int ms_time_chunk_supports(int dk, int dv) { return dk >= 8 && dk <= 128 && dk % 8 == 0 && dv >= 8 && dv % 8 == 0; }

// o [T, H, dv] float32, or (o null, dv <= 64) out [T, H * dv] bfloat16 = o over its root mean square per head, times norm_w, times silu(gate);
// state [slots, H, dv, dk] float32; r, k [T, H * dk], v [T, H * dv] bfloat16 rows, z [T, H * dk] float32 rows. Scratch
// [max_chunks, H, dv, dk]: added float32, before_hi and before_lo bfloat16; passed float32 [max_chunks, H, dk].
MS_EXPORT int ms_time_chunks(float* o, void* out, const void* gate, int ld_gate, const float* norm_w, float eps, float* state, const void* r, int ld_r, const void* k, int ld_k, const void* v, int ld_v, const float* z, int ld_z,
                             const float* w0, const float* u, float* added, void* before_hi, void* before_lo, float* passed, const int* tab,
                             const int* row_first, const int* cu_q, const int* q_start, const int* state_slot, int num_rows, int max_chunks, int H,
                             int dk, int dv, cudaStream_t stream) {
  if (num_rows == 0 || max_chunks == 0) return 0;
  MS_CHECK_ARG(ms_time_chunk_supports(dk, dv) && H > 0 && H <= 65535 && num_rows <= 65535 && (long long)H * dv * dk < (1LL << 31),
               "time_chunks: %d heads of %d x %d, %d rows", H, dk, dv, num_rows);
  MS_CHECK_ARG((o != nullptr) != (out != nullptr) && (!out || (dv <= TC_DV && gate && norm_w && ld_gate % 2 == 0 && (uintptr_t)gate % 4 == 0 &&
                                                              (uintptr_t)out % 4 == 0 && (uintptr_t)norm_w % 8 == 0)),
               "time_chunks: either o, or for heads of up to %d values the gated output", TC_DV);
  const HeadGate hg{(__nv_bfloat16*)out, (const __nv_bfloat16*)gate, ld_gate, norm_w, eps};
  MS_CHECK_ARG(ld_z % 2 == 0 && (uintptr_t)z % 8 == 0 && (uintptr_t)w0 % 8 == 0, "time_chunks: the decays' logits are read two at a time");
  MS_CHECK_ARG(ld_r % 8 == 0 && ld_k % 8 == 0 && ld_v % 8 == 0 && (uintptr_t)r % 16 == 0 && (uintptr_t)k % 16 == 0 && (uintptr_t)v % 16 == 0 &&
                   (uintptr_t)o % 8 == 0 && (uintptr_t)state % 16 == 0 && (uintptr_t)added % 16 == 0 && (uintptr_t)before_hi % 16 == 0 &&
                   (uintptr_t)before_lo % 16 == 0 && (uintptr_t)passed % 16 == 0 && (uintptr_t)u % 16 == 0,
               "time_chunks: operands must be aligned");
  const ChunkPlace pl{reinterpret_cast<const int2*>(tab), row_first, cu_q, q_start, state_slot, num_rows};
  const __nv_bfloat16 *rb = (const __nv_bfloat16*)r, *kb = (const __nv_bfloat16*)k, *vb = (const __nv_bfloat16*)v;
  if (dk <= 64)
    return launch_chunks<64>(o, hg, state, rb, ld_r, kb, ld_k, vb, ld_v, z, ld_z, w0, u, added, (__nv_bfloat16*)before_hi, (__nv_bfloat16*)before_lo, passed,
                             pl, max_chunks, H, dk, dv, stream);
  return launch_chunks<128>(o, hg, state, rb, ld_r, kb, ld_k, vb, ld_v, z, ld_z, w0, u, added, (__nv_bfloat16*)before_hi, (__nv_bfloat16*)before_lo, passed,
                            pl, max_chunks, H, dk, dv, stream);
}
