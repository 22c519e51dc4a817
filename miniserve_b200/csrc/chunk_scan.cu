// The decay rule with one decay per head, over chunks of a prompt on the tensor cores.
//
//   S_t = a_t S_(t-1) + w_t k_t v_t^T,  o_t = S_t^T (q_t q_scale)      (a_t in [0, 1], w_t: float32 per token and head)
//
// Inside a chunk of 64 tokens this is attention without a softmax: with D_ij = w_j a_(j+1) .. a_i for j <= i,
//   o_i = q_scale (sum_j D_ij (q_i . k_j) v_j + (a_first .. a_i) S_before^T q_i),
// and a chunk changes the state by S_after = (a_first .. a_last) S_before + sum_j D_(last, j) k_j v_j^T. Three launches:
//   states    what every chunk adds to the state, sum_j D_(last, j) k_j v_j^T, all chunks at once;
//   carry     the states before every chunk (a short walk over a row's chunks, elementwise) and the row's last state;
//   outputs   both terms of o, all chunks at once.
// q, k and v are bfloat16. What multiplies them and is not exact in bfloat16 (v w, the weighted scores, the state) goes to the
// tensor cores as two bfloat16 numbers, hi = round(x) and lo = round(x - hi), one product each, accumulated in float32: about
// 17 bits of x. The state is carried in float32. Products of decays are worked out as products (they go to zero where they must), by
// blocks of 16 tokens: all pairs within a block, and from a block's ends across the blocks between.
//
// With `ones` there is one more value column whose value is one (the decayed sum of the keys): it is summed in float32 and
// comes out behind the dv columns.
//
// A table on the device says which row and tokens a chunk has; grids are sized for the most chunks that a step of so many
// tokens and rows can have, surplus CTAs leave at once.
#include "chunk_mma.cuh"

namespace ms {

constexpr int CS_DV = 128, CS_DKT = 128;
constexpr int CS_KB = 32;  // key channels of the state staged at a time by the outputs kernel

// tab[c] = (row, first flat token) of chunk c, row_first[r] the row's first chunk (row_first[num_rows]: how many chunks there are)
__global__ void __launch_bounds__(CS_THREADS)
chunk_table_kernel(int2* __restrict__ tab, int* __restrict__ row_first, const int* __restrict__ cu_q, int num_rows) {
  pdl_prologue();
  __shared__ int part[CS_THREADS];
  __shared__ int base;
  if (threadIdx.x == 0) base = 0;
  __syncthreads();
  for (int r0 = 0; r0 < num_rows; r0 += CS_THREADS) {
    const int r = r0 + threadIdx.x;
    const int t0 = r < num_rows ? cu_q[r] : 0, len = r < num_rows ? cu_q[r + 1] - t0 : 0;
    const int mine = (len + CS_TOK - 1) / CS_TOK;
    part[threadIdx.x] = mine;
    __syncthreads();
    int before = base;
    for (int i = 0; i < (int)threadIdx.x; ++i) before += part[i];
    if (r < num_rows) {
      row_first[r] = before;
      for (int c = 0; c < mine; ++c) tab[before + c] = make_int2(r, t0 + c * CS_TOK);
    }
    __syncthreads();
    if (threadIdx.x == CS_THREADS - 1) base = before + mine;
    __syncthreads();
  }
  if (threadIdx.x == 0) row_first[num_rows] = base;
}

// A chunk's decays in shared memory, from a [T, H]: per token the product of the decays from the first token of its block of 16 to it
// and the product behind it to the block's end; the products between all pairs of a block; per pair of blocks the product of the whole
// blocks between.
struct ChunkDecays {
  float pre[CS_TOK], suf[CS_TOK], w[CS_TOK];
  float inside[4][16][16];  // [block][j][i]: a_(j+1) .. a_i
  float whole[4], between[4][4], before[4];  // before[b]: the product of the blocks ahead of block b
};

// Tokens from n on count as decay 1 and factor 0. Ends with a barrier.
__device__ __forceinline__ void chunk_decays(ChunkDecays& cd, const float* __restrict__ decay, const float* __restrict__ write, int t0, int n, int H,
                                             int h) {
  if (threadIdx.x < CS_TOK) {
    const int i = threadIdx.x, in = i & 15;
    const float a = i < n ? decay[(size_t)(t0 + i) * H + h] : 1.f;
    cd.w[i] = i < n ? (write ? write[(size_t)(t0 + i) * H + h] : 1.f) : 0.f;
    float p = a, s = a;
#pragma unroll
    for (int o = 1; o < 16; o <<= 1) {
      const float pp = __shfl_up_sync(0xffffffffu, p, o, 16), ps = __shfl_down_sync(0xffffffffu, s, o, 16);
      if (in >= o) p *= pp;
      if (in + o < 16) s *= ps;
    }
    const float behind = __shfl_down_sync(0xffffffffu, s, 1, 16);
    cd.pre[i] = p;
    cd.suf[i] = in == 15 ? 1.f : behind;
    if (in == 15) cd.whole[i >> 4] = p;
    float run = 1.f;
#pragma unroll
    for (int j = 0; j < 16; ++j) {  // this token's row: times the next tokens' decays in turn
      const float next = __shfl_sync(0xffffffffu, a, j, 16);
      if (j > in) run *= next;
      cd.inside[i >> 4][in][j] = run;
    }
  }
  __syncthreads();
  if (threadIdx.x < 16) {
    const int bj = threadIdx.x >> 2, bi = threadIdx.x & 3;
    float f = 1.f;
    for (int b = bj + 1; b < bi; ++b) f *= cd.whole[b];
    cd.between[bj][bi] = f;
    if (bj == 0) {
      float g = 1.f;
      for (int b = 0; b < bi; ++b) g *= cd.whole[b];
      cd.before[bi] = g;
    }
  }
  __syncthreads();
}
// a_(j+1) .. a_i for j <= i
__device__ __forceinline__ float decay_between(const ChunkDecays& cd, int j, int i) {
  const int bj = j >> 4, bi = i >> 4;
  return bj == bi ? cd.inside[bi][j & 15][i & 15] : cd.suf[j] * cd.between[bj][bi] * cd.pre[i];
}

// ---------------------------------------------------------------- states
// ds [chunks, H, dv (+ 1), dk] float32, chunk_decay [chunks, H]. grid (chunks, H, dv tiles * dk tiles).
struct StatesSmem {
  __nv_bfloat16 vhi[CS_TOK][CS_DV + 8], vlo[CS_TOK][CS_DV + 8], k[CS_TOK][CS_DKT + 8];
  ChunkDecays cd;
  float wl[CS_TOK];  // D_(last, j)
};

__global__ void __launch_bounds__(CS_THREADS)
chunk_states_kernel(float* __restrict__ ds, float* __restrict__ chunk_decay, const __nv_bfloat16* __restrict__ k, int ld_k, int qk_group,
                    const __nv_bfloat16* __restrict__ v, int ld_v, const float* __restrict__ decay, const float* __restrict__ write,
                    const int2* __restrict__ tab, const int* __restrict__ row_first, const int* __restrict__ cu_q, int num_rows, int H, int dk,
                    int dv, int dk_tiles, int ones) {
  extern __shared__ __align__(16) unsigned char cs_raw[];
  StatesSmem& sm = *reinterpret_cast<StatesSmem*>(cs_raw);
  pdl_prologue();
  const int chunk = blockIdx.x, h = blockIdx.y;
  if (chunk >= row_first[num_rows]) return;
  const int2 at = tab[chunk];
  const int t0 = at.y, n = min(CS_TOK, cu_q[at.x + 1] - t0);
  const int vt = blockIdx.z / dk_tiles, kt = blockIdx.z - vt * dk_tiles;
  const int v0 = vt * CS_DV, k0 = kt * CS_DKT;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const __nv_bfloat16* kh = k + (size_t)(h / qk_group) * dk + k0;
  for (int idx = tid; idx < CS_TOK * (CS_DKT / 8); idx += CS_THREADS) {
    const int tt = idx / (CS_DKT / 8), c = (idx - tt * (CS_DKT / 8)) * 8;
    const bool in = tt < n && k0 + c < dk;
    cs_cp16(&sm.k[tt][c], in ? (const void*)(kh + (size_t)(t0 + tt) * ld_k + c) : (const void*)k, in);
  }
  cs_commit();
  chunk_decays(sm.cd, decay, write, t0, n, H, h);
  if (tid < CS_TOK) sm.wl[tid] = tid < n ? decay_between(sm.cd, tid, n - 1) * sm.cd.w[tid] : 0.f;
  if (tid == 0 && blockIdx.z == 0) chunk_decay[(size_t)chunk * H + h] = sm.cd.before[(n - 1) >> 4] * sm.cd.pre[n - 1];
  __syncthreads();
  const __nv_bfloat16* vh = v + (size_t)h * dv + v0;
  for (int idx = tid; idx < CS_TOK * (CS_DV / 8); idx += CS_THREADS) {
    const int tt = idx / (CS_DV / 8), c = (idx - tt * (CS_DV / 8)) * 8;
    float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (tt < n && v0 + c < dv) bf16x8_to_float(*reinterpret_cast<const uint4*>(vh + (size_t)(t0 + tt) * ld_v + c), f);
    const float w = sm.wl[tt];
    __align__(16) __nv_bfloat16 hi[8];
    __align__(16) __nv_bfloat16 lo[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) cs_split(f[e] * w, hi[e], lo[e]);
    *reinterpret_cast<uint4*>(&sm.vhi[tt][c]) = *reinterpret_cast<const uint4*>(hi);
    *reinterpret_cast<uint4*>(&sm.vlo[tt][c]) = *reinterpret_cast<const uint4*>(lo);
  }
  cs_wait<0>();
  __syncthreads();
  const int wm = (warp >> 1) * 32, wn = (warp & 1) * 64;  // 4 x 2 warps of 32 value rows x 64 key columns
  float acc[2][8][4] = {};
  const int i8 = lane & 7, mat = lane >> 3;
#pragma unroll
  for (int kk = 0; kk < CS_TOK; kk += 16) {
    uint32_t ah[2][4], al[2][4];
#pragma unroll
    for (int mi = 0; mi < 2; ++mi) {
      const int row = kk + i8 + (mat >= 2 ? 8 : 0), col = wm + mi * 16 + (mat & 1 ? 8 : 0);
      cs_ldsm_t(ah[mi], &sm.vhi[row][col]);
      cs_ldsm_t(al[mi], &sm.vlo[row][col]);
    }
#pragma unroll
    for (int nj = 0; nj < 4; ++nj) {
      uint32_t b[4];
      cs_ldsm_t(b, &sm.k[kk + i8 + (mat & 1 ? 8 : 0)][wn + nj * 16 + (mat >= 2 ? 8 : 0)]);
#pragma unroll
      for (int mi = 0; mi < 2; ++mi) {
        cs_mma(acc[mi][2 * nj], ah[mi], b[0], b[1]);
        cs_mma(acc[mi][2 * nj], al[mi], b[0], b[1]);
        cs_mma(acc[mi][2 * nj + 1], ah[mi], b[2], b[3]);
        cs_mma(acc[mi][2 * nj + 1], al[mi], b[2], b[3]);
      }
    }
  }
  float* out = ds + ((size_t)chunk * H + h) * (size_t)(dv + ones) * dk;
  const int g = lane >> 2, tg = (lane & 3) * 2;
#pragma unroll
  for (int mi = 0; mi < 2; ++mi)
#pragma unroll
    for (int ni = 0; ni < 8; ++ni)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int row = v0 + wm + mi * 16 + g + half * 8, col = k0 + wn + ni * 8 + tg;  // (dk is even: a pair is inside or outside)
        if (row < dv && col < dk) *reinterpret_cast<float2*>(out + (size_t)row * dk + col) = make_float2(acc[mi][ni][2 * half], acc[mi][ni][2 * half + 1]);
      }
  if (ones && vt == 0 && tid < CS_DKT && k0 + tid < dk) {
    float s = 0.f;
    for (int j = 0; j < n; ++j) s = fmaf(sm.wl[j], __bfloat162float(sm.k[j][tid]), s);
    out[(size_t)dv * dk + k0 + tid] = s;
  }
}

// ---------------------------------------------------------------- carry
// before_hi / before_lo [chunks, H, dv (+ 1), dk]: the state before every chunk as two bfloat16; the row's slot of state
// [slots, H, dv (+ 1), dk] gets the state behind its last chunk. Four elements per thread; grid (elements of a row's state, rows).
__global__ void __launch_bounds__(CS_THREADS)
chunk_carry_kernel(float* __restrict__ state, __nv_bfloat16* __restrict__ before_hi, __nv_bfloat16* __restrict__ before_lo,
                   const float* __restrict__ ds, const float* __restrict__ chunk_decay, const int* __restrict__ row_first,
                   const int* __restrict__ q_start, const int* __restrict__ state_slot, int H, int per_head, int total4) {
  pdl_prologue();
  const int i4 = blockIdx.x * CS_THREADS + threadIdx.x, r = blockIdx.y;
  if (i4 >= total4) return;
  const int h = i4 * 4 / per_head;
  const int c0 = row_first[r], c1 = row_first[r + 1];
  if (c1 <= c0) return;
  float4* slot = reinterpret_cast<float4*>(state) + (size_t)state_slot[r] * total4 + i4;
  float4 S = q_start[r] == 0 ? make_float4(0.f, 0.f, 0.f, 0.f) : *slot;
#pragma unroll 4
  for (int c = c0; c < c1; ++c) {
    const size_t at = (size_t)c * total4 + i4;
    const float4 d = reinterpret_cast<const float4*>(ds)[at];
    const float a = chunk_decay[(size_t)c * H + h];
    __align__(8) __nv_bfloat16 hi[4];
    __align__(8) __nv_bfloat16 lo[4];
    cs_split(S.x, hi[0], lo[0]);
    cs_split(S.y, hi[1], lo[1]);
    cs_split(S.z, hi[2], lo[2]);
    cs_split(S.w, hi[3], lo[3]);
    reinterpret_cast<uint2*>(before_hi)[at] = *reinterpret_cast<const uint2*>(hi);
    reinterpret_cast<uint2*>(before_lo)[at] = *reinterpret_cast<const uint2*>(lo);
    S = make_float4(fmaf(a, S.x, d.x), fmaf(a, S.y, d.y), fmaf(a, S.z, d.z), fmaf(a, S.w, d.w));
  }
  *slot = S;
}

// ---------------------------------------------------------------- outputs
// o [T, H, ld_o] float32: dv columns (and with `ones` the column behind them). grid (chunks, H, dv tiles).
// shared memory: decays | row sums [2][64] | state stages [2][2][128][40] | V [64][136] | Q [64][dkp + 8] | K [64][dkp + 8], whose place the
// weighted scores P hi, lo [64][72] take once every warp has read it
constexpr int CS_LDP = CS_TOK + 8, CS_LDS = CS_KB + 8, CS_LDV = CS_DV + 8;
constexpr size_t CS_OUT_FIXED = sizeof(ChunkDecays) + 2 * CS_TOK * 4 + 4 * CS_DV * CS_LDS * 2 + CS_TOK * CS_LDV * 2;
constexpr size_t CS_P_BYTES = 2 * CS_TOK * CS_LDP * 2;
static_assert(sizeof(ChunkDecays) % 16 == 0, "what follows the decays starts on 16 bytes");

__global__ void __launch_bounds__(CS_THREADS)
chunk_outputs_kernel(float* __restrict__ o, int ld_o, const __nv_bfloat16* __restrict__ q, int ld_q, const __nv_bfloat16* __restrict__ k, int ld_k,
                     int qk_group, const __nv_bfloat16* __restrict__ v, int ld_v, const float* __restrict__ decay,
                     const float* __restrict__ write, const __nv_bfloat16* __restrict__ before_hi, const __nv_bfloat16* __restrict__ before_lo,
                     const int2* __restrict__ tab, const int* __restrict__ row_first, const int* __restrict__ cu_q,
                     const int* __restrict__ q_start, int num_rows, int H, int dk, int dv, float q_scale, int ones) {
  extern __shared__ __align__(16) unsigned char cs_raw[];
  ChunkDecays& cd = *reinterpret_cast<ChunkDecays*>(cs_raw);
  float (*rs)[CS_TOK] = reinterpret_cast<float (*)[CS_TOK]>(cs_raw + sizeof(ChunkDecays));
  __nv_bfloat16* stage = reinterpret_cast<__nv_bfloat16*>(rs + 2);  // [buffer][hi, lo][CS_DV][CS_LDS]
  __nv_bfloat16* vs = stage + 4 * CS_DV * CS_LDS;                   // [CS_TOK][CS_LDV]
  const int dkp = (dk + 15) & ~15, ldk = dkp + 8;
  __nv_bfloat16* qs = vs + CS_TOK * CS_LDV;
  __nv_bfloat16* ks = qs + CS_TOK * ldk;
  __nv_bfloat16* p_hi = ks;
  __nv_bfloat16* p_lo = p_hi + CS_TOK * CS_LDP;
  pdl_prologue();
  const int chunk = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * CS_DV;
  if (chunk >= row_first[num_rows]) return;
  const int2 at = tab[chunk];
  const int t0 = at.y, n = min(CS_TOK, cu_q[at.x + 1] - t0);
  const bool has_state = !(q_start[at.x] == 0 && chunk == row_first[at.x]);  // else nothing came before
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int i8 = lane & 7, mat = lane >> 3, g = lane >> 2, tg = (lane & 3) * 2;
  {
    const size_t head = (size_t)(h / qk_group) * dk;
    const int groups = dkp / 8;
    for (int idx = tid; idx < CS_TOK * groups; idx += CS_THREADS) {
      const int tt = idx / groups, c = (idx - tt * groups) * 8;
      const bool in = tt < n && c < dk;
      cs_cp16(qs + tt * ldk + c, in ? (const void*)(q + (size_t)(t0 + tt) * ld_q + head + c) : (const void*)q, in);
      cs_cp16(ks + tt * ldk + c, in ? (const void*)(k + (size_t)(t0 + tt) * ld_k + head + c) : (const void*)k, in);
    }
  }
  cs_commit();
  const size_t st_at = ((size_t)chunk * H + h) * (size_t)(dv + ones) * dk;
  auto load_state = [&](int buf, int kb) {
    for (int idx = tid; idx < CS_DV * (CS_KB / 8); idx += CS_THREADS) {
      const int row = idx / (CS_KB / 8), c = (idx - row * (CS_KB / 8)) * 8;
      const bool in = v0 + row < dv && kb + c < dk;
      const size_t src = in ? st_at + (size_t)(v0 + row) * dk + kb + c : 0;
      __nv_bfloat16* dst = stage + (size_t)(buf * 2) * CS_DV * CS_LDS + row * CS_LDS + c;
      cs_cp16(dst, before_hi + src, in);
      cs_cp16(dst + CS_DV * CS_LDS, before_lo + src, in);
    }
  };
  for (int idx = tid; idx < CS_TOK * (CS_DV / 8); idx += CS_THREADS) {
    const int tt = idx / (CS_DV / 8), c = (idx - tt * (CS_DV / 8)) * 8;
    const bool in = tt < n && v0 + c < dv;
    cs_cp16(vs + tt * CS_LDV + c, in ? (const void*)(v + (size_t)(t0 + tt) * ld_v + (size_t)h * dv + v0 + c) : (const void*)v, in);
  }
  if (has_state) load_state(0, 0);
  cs_commit();
  chunk_decays(cd, decay, write, t0, n, H, h);
  cs_wait<1>();  // q and k
  __syncthreads();

  // the weighted scores: 4 x 2 warps of 16 tokens x 32 tokens
  const int wm = (warp >> 1) * 16, wn2 = warp & 1;
  {
    float s[4][4] = {};
    const int j0 = wn2 * 32;
    if (j0 <= wm + 15) {
      for (int kk = 0; kk < dkp; kk += 16) {
        uint32_t a[4];
        cs_ldsm(a, qs + (wm + i8 + (mat & 1 ? 8 : 0)) * ldk + kk + (mat >= 2 ? 8 : 0));
#pragma unroll
        for (int nj = 0; nj < 2; ++nj) {
          uint32_t b[4];
          cs_ldsm(b, ks + (j0 + nj * 16 + i8 + (mat >= 2 ? 8 : 0)) * ldk + kk + (mat & 1 ? 8 : 0));
          cs_mma(s[2 * nj], a, b[0], b[1]);
          cs_mma(s[2 * nj + 1], a, b[2], b[3]);
        }
      }
    }
    __syncthreads();  // every warp is done with K
    float sum[2] = {0.f, 0.f};
#pragma unroll
    for (int nj = 0; nj < 4; ++nj)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int i = wm + g + half * 8, j = j0 + nj * 8 + tg;
        __align__(4) __nv_bfloat16 hi[2];
        __align__(4) __nv_bfloat16 lo[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float x = 0.f;
          if (j + e <= i) x = s[nj][2 * half + e] * q_scale * decay_between(cd, j + e, i) * cd.w[j + e];  // (tokens from n on have w = 0)
          sum[half] += x;
          cs_split(x, hi[e], lo[e]);
        }
        *reinterpret_cast<uint32_t*>(p_hi + i * CS_LDP + j) = *reinterpret_cast<const uint32_t*>(hi);
        *reinterpret_cast<uint32_t*>(p_lo + i * CS_LDP + j) = *reinterpret_cast<const uint32_t*>(lo);
      }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      float x = sum[half];
      x += __shfl_xor_sync(0xffffffffu, x, 1);
      x += __shfl_xor_sync(0xffffffffu, x, 2);
      if ((lane & 3) == 0) rs[wn2][wm + g + half * 8] = x;
    }
  }

  // what came before the chunk: 4 x 2 warps of 16 tokens x 64 value columns
  const int wn = wn2 * 64;
  float acc[8][4] = {};
  if (has_state) {
    int buf = 0;
    for (int kb = 0; kb < dkp; kb += CS_KB, buf ^= 1) {
      cs_wait<0>();
      __syncthreads();  // this stage is there, and the other one is free
      if (kb + CS_KB < dkp) load_state(buf ^ 1, kb + CS_KB);
      cs_commit();
      const __nv_bfloat16* hi = stage + (size_t)(buf * 2) * CS_DV * CS_LDS;
#pragma unroll
      for (int kk = 0; kk < CS_KB; kk += 16) {
        if (kb + kk >= dkp) break;
        uint32_t a[4];
        cs_ldsm(a, qs + (wm + i8 + (mat & 1 ? 8 : 0)) * ldk + kb + kk + (mat >= 2 ? 8 : 0));
#pragma unroll
        for (int nj = 0; nj < 4; ++nj) {
          uint32_t bh[4], bl[4];
          const int at_b = (wn + nj * 16 + i8 + (mat >= 2 ? 8 : 0)) * CS_LDS + kk + (mat & 1 ? 8 : 0);
          cs_ldsm(bh, hi + at_b);
          cs_ldsm(bl, hi + CS_DV * CS_LDS + at_b);
          cs_mma(acc[2 * nj], a, bh[0], bh[1]);
          cs_mma(acc[2 * nj], a, bl[0], bl[1]);
          cs_mma(acc[2 * nj + 1], a, bh[2], bh[3]);
          cs_mma(acc[2 * nj + 1], a, bl[2], bl[3]);
        }
      }
    }
    const float c0 = cd.before[(wm + g) >> 4] * cd.pre[wm + g] * q_scale, c1 = cd.before[(wm + g + 8) >> 4] * cd.pre[wm + g + 8] * q_scale;
#pragma unroll
    for (int ni = 0; ni < 8; ++ni) {
      acc[ni][0] *= c0;
      acc[ni][1] *= c0;
      acc[ni][2] *= c1;
      acc[ni][3] *= c1;
    }
  }
  cs_wait<0>();
  __syncthreads();  // the scores and V are there
  for (int kk = 0; kk <= wm; kk += 16) {  // (later tokens have no weight)
    uint32_t ah[4], al[4];
    const int at_a = (wm + i8 + (mat & 1 ? 8 : 0)) * CS_LDP + kk + (mat >= 2 ? 8 : 0);
    cs_ldsm(ah, p_hi + at_a);
    cs_ldsm(al, p_lo + at_a);
#pragma unroll
    for (int nj = 0; nj < 4; ++nj) {
      uint32_t b[4];
      cs_ldsm_t(b, vs + (kk + i8 + (mat & 1 ? 8 : 0)) * CS_LDV + wn + nj * 16 + (mat >= 2 ? 8 : 0));
      cs_mma(acc[2 * nj], ah, b[0], b[1]);
      cs_mma(acc[2 * nj], al, b[0], b[1]);
      cs_mma(acc[2 * nj + 1], ah, b[2], b[3]);
      cs_mma(acc[2 * nj + 1], al, b[2], b[3]);
    }
  }
#pragma unroll
  for (int ni = 0; ni < 8; ++ni)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int i = wm + g + half * 8, col = v0 + wn + ni * 8 + tg;
      if (i < n && col < dv) *reinterpret_cast<float2*>(o + ((size_t)(t0 + i) * H + h) * ld_o + col) = make_float2(acc[ni][2 * half], acc[ni][2 * half + 1]);
    }
  if (ones && blockIdx.z == 0) {
    const __nv_bfloat16* nh = before_hi + st_at + (size_t)dv * dk;
    const __nv_bfloat16* nl = before_lo + st_at + (size_t)dv * dk;
    for (int i = warp; i < n; i += CS_THREADS / 32) {
      float x = 0.f;
      if (has_state) {
        for (int c = lane; c < dk; c += 32)
          x = fmaf(__bfloat162float(qs[i * ldk + c]), __bfloat162float(nh[c]) + __bfloat162float(nl[c]), x);
        x = warp_sum(x) * (cd.before[i >> 4] * cd.pre[i] * q_scale);
      }
      if (lane == 0) o[((size_t)(t0 + i) * H + h) * ld_o + dv] = x + (rs[0][i] + rs[1][i]);
    }
  }
}

}  // namespace ms

using namespace ms;

// The most chunks that a step of so many tokens in so many rows can have.
MS_EXPORT int ms_chunk_max(int tokens, int rows) { return tokens / CS_TOK + rows; }

// 1 if the kernels take these sizes.
MS_EXPORT int ms_chunk_supports(int dk, int dv) { return dk >= 8 && dk <= 256 && dk % 8 == 0 && dv >= 8 && dv % 8 == 0; }

MS_EXPORT int ms_chunk_table(int* tab, int* row_first, const int* cu_q, int num_rows, cudaStream_t stream) {
  if (num_rows == 0) return 0;
  MS_LAUNCH(chunk_table_kernel, 1, CS_THREADS, 0, stream, reinterpret_cast<int2*>(tab), row_first, cu_q, num_rows);
  return 0;
}

// o [T, H, ld_o] float32; state [slots, H, dv + ones, dk] float32. Scratch: ds float32 and before_hi, before_lo bfloat16, each
// [max_chunks, H, dv + ones, dk]; chunk_decay float32 [max_chunks, H].
MS_EXPORT int ms_chunk_scan(float* o, int ld_o, float* state, const void* q, int ld_q, const void* k, int ld_k, int qk_group, const void* v, int ld_v,
                            const float* decay, const float* write, float* ds, void* before_hi, void* before_lo, float* chunk_decay,
                            const int* tab, const int* row_first, const int* cu_q, const int* q_start, const int* state_slot, int num_rows,
                            int max_chunks, int H, int dk, int dv, float q_scale, int ones, cudaStream_t stream) {
  if (num_rows == 0 || max_chunks == 0) return 0;
  MS_CHECK_ARG(ms_chunk_supports(dk, dv) && (ones == 0 || ones == 1), "chunk_scan: heads of %d x %d", dk, dv);
  MS_CHECK_ARG(qk_group > 0 && H % qk_group == 0 && H <= 65535 && num_rows <= 65535, "chunk_scan: %d heads in groups of %d, %d rows", H, qk_group, num_rows);
  MS_CHECK_ARG(ld_q % 8 == 0 && ld_k % 8 == 0 && ld_v % 8 == 0 && ld_o % 2 == 0 && ld_o >= dv + ones && (uintptr_t)q % 16 == 0 && (uintptr_t)k % 16 == 0 &&
                   (uintptr_t)v % 16 == 0 && (uintptr_t)o % 8 == 0 && (uintptr_t)state % 16 == 0 && (uintptr_t)ds % 16 == 0 &&
                   (uintptr_t)before_hi % 16 == 0 && (uintptr_t)before_lo % 16 == 0,
               "chunk_scan: operands must be aligned");
  const __nv_bfloat16 *qb = (const __nv_bfloat16*)q, *kb = (const __nv_bfloat16*)k, *vb = (const __nv_bfloat16*)v;
  const int2* tb = reinterpret_cast<const int2*>(tab);
  const int v_tiles = ceil_div(dv, CS_DV), k_tiles = ceil_div(dk, CS_DKT);
  static size_t configured = 0;
  const size_t qk_bytes = (size_t)CS_TOK * (((dk + 15) & ~15) + 8) * 2;
  const size_t out_smem = CS_OUT_FIXED + qk_bytes + (qk_bytes > CS_P_BYTES ? qk_bytes : CS_P_BYTES);
  if (configured == 0)
    MS_CHECK_CUDA(cudaFuncSetAttribute(chunk_states_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(StatesSmem)));
  if (out_smem > configured) {
    MS_CHECK_CUDA(cudaFuncSetAttribute(chunk_outputs_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)out_smem));
    configured = out_smem;
  }
  MS_LAUNCH(chunk_states_kernel, dim3(max_chunks, H, v_tiles * k_tiles), CS_THREADS, sizeof(StatesSmem), stream, ds, chunk_decay, kb, ld_k,
            qk_group, vb, ld_v, decay, write, tb, row_first, cu_q, num_rows, H, dk, dv, k_tiles, ones);
  const int per_head = (dv + ones) * dk;
  const long long total = (long long)H * per_head;
  MS_CHECK_ARG(total < (1LL << 31), "chunk_scan: a state of %lld numbers", total);
  const int total4 = (int)(total / 4);
  MS_LAUNCH(chunk_carry_kernel, dim3((unsigned)((total4 + CS_THREADS - 1) / CS_THREADS), num_rows), CS_THREADS, 0, stream, state,
            (__nv_bfloat16*)before_hi, (__nv_bfloat16*)before_lo, ds, chunk_decay, row_first, q_start, state_slot, H, per_head, total4);
  MS_LAUNCH(chunk_outputs_kernel, dim3(max_chunks, H, v_tiles), CS_THREADS, out_smem, stream, o, ld_o, qb, ld_q, kb, ld_k, qk_group, vb, ld_v,
            decay, write, (const __nv_bfloat16*)before_hi, (const __nv_bfloat16*)before_lo, tb, row_first, cu_q, q_start, num_rows, H, dk, dv,
            q_scale, ones);
  return 0;
}
