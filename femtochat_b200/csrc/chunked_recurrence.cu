// The recurrences of recurrence.cu for a run of tokens, in chunks of 64, on the tensor cores.
//
// With Gamma_t the product of a chunk's decays up to token t (per key channel), S_0 the state before the chunk and
//   A_tj = sum_d k_t[d] k_j[d] Gamma_t[d] / Gamma_j[d]   (j < t),     B_tj likewise with q_t (j <= t),
// the gated delta rule over a chunk is
//   U = (I + diag(beta) A)^-1 diag(beta) (V - K~ S_0),   K~_t = Gamma_t k_t,
//   O = Q~ S_0 + B U,                                     Q~_t = Gamma_t q_t,
//   S = Gamma_C S_0 + K^ ^T U,                            K^_j = Gamma_C / Gamma_j k_j.
// k_chunk_local computes everything that does not need S_0, for all chunks at once: W = (..)^-1 diag(beta) K~,
// U_0 = (..)^-1 diag(beta) V, Q~, K^ and B.  k_chunk_scan walks the chunks: U = U_0 - W S_0, then O and the next state.
// The plain decayed sum (lightning attention) is the case without A: U = V.
//
// Everything here is fp32 or a sum of two bf16 numbers: a product of two fp32 matrices is three bf16 products
// (high high, high low, low high; relative error about 2^-16) accumulated in fp32, and the state itself stays in fp32
// registers.  Quotients of decays are formed as exponentials of differences of cumulated logarithms.  Between
// different blocks of 16 tokens both exponents are taken from the later block's start and are never positive; inside
// a block the exponent of the earlier token is positive and bounded by RANGE, or the block is computed pair by pair.
//
// The tiles are 16 columns of the state wide because the chunks of a head follow one another: with 64 or 128 rows, as
// tcgen05 wants them, a prompt of one sequence would occupy one SM per head.
#include <algorithm>

#include "decoder.cuh"
#include "sm100_ptx.cuh"

using namespace sm100;

namespace {

constexpr int C = 64;                 // tokens per chunk
constexpr int LOCAL_WARPS = 16, LOCAL_THREADS = LOCAL_WARPS * 32;
constexpr int SCAN_THREADS = 256;
constexpr int MAX_TAPS = 8;
constexpr float LOG2E = 1.4426950408889634f;
constexpr float RANGE = 100.f;        // largest positive exponent (base 2) inside a block of 16 tokens

// ---- workspace of one (column, head, chunk): bf16 tiles [64][DP] or [64][64], 16-byte units of row r permuted by r & 7
template <int DP> struct Item {
  static constexpr size_t TILE = (size_t)C * DP * 2, BT = (size_t)C * C * 2;
  static constexpr size_t W = 0, Q = 2 * TILE, X_BYTES = 4 * TILE;              // first half of a chunk: W and Q~, high and low
  static constexpr size_t K = X_BYTES, B = K + 2 * TILE, G = B + 2 * BT;       // second half: K^, B, Gamma_C (fp32)
  static constexpr size_t Y_BYTES = 2 * TILE + 2 * BT + DP * 4;
  static constexpr size_t U = X_BYTES + Y_BYTES;                                // U_0: fp32 [vdim / 16][64][16]
  static size_t bytes(int E) { return U + (size_t)(E + 15) / 16 * 16 * C * 4; }
};

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

__device__ __forceinline__ uint32_t bf2(float lo, float hi) {
  __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&h);
}
// (x, y) as a high and a low pair of bf16 numbers
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = bf2(x - __bfloat162float(h.x), y - __bfloat162float(h.y));
}
// D += A (16 x 16, row) B (16 x 8, col)
__device__ __forceinline__ void mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)) : "memory");
}
// element offset of (row, col) in a tile of `width` columns
__device__ __forceinline__ int swz(int row, int col, int width) { return row * width + ((((col >> 3) ^ (row & 7)) << 3) | (col & 7)); }

// ---- local part -------------------------------------------------------------------------------------------------------
template <int DP, bool DELTA>
__global__ void __launch_bounds__(LOCAL_THREADS, 1) k_chunk_local(const ChunkArgs a) {
  pdl_trigger();
  constexpr int ST = DP + 8, AT = C + 4;
  extern __shared__ __align__(16) float sm[];
  float* sk = sm;                         // [64][ST] k
  float* sq = sk + C * ST;                // [64][ST] q
  float* sl = sq + C * ST;                // [64][ST] cumulated log2 decays; later v
  float* sf = sl + C * ST;                // [64][ST] 2^(L_t - L at the block's start)   (DELTA only, as is A)
  float* sA = sf + (DELTA ? C * ST : 0);  // [64][AT] diag(beta) A, then scratch of the inverse
  float* sX = sA + (DELTA ? C * AT : 0);  // [64][AT] the inverse, times diag(beta)
  float* sB = sX + (DELTA ? C * AT : 0);  // [64][AT] B
  float* pw = sB + C * AT;                // [65] powers of the decay, or [64] beta
  float* cw = pw + 72;                    // [3][MAX_TAPS][128] taps
  int* slow = reinterpret_cast<int*>(cw + (DELTA ? 3 * MAX_TAPS * 128 : 0));   // [4]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int chunk = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const int D = a.dim, E = a.vdim, H = a.heads, qh = h / (H / a.qk_heads);
  const int t0 = a.t0 + chunk * C, n = min(C, a.T - t0);
  const long long r0 = (long long)b * a.T + t0;
  char* item = a.ws + (((long long)b * H + h) * gridDim.x + chunk) * a.item_bytes;
  const bf16* proj = reinterpret_cast<const bf16*>(a.proj);
  const int G = a.qk_heads, channels = 2 * G * D + H * E, keep = a.taps - 1;
  const bf16* tail = reinterpret_cast<const bf16*>(a.tail_in) + (long long)b * keep * channels;
  // input of a convolution `back` tokens before token t of this chunk
  auto input = [&](int t, int back, int seg, int chan) {
    const int r = t0 + t - back;
    return __bfloat162float(r >= 0 ? proj[(r0 + t - back) * a.ldp + seg] : tail[(long long)(keep + r) * channels + chan]);
  };
  if (DELTA) {
    for (int i = tid; i < 3 * a.taps * 128; i += LOCAL_THREADS) {
      const int which = i / (a.taps * 128), j = i / 128 % a.taps, c = i % 128;
      const float* src = which == 0 ? a.conv_q : which == 1 ? a.conv_k : a.conv_v;
      const int size = which == 2 ? E : D, head = which == 2 ? h : qh;
      cw[(which * MAX_TAPS + j) * 128 + c] = c < size ? src[(long long)(head * size + c) * a.taps + j] : 0.f;
    }
    if (tid < C) pw[tid] = tid < n ? 1.f / (1.f + expf(-__bfloat162float(proj[(r0 + tid) * a.ldp + a.s_b + h]))) : 0.f;
    if (tid < 4) slow[tid] = 0;
    __syncthreads();
  } else if (tid <= C) {
    pw[tid] = powf(a.decay[h], (float)tid);
  }
  // q and k: one warp per (token, which)
  for (int it = warp; it < 2 * C; it += LOCAL_WARPS) {
    const int t = it >> 1, which = it & 1;
    float* dst = (which ? sk : sq) + t * ST;
    float y[DP / 32], ss = 0.f;
#pragma unroll
    for (int i = 0; i < DP / 32; i++) {
      const int c = i * 32 + lane;
      y[i] = 0.f;
      if (t < n && c < D) {
        const int seg = (which ? a.s_k : a.s_q) + qh * D + c;
        if (DELTA) {
          float acc = 0.f;
          for (int j = 0; j < a.taps; j++)
            acc += cw[(which * MAX_TAPS + j) * 128 + c] * input(t, keep - j, seg, (which ? G * D : 0) + qh * D + c);
          y[i] = silu_f(acc);
          ss += y[i] * y[i];
        } else {
          y[i] = silu_f(__bfloat162float(proj[(r0 + t) * a.ldp + seg]));
        }
      }
    }
    float f = 1.f;
    if (DELTA) {
      f = 1.f / sqrtf(warp_sum(ss) + 1e-6f);
      if (!which) f *= 1.f / sqrtf((float)D);
    }
#pragma unroll
    for (int i = 0; i < DP / 32; i++) dst[i * 32 + lane] = y[i] * f;
  }
  if (DELTA) {
    const float rate = expf(a.a_log[h]) * LOG2E;
    for (int i = tid; i < C * DP; i += LOCAL_THREADS) {
      const int t = i / DP, d = i % DP;
      sl[t * ST + d] = t < n && d < D ? -rate * softplus_f(a.graw[(r0 + t) * ((long long)H * D) + (long long)h * D + d] + a.dt_bias[h * D + d]) : 0.f;
    }
    __syncthreads();
    if (tid < DP) {
      float acc = 0.f;
      for (int t = 0; t < C; t++) { acc += sl[t * ST + tid]; sl[t * ST + tid] = acc; }
    }
    __syncthreads();
    for (int i = tid; i < C * DP; i += LOCAL_THREADS) {
      const int t = i / DP, d = i % DP, first = t & ~15;
      const float ref = first ? sl[(first - 1) * ST + d] : 0.f;
      const float x = sl[t * ST + d] - ref;
      sf[t * ST + d] = fast_exp2(x);
      if ((t & 15) == 15 && x < -RANGE) slow[t >> 4] = 1;
    }
  }
  __syncthreads();
  // A and B: 20 tasks (block of 16 rows, 8 columns), both matrices share the right operand
  for (int task = warp; task < 20; task += LOCAL_WARPS) {
    const int I = task < 2 ? 0 : task < 6 ? 1 : task < 12 ? 2 : 3;
    const int j0 = (task - I * (I + 1)) * 8;                    // first column
    const int g = lane >> 2, c2 = 2 * (lane & 3);
    if (DELTA && j0 >= 16 * I && slow[I]) continue;             // pair by pair below
    float aA[3][4] = {}, aB[3][4] = {};
    const int j = j0 + g, ra = 16 * I + g;
    for (int k0 = 0; k0 < DP; k0 += 16) {
      float2 r[2];
#pragma unroll
      for (int e = 0; e < 2; e++) {
        const int d = k0 + e * 8 + c2;
        r[e] = *reinterpret_cast<const float2*>(&sk[j * ST + d]);
        if (DELTA) {
          const float2 l = *reinterpret_cast<const float2*>(&sl[j * ST + d]);
          const float2 ref = I ? *reinterpret_cast<const float2*>(&sl[(16 * I - 1) * ST + d]) : make_float2(0.f, 0.f);
          r[e].x *= fast_exp2(ref.x - l.x); r[e].y *= fast_exp2(ref.y - l.y);
        }
      }
      uint32_t bh[2], bl[2];
      split2(r[0].x, r[0].y, bh[0], bl[0]); split2(r[1].x, r[1].y, bh[1], bl[1]);
      uint32_t kh[4], kl[4], qh_[4], ql[4];
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const int at = (ra + (e & 1) * 8) * ST + k0 + (e >> 1) * 8 + c2;
        float2 q = *reinterpret_cast<const float2*>(&sq[at]);
        if (DELTA) {
          const float2 f = *reinterpret_cast<const float2*>(&sf[at]);
          float2 k = *reinterpret_cast<const float2*>(&sk[at]);
          split2(k.x * f.x, k.y * f.y, kh[e], kl[e]);
          q.x *= f.x; q.y *= f.y;
        }
        split2(q.x, q.y, qh_[e], ql[e]);
      }
      if (DELTA) { mma(aA[0], kh, bh[0], bh[1]); mma(aA[1], kh, bl[0], bl[1]); mma(aA[2], kl, bh[0], bh[1]); }
      mma(aB[0], qh_, bh[0], bh[1]); mma(aB[1], qh_, bl[0], bl[1]); mma(aB[2], ql, bh[0], bh[1]);
    }
#pragma unroll
    for (int e = 0; e < 4; e++) {
      const int t = ra + (e >> 1) * 8, jj = j0 + c2 + (e & 1);
      const float vb = aB[0][e] + (aB[1][e] + aB[2][e]);
      if (DELTA) {
        const float va = aA[0][e] + (aA[1][e] + aA[2][e]);
        sA[t * AT + jj] = jj < t ? va * pw[t] : 0.f;
        sB[t * AT + jj] = jj <= t ? vb : 0.f;
      } else {
        sB[t * AT + jj] = jj <= t ? vb * pw[t - jj] : 0.f;
      }
    }
  }
  for (int i = tid; i < C * C; i += LOCAL_THREADS) {            // right of the diagonal blocks
    const int t = i / C, j = i % C;
    if (j >= (t & ~15) + 16) { sB[t * AT + j] = 0.f; if (DELTA) { sA[t * AT + j] = 0.f; sX[t * AT + j] = 0.f; } }
  }
  if (DELTA) {
    for (int I = 0; I < 4; I++) {
      if (!slow[I]) continue;
      for (int i = tid; i < 256; i += LOCAL_THREADS) {
        const int t = 16 * I + i / 16, j = 16 * I + i % 16;
        float va = 0.f, vb = 0.f;
        if (j <= t)
          for (int d = 0; d < D; d++) {
            const float f = sk[j * ST + d] * fast_exp2(sl[t * ST + d] - sl[j * ST + d]);
            va = fmaf(sk[t * ST + d], f, va); vb = fmaf(sq[t * ST + d], f, vb);
          }
        sA[t * AT + j] = j < t ? va * pw[t] : 0.f;
        sB[t * AT + j] = vb;
      }
    }
  }
  __syncthreads();
  // Q~, K^, B and Gamma_C leave; K~ replaces sf
  {
    bf16* tq = reinterpret_cast<bf16*>(item + Item<DP>::Q);
    bf16* tk = reinterpret_cast<bf16*>(item + Item<DP>::K);
    for (int i = tid; i < C * DP / 2; i += LOCAL_THREADS) {
      const int t = i / (DP / 2), d = i % (DP / 2) * 2, at = t * ST + d, o = swz(t, d, DP);
      float2 q = *reinterpret_cast<const float2*>(&sq[at]), k = *reinterpret_cast<const float2*>(&sk[at]);
      if (DELTA) {
        const float2 l = *reinterpret_cast<const float2*>(&sl[at]), lc = *reinterpret_cast<const float2*>(&sl[(C - 1) * ST + d]);
        const int first = t & ~15;
        const float2 ref = first ? *reinterpret_cast<const float2*>(&sl[(first - 1) * ST + d]) : make_float2(0.f, 0.f);
        float2 f = *reinterpret_cast<const float2*>(&sf[at]);
        f.x *= fast_exp2(ref.x); f.y *= fast_exp2(ref.y);      // Gamma_t
        q.x *= f.x; q.y *= f.y;
        *reinterpret_cast<float2*>(&sf[at]) = make_float2(k.x * f.x, k.y * f.y);
        k.x *= fast_exp2(lc.x - l.x); k.y *= fast_exp2(lc.y - l.y);
      } else {
        q.x *= pw[t + 1]; q.y *= pw[t + 1];
        const float f = t < n ? pw[n - 1 - t] : 0.f;
        k.x *= f; k.y *= f;
      }
      uint32_t hi, lo;
      split2(q.x, q.y, hi, lo);
      *reinterpret_cast<uint32_t*>(tq + o) = hi; *reinterpret_cast<uint32_t*>(tq + C * DP + o) = lo;
      split2(k.x, k.y, hi, lo);
      *reinterpret_cast<uint32_t*>(tk + o) = hi; *reinterpret_cast<uint32_t*>(tk + C * DP + o) = lo;
    }
    bf16* tb = reinterpret_cast<bf16*>(item + Item<DP>::B);
    for (int i = tid; i < C * C / 2; i += LOCAL_THREADS) {
      const int t = i / (C / 2), j = i % (C / 2) * 2, o = swz(t, j, C);
      uint32_t hi, lo;
      split2(sB[t * AT + j], sB[t * AT + j + 1], hi, lo);
      *reinterpret_cast<uint32_t*>(tb + o) = hi; *reinterpret_cast<uint32_t*>(tb + C * C + o) = lo;
    }
    float* tg = reinterpret_cast<float*>(item + Item<DP>::G);
    if (tid < DP) tg[tid] = DELTA ? fast_exp2(sl[(C - 1) * ST + tid]) : pw[n];
  }
  float* tu = reinterpret_cast<float*>(item + Item<DP>::U);
  if (!DELTA) {
    const int EP = (E + 15) / 16 * 16;
    for (int i = tid; i < C * EP; i += LOCAL_THREADS) {
      const int t = i / EP, e = i % EP;
      tu[((e >> 4) * C + t) * 16 + (e & 15)] = t < n && e < E ? silu_f(__bfloat162float(proj[(r0 + t) * a.ldp + a.s_v + h * E + e])) : 0.f;
    }
    return;
  }
  __syncthreads();
  // v into sl (E <= 128 <= ST only when DP = 128: rows of 136 floats either way)
  constexpr int VT = 136;
  float* sv = sl;      // [64][VT]: with DP = 64 it runs on over sf's first half, which is saved in sq first
  float* kt = sf;
  if (DP < 128) {
    for (int i = tid; i < C * ST; i += LOCAL_THREADS) sq[i] = sf[i];
    kt = sq;
    __syncthreads();
  }
  for (int it = warp; it < C; it += LOCAL_WARPS)
    for (int e = lane; e < 128; e += 32) {
      float acc = 0.f;
      if (it < n && e < E) {
        for (int j = 0; j < a.taps; j++) acc += cw[(2 * MAX_TAPS + j) * 128 + e] * input(it, keep - j, a.s_v + h * E + e, 2 * G * D + h * E + e);
        acc = __bfloat162float(__float2bfloat16_rn(silu_f(acc)));
      }
      sv[it * VT + e] = acc;
    }
  // inverse of I + diag(beta) A: the four 16 x 16 diagonal blocks, then the blocks below them by distance
  if (warp < 4 && lane < 16) {
    const float* m = sA + (16 * warp) * AT + 16 * warp;
    float x[16];
#pragma unroll
    for (int r = 0; r < 16; r++) {
      float acc = r == lane ? 1.f : 0.f;
#pragma unroll
      for (int j = 0; j < r; j++) acc = fmaf(-m[r * AT + j], x[j], acc);
      x[r] = acc;
      sX[(16 * warp + r) * AT + 16 * warp + lane] = acc;
    }
  }
  __syncthreads();
  for (int dist = 1; dist < 4; dist++) {
    // Y_IJ = sum_K M_IK X_KJ goes to the free block (J, I) of sA; X_IJ = -X_II Y_IJ
    for (int i = tid; i < (4 - dist) * 256; i += LOCAL_THREADS) {
      const int J = i / 256, I = J + dist, r = i % 256 / 16, c = i % 16;
      float y = 0.f;
      for (int k = 16 * J; k < 16 * I; k++) y = fmaf(sA[(16 * I + r) * AT + k], sX[k * AT + 16 * J + c], y);
      sA[(16 * J + r) * AT + 16 * I + c] = y;
    }
    __syncthreads();
    for (int i = tid; i < (4 - dist) * 256; i += LOCAL_THREADS) {
      const int J = i / 256, I = J + dist, r = i % 256 / 16, c = i % 16;
      float x = 0.f;
#pragma unroll
      for (int k = 0; k < 16; k++) x = fmaf(sX[(16 * I + r) * AT + 16 * I + k], sA[(16 * J + k) * AT + 16 * I + c], x);
      sX[(16 * I + r) * AT + 16 * J + c] = -x;
    }
    __syncthreads();
  }
  for (int i = tid; i < C * C; i += LOCAL_THREADS) sX[i / C * AT + i % C] *= pw[i % C];
  __syncthreads();
  // W = X K~ and U_0 = X V: one task per 8 columns
  const int wt = DP / 8, ut = (E + 15) / 16 * 2;
  bf16* tw = reinterpret_cast<bf16*>(item + Item<DP>::W);
  for (int task = warp; task < wt + ut; task += LOCAL_WARPS) {
    const bool is_w = task < wt;
    const float* src = is_w ? kt : sv;
    const int ld = is_w ? ST : VT, n0 = (is_w ? task : task - wt) * 8, g = lane >> 2, c2 = 2 * (lane & 3);
    float acc[4][4] = {}, low[4][4] = {};
#pragma unroll
    for (int kk = 0; kk < 4; kk++) {
      uint32_t bh[2], bl[2];
#pragma unroll
      for (int e = 0; e < 2; e++) {
        const int k = 16 * kk + 8 * e + c2;
        split2(src[k * ld + n0 + g], src[(k + 1) * ld + n0 + g], bh[e], bl[e]);
      }
#pragma unroll
      for (int m = kk; m < 4; m++) {
        uint32_t ah[4], al[4];
#pragma unroll
        for (int e = 0; e < 4; e++) {
          const float2 x = *reinterpret_cast<const float2*>(&sX[(16 * m + g + (e & 1) * 8) * AT + 16 * kk + (e >> 1) * 8 + c2]);
          split2(x.x, x.y, ah[e], al[e]);
        }
        mma(acc[m], ah, bh[0], bh[1]);
        mma(low[m], al, bh[0], bh[1]);
        if (is_w) mma(low[m], ah, bl[0], bl[1]);     // v is a bf16 number
      }
    }
#pragma unroll
    for (int m = 0; m < 4; m++)
#pragma unroll
      for (int e = 0; e < 2; e++) {
        const int t = 16 * m + g + 8 * e, d = n0 + c2;
        const float x = acc[m][2 * e] + low[m][2 * e], y = acc[m][2 * e + 1] + low[m][2 * e + 1];
        if (is_w) {
          uint32_t hi, lo;
          split2(x, y, hi, lo);
          const int o = swz(t, d, DP);
          *reinterpret_cast<uint32_t*>(tw + o) = hi; *reinterpret_cast<uint32_t*>(tw + C * DP + o) = lo;
        } else {
          *reinterpret_cast<float2*>(&tu[((d >> 4) * C + t) * 16 + (d & 15)]) = make_float2(x, y);
        }
      }
  }
}

// ---- scan over the chunks -----------------------------------------------------------------------------------------------
// One block: 16 columns of one head's state.  Warp w computes U and O of tokens 8w .. 8w+7 and owns 1/8 of the state's rows.
template <int DP, bool DELTA>
__global__ void __launch_bounds__(SCAN_THREADS, 1) k_chunk_scan(const ChunkArgs a) {
  pdl_trigger();
  typedef Item<DP> It;
  constexpr int NT = DP / 64;                  // 8-column tiles of the state's rows per warp
  constexpr size_t X0 = DELTA ? 0 : It::Q, XB = It::X_BYTES - X0;      // without A there is no W
  constexpr size_t UB = (size_t)C * 16 * 4, XS = XB + UB;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 127) & ~(uintptr_t)127);
  uint8_t* sx = smem;                          // 2 stages of [W, Q~ | U_0 slice]
  uint8_t* sy = sx + 2 * XS;                   // [K^, B, Gamma_C]
  bf16* sS = reinterpret_cast<bf16*>(sy + It::Y_BYTES);      // state^T [16][DP], high and low
  bf16* sU = sS + 2 * 16 * DP;                 // U^T [16][64], high and low
  uint64_t* bars = reinterpret_cast<uint64_t*>(sU + 2 * 16 * C);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(bars + 3);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c2 = 2 * (lane & 3);
  const int eb = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const int D = a.dim, E = a.vdim, H = a.heads;
  const char* items = a.ws + ((long long)b * H + h) * a.chunks * a.item_bytes;
  if (threadIdx.x == 0) {
    for (int i = 0; i < 3; i++) mbar_init(&bars[i], 1);
    *abort_flag = 0;
    fence_barrier_init();
  }
  __syncthreads();
  auto load_x = [&](int c) {
    const char* it = items + (long long)c * a.item_bytes;
    uint8_t* dst = sx + (c & 1) * XS;
    mbar_expect_tx(&bars[c & 1], (uint32_t)XS);
    bulk_load_1d(dst, it + X0, (uint32_t)XB, &bars[c & 1]);
    bulk_load_1d(dst + XB, it + It::U + eb * UB, (uint32_t)UB, &bars[c & 1]);
  };
  auto load_y = [&](int c) {
    mbar_expect_tx(&bars[2], (uint32_t)It::Y_BYTES);
    bulk_load_1d(sy, items + (long long)c * a.item_bytes + It::K, (uint32_t)It::Y_BYTES, &bars[2]);
  };
  if (threadIdx.x == 0) {
    load_x(0);
    load_y(0);
    if (a.chunks > 1) load_x(1);
  }
  // the state: rows d0 .. of column e in accumulator fragments, and its two bf16 parts in shared memory
  const int d0 = warp * 8 * NT;
  float S[NT][4];
  auto publish = [&]() {
#pragma unroll
    for (int i = 0; i < NT; i++)
#pragma unroll
      for (int e = 0; e < 2; e++) {
        uint32_t hi, lo;
        split2(S[i][2 * e], S[i][2 * e + 1], hi, lo);
        const int o = swz(g + 8 * e, d0 + 8 * i + c2, DP);
        *reinterpret_cast<uint32_t*>(sS + o) = hi; *reinterpret_cast<uint32_t*>(sS + 16 * DP + o) = lo;
      }
  };
  auto state_at = [&](int e, int d) { return a.S + (((long long)b * H + h) * E + e) * D + d; };
#pragma unroll
  for (int i = 0; i < NT; i++)
#pragma unroll
    for (int e = 0; e < 4; e++) {
      const int col = eb * 16 + g + 8 * (e >> 1), d = d0 + 8 * i + c2 + (e & 1);
      S[i][e] = col < E && d < D ? *state_at(col, d) : 0.f;
    }
  publish();
  bool ok = true;
  int c = 0;
  for (; c < a.chunks; c++) {
    if (!mbar_wait(&bars[c & 1], (c >> 1) & 1, abort_flag, a.status)) ok = false;
    if (!__syncthreads_and(ok)) break;         // also: the published state is complete
    const uint8_t* x = sx + (c & 1) * XS;
    const bf16* tw = reinterpret_cast<const bf16*>(x);
    const bf16* tq = reinterpret_cast<const bf16*>(x + (It::Q - X0));
    const float* u0 = reinterpret_cast<const float*>(x + XB);
    float u[3][4] = {}, o[3][4] = {};
#pragma unroll
    for (int k0 = 0; k0 < DP; k0 += 32) {
      // operand rows are tokens 8 warp + 0..7, four 8-channel units (two k steps) per load
      const int at = swz(8 * warp + (lane & 7), k0 + 8 * (lane >> 3), DP);
      uint32_t wh[4], wl[4], qh[4], ql[4];
      if (DELTA) { ldsm4(wh, tw + at); ldsm4(wl, tw + C * DP + at); }
      ldsm4(qh, tq + at); ldsm4(ql, tq + C * DP + at);
#pragma unroll
      for (int k = 0; k < 2; k++) {
        uint32_t sh[4], sl[4];
        const int as = swz(lane & 15, k0 + 16 * k + 8 * (lane >> 4), DP);
        ldsm4(sh, sS + as); ldsm4(sl, sS + 16 * DP + as);
        if (DELTA) { mma(u[0], sh, wh[2 * k], wh[2 * k + 1]); mma(u[1], sh, wl[2 * k], wl[2 * k + 1]); mma(u[2], sl, wh[2 * k], wh[2 * k + 1]); }
        mma(o[0], sh, qh[2 * k], qh[2 * k + 1]); mma(o[1], sh, ql[2 * k], ql[2 * k + 1]); mma(o[2], sl, qh[2 * k], qh[2 * k + 1]);
      }
    }
#pragma unroll
    for (int e = 0; e < 2; e++) {
      float v[2];
#pragma unroll
      for (int i = 0; i < 2; i++) v[i] = u0[(8 * warp + c2 + i) * 16 + g + 8 * e] - (DELTA ? u[0][2 * e + i] + (u[1][2 * e + i] + u[2][2 * e + i]) : 0.f);
      uint32_t hi, lo;
      split2(v[0], v[1], hi, lo);
      const int at = swz(g + 8 * e, 8 * warp + c2, C);
      *reinterpret_cast<uint32_t*>(sU + at) = hi; *reinterpret_cast<uint32_t*>(sU + 16 * C + at) = lo;
    }
    if (!mbar_wait(&bars[2], c & 1, abort_flag, a.status)) ok = false;
    if (!__syncthreads_and(ok)) break;         // U is complete, this chunk's W, Q~ and the old state have been read
    if (threadIdx.x == 0 && c + 2 < a.chunks) load_x(c + 2);
    const bf16* tk = reinterpret_cast<const bf16*>(sy);
    const bf16* tb = reinterpret_cast<const bf16*>(sy + (It::B - It::K));
    const float* gam = reinterpret_cast<const float*>(sy + (It::G - It::K));
    uint32_t uh[4][4], ul[4][4];
#pragma unroll
    for (int k = 0; k < 4; k++) {
      const int at = swz(lane & 15, 16 * k + 8 * (lane >> 4), C);
      ldsm4(uh[k], sU + at); ldsm4(ul[k], sU + 16 * C + at);
    }
    float low[NT][4] = {};
#pragma unroll
    for (int i = 0; i < NT; i++)
#pragma unroll
      for (int e = 0; e < 4; e++) S[i][e] *= gam[d0 + 8 * i + c2 + (e & 1)];
#pragma unroll
    for (int k = 0; k < 4; k += 2) {
      uint32_t bh[4], bl[4];
      if (16 * k <= 8 * warp + 7) {            // later tokens do not reach these
        const int at = swz(8 * warp + (lane & 7), 16 * k + 8 * (lane >> 3), C);
        ldsm4(bh, tb + at); ldsm4(bl, tb + C * C + at);
#pragma unroll
        for (int i = 0; i < 2; i++) {
          mma(o[0], uh[k + i], bh[2 * i], bh[2 * i + 1]); mma(o[1], uh[k + i], bl[2 * i], bl[2 * i + 1]); mma(o[2], ul[k + i], bh[2 * i], bh[2 * i + 1]);
        }
      }
#pragma unroll
      for (int i = 0; i < 2; i++) {
        uint32_t kh[4], kl[4];
        if (NT == 2) {
          const int at = swz(16 * (k + i) + (lane & 15), d0 + 8 * (lane >> 4), DP);
          ldsm4t(kh, tk + at); ldsm4t(kl, tk + C * DP + at);
        } else {                               // one tile of 8 rows: the second pair of matrices is the low part
          const int at = swz(16 * (k + i) + (lane & 15), d0, DP);
          ldsm4t(kh, tk + (lane >> 4) * (C * DP) + at);
          kl[0] = kh[2]; kl[1] = kh[3];
        }
#pragma unroll
        for (int j = 0; j < NT; j++) {
          mma(S[j], uh[k + i], kh[2 * j], kh[2 * j + 1]);
          mma(low[j], uh[k + i], kl[2 * j], kl[2 * j + 1]); mma(low[j], ul[k + i], kh[2 * j], kh[2 * j + 1]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < NT; i++)
#pragma unroll
      for (int e = 0; e < 4; e++) S[i][e] += low[i][e];
    publish();
    const int t0 = a.t0 + c * C + 8 * warp + c2;
#pragma unroll
    for (int e = 0; e < 4; e++) {
      const int t = t0 + (e & 1), col = eb * 16 + g + 8 * (e >> 1);
      if (t < a.T && col < E)
        reinterpret_cast<bf16*>(a.o)[((long long)b * a.T + t) * ((long long)H * E) + (long long)h * E + col] = __float2bfloat16_rn(o[0][e] + (o[1][e] + o[2][e]));
    }
    __syncthreads();                           // K^, B have been read
    if (threadIdx.x == 0 && c + 1 < a.chunks) load_y(c + 1);
  }
  if (c < a.chunks) {                          // a wait ran out: let the copies in flight land before the block ends
    if (threadIdx.x == 0)
      for (int i = 0; i < 3; i++)
        for (uint32_t it = 0; it < WAIT_LIMIT && !mbar_try_wait(&bars[i], i < 2 ? (((c + ((c ^ i) & 1)) >> 1) & 1) : (c & 1)); ++it) {}
    return;
  }
#pragma unroll
  for (int i = 0; i < NT; i++)
#pragma unroll
    for (int e = 0; e < 4; e++) {
      const int col = eb * 16 + g + 8 * (e >> 1), d = d0 + 8 * i + c2 + (e & 1);
      if (col < E && d < D) *state_at(col, d) = S[i][e];
    }
}

template <int DP, bool DELTA> int run(ChunkArgs a, cudaStream_t s) {
  typedef Item<DP> It;
  const size_t local = 4 * (size_t)((DELTA ? 4 : 3) * C * (DP + 8) + (DELTA ? 3 : 1) * C * (C + 4) + 72 + (DELTA ? 3 * MAX_TAPS * 128 : 0) + 4);
  const size_t x = (DELTA ? It::X_BYTES : It::X_BYTES - It::Q) + (size_t)C * 16 * 4;
  const size_t scan = 2 * x + It::Y_BYTES + 2 * 16 * DP * 2 + 2 * 16 * C * 2 + 64 + 128;
  static PerDevice attr;
  const int dev = PerDevice::current();
  if (dev < 0 || !attr.done[dev]) {
    CUDA_TRY(cudaFuncSetAttribute(k_chunk_local<DP, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)local));
    CUDA_TRY(cudaFuncSetAttribute(k_chunk_scan<DP, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)scan));
    if (dev >= 0) attr.done[dev] = true;
  }
  a.item_bytes = (It::bytes(a.vdim) + 127) / 128 * 128;
  const int total = cdiv(a.T, C);
  const int seg = (int)std::min<long long>(total, (long long)a.ws_bytes / ((long long)a.item_bytes * a.B * a.heads));
  if (seg <= 0) return femto_fail(FEMTO_ERR_NOMEM, "chunked recurrence: workspace too small for %d columns of %d heads", a.B, a.heads);
  for (int c0 = 0; c0 < total; c0 += seg) {
    a.t0 = c0 * C; a.chunks = std::min(seg, total - c0);
    k_chunk_local<DP, DELTA><<<dim3(a.chunks, a.heads, a.B), LOCAL_THREADS, local, s>>>(a);
    KERNEL_CHECK();
    k_chunk_scan<DP, DELTA><<<dim3(cdiv(a.vdim, 16), a.heads, a.B), SCAN_THREADS, scan, s>>>(a);
    KERNEL_CHECK();
  }
  return 0;
}

}  // namespace

size_t chunked_recurrence_item_bytes(int dim, int vdim) { return ((dim <= 64 ? Item<64>::bytes(vdim) : Item<128>::bytes(vdim)) + 127) / 128 * 128; }

bool chunked_recurrence_supported(const ChunkArgs& a) {
  return a.T >= 32 && a.dim <= 128 && a.vdim <= 128 && a.taps <= MAX_TAPS &&
         a.ws_bytes / ((size_t)a.B * a.heads) >= chunked_recurrence_item_bytes(a.dim, a.vdim);
}

int chunked_recurrence(const ChunkArgs& a, cudaStream_t s) {
  const bool delta = a.graw != nullptr;
  if (a.dim <= 64) return delta ? run<64, true>(a, s) : run<64, false>(a, s);
  return delta ? run<128, true>(a, s) : run<128, false>(a, s);
}
