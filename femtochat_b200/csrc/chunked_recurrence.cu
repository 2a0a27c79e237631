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

// (an activation: bf16 numbers go in, so the special-function unit's 2^-21 is plenty)
__device__ __forceinline__ float silu_f(float z) { return z * __fdividef(1.f, 1.f + __expf(-z)); }
// log(1 + e^z) = max(z, 0) + log(1 + x), x = e^-|z| in (0, 1], with log(1 + x) = 2 artanh(s), s = x / (2 + x) <= 1/3: eight terms
// of the artanh series leave a relative error of 3e-9
__device__ __forceinline__ float softplus_f(float z) {
  const float x = expf(-fabsf(z)), s = __fdividef(x, 2.f + x), t = s * s;
  float p = 1.f / 15.f;
  p = fmaf(p, t, 1.f / 13.f); p = fmaf(p, t, 1.f / 11.f); p = fmaf(p, t, 1.f / 9.f); p = fmaf(p, t, 1.f / 7.f);
  p = fmaf(p, t, 1.f / 5.f); p = fmaf(p, t, 1.f / 3.f); p = fmaf(p, t, 1.f);
  return fmaf(2.f * s, p, fmaxf(z, 0.f));
}

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
// eight consecutive channels c .. c + 7 of a row of `size` channels (zeros beyond it)
__device__ __forceinline__ void load8(const bf16* row, int c, int size, bool vec, float (&f)[8]) {
  if (vec) {
    if (c < size) load_vec<bf16, 8>(row + c, f);
    else
#pragma unroll
      for (int e = 0; e < 8; e++) f[e] = 0.f;
  } else {
#pragma unroll
    for (int e = 0; e < 8; e++) f[e] = c + e < size ? __bfloat162float(row[c + e]) : 0.f;
  }
}
__device__ __forceinline__ void split8(const float (&f)[8], uint4& hi, uint4& lo) {
  split2(f[0], f[1], hi.x, lo.x); split2(f[2], f[3], hi.y, lo.y); split2(f[4], f[5], hi.z, lo.z); split2(f[6], f[7], hi.w, lo.w);
}
// Task 0 .. 19 -> block I of 16 rows and first column j0 <= 16 I + 8 of an 8-column tile of the lower triangle
__device__ __forceinline__ void triangle_task(int task, int& I, int& j0) {
  I = task < 2 ? 0 : task < 6 ? 1 : task < 12 ? 2 : 3;
  j0 = (task - I * (I + 1)) * 8;
}
__device__ __forceinline__ void zero_above(bf16* tile, int tid) {      // blocks right of the diagonal blocks, high and low
  for (int i = tid; i < 2 * C * C / 8; i += LOCAL_THREADS) {
    const int part = i / (C * C / 8), t = i % (C * C / 8) / 8, j = i % 8 * 8;
    if (j >= (t & ~15) + 16) *reinterpret_cast<uint4*>(tile + part * C * C + swz(t, j, C)) = make_uint4(0, 0, 0, 0);
  }
}

// Decayed sum: Q~ = decay^(t+1) q, K^ = decay^(n-1-t) k, U_0 = v and B = (q k^T) decay^(t-j).
template <int DP>
__global__ void __launch_bounds__(LOCAL_THREADS) k_chunk_local_sum(const ChunkArgs a) {
  pdl_trigger();
  extern __shared__ __align__(16) uint8_t smem_raw[];
  bf16* tq = reinterpret_cast<bf16*>(smem_raw);    // q, high and low
  bf16* tk = tq + 2 * C * DP;                      // k
  __shared__ float pw[C + 1];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int chunk = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const int D = a.dim, E = a.vdim;
  const int t0 = a.t0 + chunk * C, n = min(C, a.T - t0);
  const bf16* proj = reinterpret_cast<const bf16*>(a.proj) + ((long long)b * a.T + t0) * a.ldp;
  char* item = a.ws + (((long long)b * a.heads + h) * gridDim.x + chunk) * a.item_bytes;
  if (tid <= C) pw[tid] = powf(a.decay[h], (float)tid);
  __syncthreads();
  const bool vec = (((D | E) & 7) == 0) && (a.ldp & 7) == 0;
  bf16* gq = reinterpret_cast<bf16*>(item + Item<DP>::Q);
  bf16* gk = reinterpret_cast<bf16*>(item + Item<DP>::K);
  for (int i = tid; i < 2 * C * (DP / 8); i += LOCAL_THREADS) {
    const int which = i / (C * (DP / 8)), t = i / (DP / 8) % C, c = i % (DP / 8) * 8, o = swz(t, c, DP);
    float f[8] = {};
    if (t < n) load8(proj + t * a.ldp + (which ? a.s_k : a.s_q) + h * D, c, D, vec, f);
#pragma unroll
    for (int e = 0; e < 8; e++) f[e] = silu_f(f[e]);
    uint4 hi, lo;
    split8(f, hi, lo);
    bf16* st = which ? tk : tq;
    *reinterpret_cast<uint4*>(st + o) = hi; *reinterpret_cast<uint4*>(st + C * DP + o) = lo;
    const float p = which ? (t < n ? pw[n - 1 - t] : 0.f) : pw[t + 1];
#pragma unroll
    for (int e = 0; e < 8; e++) f[e] *= p;
    split8(f, hi, lo);
    bf16* gt = which ? gk : gq;
    *reinterpret_cast<uint4*>(gt + o) = hi; *reinterpret_cast<uint4*>(gt + C * DP + o) = lo;
  }
  float* tu = reinterpret_cast<float*>(item + Item<DP>::U);
  const int EP8 = (E + 15) / 16 * 2;
  for (int i = tid; i < C * EP8; i += LOCAL_THREADS) {
    const int t = i / EP8, e = i % EP8 * 8;
    float f[8] = {};
    if (t < n) load8(proj + t * a.ldp + a.s_v + h * E, e, E, vec, f);
    float* dst = tu + ((e >> 4) * C + t) * 16 + (e & 15);
    *reinterpret_cast<float4*>(dst) = make_float4(silu_f(f[0]), silu_f(f[1]), silu_f(f[2]), silu_f(f[3]));
    *reinterpret_cast<float4*>(dst + 4) = make_float4(silu_f(f[4]), silu_f(f[5]), silu_f(f[6]), silu_f(f[7]));
  }
  if (tid < DP) reinterpret_cast<float*>(item + Item<DP>::G)[tid] = pw[n];
  bf16* tb = reinterpret_cast<bf16*>(item + Item<DP>::B);
  zero_above(tb, tid);
  __syncthreads();
  for (int task = warp; task < 20; task += LOCAL_WARPS) {
    int I, j0;
    triangle_task(task, I, j0);
    float acc[3][4] = {};
#pragma unroll
    for (int k0 = 0; k0 < DP; k0 += 32) {
      uint32_t bh[4], bl[4];
      const int at = swz(j0 + (lane & 7), k0 + 8 * (lane >> 3), DP);
      ldsm4(bh, tk + at); ldsm4(bl, tk + C * DP + at);
#pragma unroll
      for (int k = 0; k < 2; k++) {
        uint32_t ah[4], al[4];
        const int aa = swz(16 * I + (lane & 15), k0 + 16 * k + 8 * (lane >> 4), DP);
        ldsm4(ah, tq + aa); ldsm4(al, tq + C * DP + aa);
        mma(acc[0], ah, bh[2 * k], bh[2 * k + 1]); mma(acc[1], ah, bl[2 * k], bl[2 * k + 1]); mma(acc[2], al, bh[2 * k], bh[2 * k + 1]);
      }
    }
#pragma unroll
    for (int e = 0; e < 2; e++) {
      const int t = 16 * I + (lane >> 2) + 8 * e, j = j0 + 2 * (lane & 3);
      const float x = j <= t ? (acc[0][2 * e] + (acc[1][2 * e] + acc[2][2 * e])) * pw[t - j] : 0.f;
      const float y = j + 1 <= t ? (acc[0][2 * e + 1] + (acc[1][2 * e + 1] + acc[2][2 * e + 1])) * pw[t - j - 1] : 0.f;
      uint32_t hi, lo;
      split2(x, y, hi, lo);
      const int o = swz(t, j, C);
      *reinterpret_cast<uint32_t*>(tb + o) = hi; *reinterpret_cast<uint32_t*>(tb + C * C + o) = lo;
    }
  }
}

// d (16 x 8) += A (16 x 16) B (16 x 8), both fp32 in shared memory with pitch ld; by one warp
__device__ __forceinline__ void block_product(float (&d)[4], const float* A, const float* B, int ld, int lane) {
  const int g = lane >> 2, c2 = 2 * (lane & 3);
  uint32_t ah[4], al[4], bh[2], bl[2];
#pragma unroll
  for (int e = 0; e < 4; e++) {
    const float2 x = *reinterpret_cast<const float2*>(&A[(g + (e & 1) * 8) * ld + (e >> 1) * 8 + c2]);
    split2(x.x, x.y, ah[e], al[e]);
  }
#pragma unroll
  for (int e = 0; e < 2; e++) split2(B[(8 * e + c2) * ld + g], B[(8 * e + c2 + 1) * ld + g], bh[e], bl[e]);
  mma(d, ah, bl[0], bl[1]); mma(d, al, bh[0], bh[1]); mma(d, ah, bh[0], bh[1]);
}

// Gated delta rule.  The raw inputs of the convolutions lie where the scaled operands and the small matrices go once the
// convolutions are done.
template <int DP> struct DeltaSmem {      // offsets in bytes
  static constexpr int ST = DP + 8, AT = C + 4, ROWS = C + MAX_TAPS - 1;
  static constexpr int K = 0, Q = K + C * ST * 4, L = Q + C * ST * 4, KF = L + C * ST * 4, QF = KF + 4 * C * DP, A = QF + 4 * C * DP,
                       X = A + C * AT * 4, V = X + C * AT * 4, CW = V + C * 128 * 2, BETA = CW + 3 * 128 * 16, SLOW = BETA + C * 4, TOTAL = SLOW + 16;
  static constexpr int RAW = KF;           // bf16 [3][ROWS][128]
  static_assert(3 * ROWS * 128 * 2 <= V - RAW, "raw inputs overlap what is live");
};

template <int DP>
__global__ void __launch_bounds__(LOCAL_THREADS, 1) k_chunk_local_delta(const ChunkArgs a) {
  pdl_trigger();
  typedef DeltaSmem<DP> Sm;
  constexpr int ST = Sm::ST, AT = Sm::AT;
  extern __shared__ __align__(16) uint8_t smem_raw[];
  float* sk = reinterpret_cast<float*>(smem_raw + Sm::K);    // [64][ST] k
  float* sq = reinterpret_cast<float*>(smem_raw + Sm::Q);    // [64][ST] q
  float* sl = reinterpret_cast<float*>(smem_raw + Sm::L);    // [64][ST] cumulated log2 decays
  bf16* kf = reinterpret_cast<bf16*>(smem_raw + Sm::KF);     // k times 2^(L_t - L at the block's start), high and low; later K~
  bf16* qf = reinterpret_cast<bf16*>(smem_raw + Sm::QF);     // q likewise
  float* sA = reinterpret_cast<float*>(smem_raw + Sm::A);    // [64][AT] diag(beta) A, then scratch of the inverse
  bf16* xs = reinterpret_cast<bf16*>(smem_raw + Sm::A);      // at the end: the inverse times diag(beta), high and low
  float* sX = reinterpret_cast<float*>(smem_raw + Sm::X);    // [64][AT] the inverse
  bf16* sv = reinterpret_cast<bf16*>(smem_raw + Sm::V);      // v [64][128]
  float4* cw = reinterpret_cast<float4*>(smem_raw + Sm::CW); // [3][128] first four taps of every channel
  float* beta = reinterpret_cast<float*>(smem_raw + Sm::BETA);
  int* slow = reinterpret_cast<int*>(smem_raw + Sm::SLOW);   // [4]
  bf16* raw = reinterpret_cast<bf16*>(smem_raw + Sm::RAW);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int chunk = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const int D = a.dim, E = a.vdim, H = a.heads, qh = h / (H / a.qk_heads);
  const int t0 = a.t0 + chunk * C, n = min(C, a.T - t0);
  const long long r0 = (long long)b * a.T + t0;
  char* item = a.ws + (((long long)b * H + h) * gridDim.x + chunk) * a.item_bytes;
  const bf16* proj = reinterpret_cast<const bf16*>(a.proj);
  const int G = a.qk_heads, channels = 2 * G * D + H * E, keep = a.taps - 1;
  const bf16* tail = reinterpret_cast<const bf16*>(a.tail_in) + (long long)b * keep * channels;
  // decay logits of this chunk, on their way while the rest is staged: thread -> 4 channels of a token
  constexpr int GV = C * DP / 4 / LOCAL_THREADS;
  float4 graw[GV];
#pragma unroll
  for (int i = 0; i < GV; i++) {
    const int t = (i * LOCAL_THREADS + tid) / (DP / 4), d = (i * LOCAL_THREADS + tid) % (DP / 4) * 4;
    const float* src = a.graw + (r0 + t) * ((long long)H * D) + (long long)h * D + d;
    graw[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (t < n) {
      if ((D & 3) == 0) { if (d < D) graw[i] = *reinterpret_cast<const float4*>(src); }
      else { if (d < D) graw[i].x = src[0]; if (d + 1 < D) graw[i].y = src[1]; if (d + 2 < D) graw[i].z = src[2]; if (d + 3 < D) graw[i].w = src[3]; }
    }
  }
  // raw rows -keep .. 63 of q, k and v: from this call's projections or from the inputs kept of earlier calls
  const int rows = C + keep;
  auto source = [&](int which, int r) -> const bf16* {
    const int t = t0 + r - keep;
    const int head = which == 2 ? h * E : qh * D;
    if (t >= 0) return proj + (r0 + r - keep) * a.ldp + (which == 0 ? a.s_q : which == 1 ? a.s_k : a.s_v) + head;
    return tail + (long long)(keep + t) * channels + (which == 0 ? 0 : which == 1 ? G * D : 2 * G * D) + head;
  };
  if (((D | E) & 7) == 0 && (a.ldp & 7) == 0) {
    const int c = tid % 16 * 8;
#pragma unroll
    for (int which = 0; which < 3; which++)
#pragma unroll
      for (int i = 0; i < 3; i++) {
        const int r = tid / 16 + i * (LOCAL_THREADS / 16);
        if (r >= rows) break;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (r < n + keep && c < (which == 2 ? E : D)) v = *reinterpret_cast<const uint4*>(source(which, r) + c);
        *reinterpret_cast<uint4*>(raw + (which * Sm::ROWS + r) * 128 + c) = v;
      }
  } else {
    for (int i = tid; i < 3 * rows * 128; i += LOCAL_THREADS) {
      const int which = i / (rows * 128), r = i / 128 % rows, c = i % 128;
      raw[(which * Sm::ROWS + r) * 128 + c] = r < n + keep && c < (which == 2 ? E : D) ? source(which, r)[c] : __float2bfloat16_rn(0.f);
    }
  }
  if (tid < 3 * 128) {
    const int which = tid / 128, c = tid % 128;
    const float* src = which == 0 ? a.conv_q : which == 1 ? a.conv_k : a.conv_v;
    float w[4] = {};
    if (c < (which == 2 ? E : D)) {
      src += (long long)((which == 2 ? h * E : qh * D) + c) * a.taps;
#pragma unroll
      for (int j = 0; j < 4; j++) if (j < a.taps) w[j] = src[j];
    }
    cw[tid] = make_float4(w[0], w[1], w[2], w[3]);
  }
  if (tid < C) beta[tid] = tid < n ? 1.f / (1.f + expf(-__bfloat162float(proj[(r0 + tid) * a.ldp + a.s_b + h]))) : 0.f;
  if (tid < 4) slow[tid] = 0;
  const float rate = expf(a.a_log[h]) * LOG2E;
#pragma unroll
  for (int i = 0; i < GV; i++) {
    const int t = (i * LOCAL_THREADS + tid) / (DP / 4), d = (i * LOCAL_THREADS + tid) % (DP / 4) * 4;
    float x[4] = {graw[i].x, graw[i].y, graw[i].z, graw[i].w};
#pragma unroll
    for (int e = 0; e < 4; e++) x[e] = t < n && d + e < D ? -rate * softplus_f(x[e] + a.dt_bias[h * D + d + e]) : 0.f;
    *reinterpret_cast<float4*>(&sl[t * ST + d]) = make_float4(x[0], x[1], x[2], x[3]);
  }
  __syncthreads();
  // convolution, silu, unit vectors: a warp takes four consecutive tokens of q, then of k, then of v; a lane two pairs of channels
  const int tb0 = 4 * warp;
  const float q_scale = rsqrtf((float)D);
#pragma unroll 1
  for (int which = 0; which < 3; which++) {
    float x[7][4];
    float4 w[4];
#pragma unroll
    for (int i = 0; i < 4; i++) w[i] = cw[which * 128 + (i >> 1) * 64 + 2 * lane + (i & 1)];
#pragma unroll
    for (int r = 0; r < 7; r++)
#pragma unroll
      for (int p = 0; p < 2; p++) {
        float2 f = make_float2(0.f, 0.f);
        if (r < 3 + a.taps) f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(raw + (which * Sm::ROWS + tb0 + r) * 128 + p * 64 + 2 * lane));
        x[r][2 * p] = f.x; x[r][2 * p + 1] = f.y;
      }
#pragma unroll
    for (int tt = 0; tt < 4; tt++) {
      const int t = tb0 + tt;
      float y[4], ss = 0.f;
#pragma unroll
      for (int i = 0; i < 4; i++) {
        float acc = w[i].x * x[tt][i];
        acc = fmaf(w[i].y, x[tt + 1][i], acc); acc = fmaf(w[i].z, x[tt + 2][i], acc); acc = fmaf(w[i].w, x[tt + 3][i], acc);
        if (a.taps > 4) {
          const int c = (i >> 1) * 64 + 2 * lane + (i & 1), size = which == 2 ? E : D, head = which == 2 ? h : qh;
          const float* src = which == 0 ? a.conv_q : which == 1 ? a.conv_k : a.conv_v;
          if (c < size)
            for (int j = 4; j < a.taps; j++)
              acc = fmaf(src[(long long)(head * size + c) * a.taps + j], __bfloat162float(raw[(which * Sm::ROWS + t + j) * 128 + c]), acc);
        }
        y[i] = t < n ? silu_f(acc) : 0.f;      // padding channels: zero
        ss += y[i] * y[i];
      }
      if (which == 2) {
#pragma unroll
        for (int p = 0; p < 2; p++) *reinterpret_cast<uint32_t*>(sv + swz(t, p * 64 + 2 * lane, 128)) = bf2(y[2 * p], y[2 * p + 1]);
      } else {
        const float f = rsqrtf(warp_sum(ss) + 1e-6f) * (which ? 1.f : q_scale);
        float* dst = (which ? sk : sq) + t * ST + 2 * lane;
#pragma unroll
        for (int p = 0; p < DP / 64; p++) *reinterpret_cast<float2*>(dst + p * 64) = make_float2(y[2 * p] * f, y[2 * p + 1] * f);
      }
    }
  }
  // cumulated decays: inside each block of 16 tokens, then over the blocks before it
  const int blk = tid / DP, dcol = tid % DP;
  if (blk < 4) {
    float acc = 0.f;
#pragma unroll
    for (int t = 0; t < 16; t++) { acc += sl[(16 * blk + t) * ST + dcol]; sl[(16 * blk + t) * ST + dcol] = acc; }
  }
  __syncthreads();                    // the raw inputs have been read as well
  for (int i = tid; i < C * DP / 2; i += LOCAL_THREADS) {
    const int t = i / (DP / 2), d = i % (DP / 2) * 2, at = t * ST + d, o = swz(t, d, DP);
    const float2 x = *reinterpret_cast<const float2*>(&sl[at]), k = *reinterpret_cast<const float2*>(&sk[at]), q = *reinterpret_cast<const float2*>(&sq[at]);
    const float2 f = make_float2(fast_exp2(x.x), fast_exp2(x.y));
    if ((t & 15) == 15 && fminf(x.x, x.y) < -RANGE) slow[t >> 4] = 1;
    uint32_t hi, lo;
    split2(k.x * f.x, k.y * f.y, hi, lo);
    *reinterpret_cast<uint32_t*>(kf + o) = hi; *reinterpret_cast<uint32_t*>(kf + C * DP + o) = lo;
    split2(q.x * f.x, q.y * f.y, hi, lo);
    *reinterpret_cast<uint32_t*>(qf + o) = hi; *reinterpret_cast<uint32_t*>(qf + C * DP + o) = lo;
  }
  __syncthreads();
  if (blk < 4 && blk > 0) {
    float before = 0.f;
    for (int k = 0; k < blk; k++) before += sl[(16 * k + 15) * ST + dcol];
    // the last row of a block is still its own sum while other threads read it: it is finished below
#pragma unroll
    for (int t = 0; t < 15; t++) sl[(16 * blk + t) * ST + dcol] += before;
  }
  __syncthreads();
  if (tid < DP) {
    float acc = sl[15 * ST + tid];
#pragma unroll
    for (int k = 1; k < 4; k++) { acc += sl[(16 * k + 15) * ST + tid]; sl[(16 * k + 15) * ST + tid] = acc; }
  }
  bf16* tb = reinterpret_cast<bf16*>(item + Item<DP>::B);
  zero_above(tb, tid);
  for (int i = tid; i < C * C; i += LOCAL_THREADS) {            // right of the diagonal blocks
    const int t = i / C, j = i % C;
    if (j >= (t & ~15) + 16) { sA[t * AT + j] = 0.f; sX[t * AT + j] = 0.f; }
  }
  __syncthreads();
  // A and B: both matrices share the right operand, k_j times 2^(L at the row block's start - L_j)
  const int g = lane >> 2, c2 = 2 * (lane & 3);
  for (int task = warp; task < 20; task += LOCAL_WARPS) {
    int I, j0;
    triangle_task(task, I, j0);
    if (j0 >= 16 * I && slow[I]) continue;                      // pair by pair below
    float aA[3][4] = {}, aB[3][4] = {};
    const int j = j0 + g;
    const float* ref = sl + (16 * I - 1) * ST;
#pragma unroll 4
    for (int k0 = 0; k0 < DP; k0 += 16) {
      uint32_t bh[2], bl[2];
#pragma unroll
      for (int e = 0; e < 2; e++) {
        const int d = k0 + e * 8 + c2;
        float2 r = *reinterpret_cast<const float2*>(&sk[j * ST + d]);
        const float2 l = *reinterpret_cast<const float2*>(&sl[j * ST + d]);
        const float2 lr = I ? *reinterpret_cast<const float2*>(ref + d) : make_float2(0.f, 0.f);
        r.x *= fast_exp2(lr.x - l.x); r.y *= fast_exp2(lr.y - l.y);
        split2(r.x, r.y, bh[e], bl[e]);
      }
      uint32_t kh[4], kl[4], qh_[4], ql[4];
      const int aa = swz(16 * I + (lane & 15), k0 + 8 * (lane >> 4), DP);
      ldsm4(kh, kf + aa); ldsm4(kl, kf + C * DP + aa); ldsm4(qh_, qf + aa); ldsm4(ql, qf + C * DP + aa);
      mma(aA[0], kh, bh[0], bh[1]); mma(aA[1], kh, bl[0], bl[1]); mma(aA[2], kl, bh[0], bh[1]);
      mma(aB[0], qh_, bh[0], bh[1]); mma(aB[1], qh_, bl[0], bl[1]); mma(aB[2], ql, bh[0], bh[1]);
    }
#pragma unroll
    for (int e = 0; e < 2; e++) {
      const int t = 16 * I + g + 8 * e, jj = j0 + c2;
      float va[2], vb[2];
#pragma unroll
      for (int i = 0; i < 2; i++) {
        va[i] = jj + i < t ? (aA[0][2 * e + i] + (aA[1][2 * e + i] + aA[2][2 * e + i])) * beta[t] : 0.f;
        vb[i] = jj + i <= t ? aB[0][2 * e + i] + (aB[1][2 * e + i] + aB[2][2 * e + i]) : 0.f;
      }
      *reinterpret_cast<float2*>(&sA[t * AT + jj]) = make_float2(va[0], va[1]);
      uint32_t hi, lo;
      split2(vb[0], vb[1], hi, lo);
      const int o = swz(t, jj, C);
      *reinterpret_cast<uint32_t*>(tb + o) = hi; *reinterpret_cast<uint32_t*>(tb + C * C + o) = lo;
    }
  }
  for (int I = 0; I < 4; I++) {
    if (!slow[I]) continue;
    for (int i = tid; i < 256; i += LOCAL_THREADS) {
      const int t = 16 * I + i / 16, j = 16 * I + i % 16, o = swz(t, j, C);
      float va = 0.f, vb = 0.f;
      if (j <= t)
        for (int d = 0; d < D; d++) {
          const float f = sk[j * ST + d] * fast_exp2(sl[t * ST + d] - sl[j * ST + d]);
          va = fmaf(sk[t * ST + d], f, va); vb = fmaf(sq[t * ST + d], f, vb);
        }
      sA[t * AT + j] = j < t ? va * beta[t] : 0.f;
      const bf16 hi = __float2bfloat16_rn(vb);
      tb[o] = hi; tb[C * C + o] = __float2bfloat16_rn(vb - __bfloat162float(hi));
    }
  }
  __syncthreads();
  // Q~ and K^ leave; K~ replaces kf
  {
    bf16* tq = reinterpret_cast<bf16*>(item + Item<DP>::Q);
    bf16* tk = reinterpret_cast<bf16*>(item + Item<DP>::K);
    for (int i = tid; i < C * DP / 2; i += LOCAL_THREADS) {
      const int t = i / (DP / 2), d = i % (DP / 2) * 2, at = t * ST + d, o = swz(t, d, DP);
      const float2 q = *reinterpret_cast<const float2*>(&sq[at]), k = *reinterpret_cast<const float2*>(&sk[at]);
      const float2 l = *reinterpret_cast<const float2*>(&sl[at]), lc = *reinterpret_cast<const float2*>(&sl[(C - 1) * ST + d]);
      const float2 f = make_float2(fast_exp2(l.x), fast_exp2(l.y));                       // Gamma_t
      uint32_t hi, lo;
      split2(k.x * f.x, k.y * f.y, hi, lo);
      *reinterpret_cast<uint32_t*>(kf + o) = hi; *reinterpret_cast<uint32_t*>(kf + C * DP + o) = lo;
      split2(q.x * f.x, q.y * f.y, hi, lo);
      *reinterpret_cast<uint32_t*>(tq + o) = hi; *reinterpret_cast<uint32_t*>(tq + C * DP + o) = lo;
      split2(k.x * fast_exp2(lc.x - l.x), k.y * fast_exp2(lc.y - l.y), hi, lo);
      *reinterpret_cast<uint32_t*>(tk + o) = hi; *reinterpret_cast<uint32_t*>(tk + C * DP + o) = lo;
    }
    if (tid < DP) reinterpret_cast<float*>(item + Item<DP>::G)[tid] = fast_exp2(sl[(C - 1) * ST + tid]);
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
  // X_IJ = -X_II sum_K M_IK X_KJ, one warp per (block, half of its columns); the inner sum goes to the free block (J, I) of sA
#pragma unroll
  for (int dist = 1; dist < 4; dist++) {
    const int J = warp >> 1, I = J + dist, nh = (warp & 1) * 8;
    if (I < 4) {
      float y[4] = {};
#pragma unroll
      for (int k = 0; k < dist; k++)
        block_product(y, sA + 16 * I * AT + 16 * (J + k), sX + 16 * (J + k) * AT + 16 * J + nh, AT, lane);
#pragma unroll
      for (int e = 0; e < 2; e++) *reinterpret_cast<float2*>(&sA[(16 * J + g + 8 * e) * AT + 16 * I + nh + c2]) = make_float2(y[2 * e], y[2 * e + 1]);
      __syncwarp();
      float x[4] = {};
      block_product(x, sX + 16 * I * AT + 16 * I, sA + 16 * J * AT + 16 * I + nh, AT, lane);
#pragma unroll
      for (int e = 0; e < 2; e++) *reinterpret_cast<float2*>(&sX[(16 * I + g + 8 * e) * AT + 16 * J + nh + c2]) = make_float2(-x[2 * e], -x[2 * e + 1]);
    }
    __syncthreads();
  }
  for (int i = tid; i < C * C / 2; i += LOCAL_THREADS) {
    const int t = i / (C / 2), j = i % (C / 2) * 2, o = swz(t, j, C);
    const float2 x = *reinterpret_cast<const float2*>(&sX[t * AT + j]);
    uint32_t hi, lo;
    split2(x.x * beta[j], x.y * beta[j + 1], hi, lo);
    *reinterpret_cast<uint32_t*>(xs + o) = hi; *reinterpret_cast<uint32_t*>(xs + C * C + o) = lo;
  }
  __syncthreads();
  // W = X K~ and U_0 = X V: one task per 16 columns
  const int wt = DP / 16, ut = (E + 15) / 16;
  bf16* tw = reinterpret_cast<bf16*>(item + Item<DP>::W);
  float* tu = reinterpret_cast<float*>(item + Item<DP>::U);
  for (int task = warp; task < wt + ut; task += LOCAL_WARPS) {
    const bool is_w = task < wt;
    const int n0 = (is_w ? task : task - wt) * 16;
    float acc[4][2][4] = {}, low[4][2][4] = {};
#pragma unroll
    for (int kk = 0; kk < 4; kk++) {
      uint32_t bh[4], bl[4];
      if (is_w) {
        const int at = swz(16 * kk + (lane & 15), n0 + 8 * (lane >> 4), DP);
        ldsm4t(bh, kf + at); ldsm4t(bl, kf + C * DP + at);
      } else {
        ldsm4t(bh, sv + swz(16 * kk + (lane & 15), n0 + 8 * (lane >> 4), 128));
      }
#pragma unroll
      for (int m = kk; m < 4; m++) {
        uint32_t ah[4], al[4];
        const int at = swz(16 * m + (lane & 15), 16 * kk + 8 * (lane >> 4), C);
        ldsm4(ah, xs + at); ldsm4(al, xs + C * C + at);
#pragma unroll
        for (int i = 0; i < 2; i++) {
          mma(acc[m][i], ah, bh[2 * i], bh[2 * i + 1]);
          mma(low[m][i], al, bh[2 * i], bh[2 * i + 1]);
          if (is_w) mma(low[m][i], ah, bl[2 * i], bl[2 * i + 1]);     // v is a bf16 number
        }
      }
    }
#pragma unroll
    for (int m = 0; m < 4; m++)
#pragma unroll
      for (int i = 0; i < 2; i++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
          const int t = 16 * m + g + 8 * e, d = n0 + 8 * i + c2;
          const float x = acc[m][i][2 * e] + low[m][i][2 * e], y = acc[m][i][2 * e + 1] + low[m][i][2 * e + 1];
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
// One block: MT tiles of 16 columns of one head's state.  Warp w computes U and O of tokens 8w .. 8w+7 and owns 1/8 of the
// state's rows.  Two tiles per block read the chunk's operands from shared memory once for both (its bandwidth is the limit);
// one tile gives more blocks when there are few heads.
template <int DP, bool DELTA, int MT>
__global__ void __launch_bounds__(SCAN_THREADS, 1) k_chunk_scan(const ChunkArgs a) {
  pdl_trigger();
  typedef Item<DP> It;
  constexpr int NT = DP / 64;                  // 8-column tiles of the state's rows per warp
  constexpr size_t X0 = DELTA ? 0 : It::Q, XB = It::X_BYTES - X0;      // without A there is no W
  // with one tile U_0 travels with W and Q~; with two the ring has no room for it and each thread loads its own, a chunk ahead
  constexpr bool RING_U = MT == 1;
  constexpr size_t UB = (size_t)C * 16 * 4, XS = XB + (RING_U ? UB : 0), SLOT = XS > It::Y_BYTES ? XS : It::Y_BYTES;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 127) & ~(uintptr_t)127);
  // ring of three half chunks: first half [W, Q~], second half [K^, B, Gamma_C]; half i lies in slot i mod 3, and half i + 3
  // is fetched as soon as half i has been read
  bf16* sS = reinterpret_cast<bf16*>(smem + 3 * SLOT);      // state^T [MT][16][DP], high and low
  bf16* sU = sS + MT * 2 * 16 * DP;            // U^T [MT][16][64], high and low
  uint64_t* bars = reinterpret_cast<uint64_t*>(sU + MT * 2 * 16 * C);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(bars + 3);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c2 = 2 * (lane & 3);
  const int e0 = blockIdx.x * MT * 16, h = blockIdx.y, b = blockIdx.z;
  const int D = a.dim, E = a.vdim, H = a.heads;
  const char* items = a.ws + ((long long)b * H + h) * a.chunks * a.item_bytes;
  if (threadIdx.x == 0) {
    for (int i = 0; i < 3; i++) mbar_init(&bars[i], 1);
    *abort_flag = 0;
    fence_barrier_init();
  }
  __syncthreads();
  auto load = [&](int i) {                     // half i
    if (i >= 2 * a.chunks) return;
    const char* it = items + (long long)(i >> 1) * a.item_bytes;
    uint64_t* bar = &bars[i % 3];
    mbar_expect_tx(bar, (uint32_t)(i & 1 ? It::Y_BYTES : XS));
    bulk_load_1d(smem + (i % 3) * SLOT, it + (i & 1 ? It::K : X0), (uint32_t)(i & 1 ? It::Y_BYTES : XB), bar);
    if (RING_U && !(i & 1)) bulk_load_1d(smem + (i % 3) * SLOT + XB, it + It::U + blockIdx.x * UB, (uint32_t)UB, bar);
  };
  auto half_bar = [&](int i) { return &bars[i % 3]; };
  auto half_phase = [&](int i) { return (uint32_t)((i / 3) & 1); };
  if (threadIdx.x == 0) { load(0); load(1); load(2); }
  // U_0 of this thread's tokens and columns
  float u0[MT][2][2];
  auto fetch_u0 = [&](int c) {
    const float* src = reinterpret_cast<const float*>(items + (long long)c * a.item_bytes + It::U);
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
      for (int e = 0; e < 2; e++)
#pragma unroll
        for (int i = 0; i < 2; i++)
          u0[m][e][i] = e0 + 16 * m < E ? __ldg(src + ((long long)(e0 / 16 + m) * C + 8 * warp + c2 + i) * 16 + g + 8 * e) : 0.f;
  };
  if (!RING_U) fetch_u0(0);
  // the state: rows d0 .. of column e in accumulator fragments, and its two bf16 parts in shared memory
  const int d0 = warp * 8 * NT;
  float S[MT][NT][4];
  auto publish = [&]() {
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
      for (int i = 0; i < NT; i++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
          uint32_t hi, lo;
          split2(S[m][i][2 * e], S[m][i][2 * e + 1], hi, lo);
          bf16* o = sS + m * 32 * DP + swz(g + 8 * e, d0 + 8 * i + c2, DP);
          *reinterpret_cast<uint32_t*>(o) = hi; *reinterpret_cast<uint32_t*>(o + 16 * DP) = lo;
        }
  };
  auto state_at = [&](int e, int d) { return a.S + (((long long)b * H + h) * E + e) * D + d; };
#pragma unroll
  for (int m = 0; m < MT; m++)
#pragma unroll
    for (int i = 0; i < NT; i++)
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const int col = e0 + 16 * m + g + 8 * (e >> 1), d = d0 + 8 * i + c2 + (e & 1);
        S[m][i][e] = col < E && d < D ? *state_at(col, d) : 0.f;
      }
  publish();
  bool ok = true;
  int c = 0;
  for (; c < a.chunks; c++) {
    if (!mbar_wait(half_bar(2 * c), half_phase(2 * c), abort_flag, a.status)) ok = false;
    if (!__syncthreads_and(ok)) break;         // also: the published state is complete
    const uint8_t* x = smem + (2 * c % 3) * SLOT;
    const bf16* tw = reinterpret_cast<const bf16*>(x);
    const bf16* tq = reinterpret_cast<const bf16*>(x + (It::Q - X0));
    if (RING_U) {
      const float* src = reinterpret_cast<const float*>(x + XB);
#pragma unroll
      for (int e = 0; e < 2; e++)
#pragma unroll
        for (int i = 0; i < 2; i++) u0[0][e][i] = src[(8 * warp + c2 + i) * 16 + g + 8 * e];
    }
    float u[MT][3][4] = {}, o[MT][3][4] = {};
#pragma unroll
    for (int k0 = 0; k0 < DP; k0 += 32) {
      // operand rows are tokens 8 warp + 0..7, four 8-channel units (two k steps) per load
      const int at = swz(8 * warp + (lane & 7), k0 + 8 * (lane >> 3), DP);
      uint32_t wh[4], wl[4], qh[4], ql[4];
      if (DELTA) { ldsm4(wh, tw + at); ldsm4(wl, tw + C * DP + at); }
      ldsm4(qh, tq + at); ldsm4(ql, tq + C * DP + at);
#pragma unroll
      for (int k = 0; k < 2; k++)
#pragma unroll
        for (int m = 0; m < MT; m++) {
          uint32_t sh[4], sl[4];
          const bf16* as = sS + m * 32 * DP + swz(lane & 15, k0 + 16 * k + 8 * (lane >> 4), DP);
          ldsm4(sh, as); ldsm4(sl, as + 16 * DP);
          if (DELTA) { mma(u[m][0], sh, wh[2 * k], wh[2 * k + 1]); mma(u[m][1], sh, wl[2 * k], wl[2 * k + 1]); mma(u[m][2], sl, wh[2 * k], wh[2 * k + 1]); }
          mma(o[m][0], sh, qh[2 * k], qh[2 * k + 1]); mma(o[m][1], sh, ql[2 * k], ql[2 * k + 1]); mma(o[m][2], sl, qh[2 * k], qh[2 * k + 1]);
        }
    }
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
      for (int e = 0; e < 2; e++) {
        float v[2];
#pragma unroll
        for (int i = 0; i < 2; i++) v[i] = u0[m][e][i] - (DELTA ? u[m][0][2 * e + i] + (u[m][1][2 * e + i] + u[m][2][2 * e + i]) : 0.f);
        uint32_t hi, lo;
        split2(v[0], v[1], hi, lo);
        bf16* to = sU + m * 32 * C + swz(g + 8 * e, 8 * warp + c2, C);
        *reinterpret_cast<uint32_t*>(to) = hi; *reinterpret_cast<uint32_t*>(to + 16 * C) = lo;
      }
    if (!mbar_wait(half_bar(2 * c + 1), half_phase(2 * c + 1), abort_flag, a.status)) ok = false;
    if (!__syncthreads_and(ok)) break;         // U is complete, this chunk's W, Q~ and the old state have been read
    if (threadIdx.x == 0) load(2 * c + 3);
    if (!RING_U && c + 1 < a.chunks) fetch_u0(c + 1);
    const uint8_t* sy = smem + ((2 * c + 1) % 3) * SLOT;
    const bf16* tk = reinterpret_cast<const bf16*>(sy);
    const bf16* tb = reinterpret_cast<const bf16*>(sy + (It::B - It::K));
    const float* gam = reinterpret_cast<const float*>(sy + (It::G - It::K));
    float low[MT][NT][4] = {};
#pragma unroll
    for (int i = 0; i < NT; i++) {
      const float2 f = *reinterpret_cast<const float2*>(&gam[d0 + 8 * i + c2]);
#pragma unroll
      for (int m = 0; m < MT; m++) { S[m][i][0] *= f.x; S[m][i][1] *= f.y; S[m][i][2] *= f.x; S[m][i][3] *= f.y; }
    }
#pragma unroll
    for (int k = 0; k < 4; k += 2) {
      uint32_t uh[MT][2][4], ul[MT][2][4];
#pragma unroll
      for (int m = 0; m < MT; m++)
#pragma unroll
        for (int i = 0; i < 2; i++) {
          const bf16* at = sU + m * 32 * C + swz(lane & 15, 16 * (k + i) + 8 * (lane >> 4), C);
          ldsm4(uh[m][i], at); ldsm4(ul[m][i], at + 16 * C);
        }
      if (16 * k <= 8 * warp + 7) {            // later tokens do not reach these
        uint32_t bh[4], bl[4];
        const int at = swz(8 * warp + (lane & 7), 16 * k + 8 * (lane >> 3), C);
        ldsm4(bh, tb + at); ldsm4(bl, tb + C * C + at);
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
          for (int i = 0; i < 2; i++) {
            mma(o[m][0], uh[m][i], bh[2 * i], bh[2 * i + 1]); mma(o[m][1], uh[m][i], bl[2 * i], bl[2 * i + 1]); mma(o[m][2], ul[m][i], bh[2 * i], bh[2 * i + 1]);
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
        for (int m = 0; m < MT; m++)
#pragma unroll
          for (int j = 0; j < NT; j++) {
            mma(S[m][j], uh[m][i], kh[2 * j], kh[2 * j + 1]);
            mma(low[m][j], uh[m][i], kl[2 * j], kl[2 * j + 1]); mma(low[m][j], ul[m][i], kh[2 * j], kh[2 * j + 1]);
          }
      }
    }
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
      for (int i = 0; i < NT; i++)
#pragma unroll
        for (int e = 0; e < 4; e++) S[m][i][e] += low[m][i][e];
    publish();
    const int t0 = a.t0 + c * C + 8 * warp + c2;
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const int t = t0 + (e & 1), col = e0 + 16 * m + g + 8 * (e >> 1);
        if (t < a.T && col < E)
          reinterpret_cast<bf16*>(a.o)[((long long)b * a.T + t) * ((long long)H * E) + (long long)h * E + col] = __float2bfloat16_rn(o[m][0][e] + (o[m][1][e] + o[m][2][e]));
      }
    __syncthreads();                           // K^, B have been read
    if (threadIdx.x == 0) load(2 * c + 4);
  }
  if (c < a.chunks) {                          // a wait ran out: let the copies in flight land before the block ends
    if (threadIdx.x == 0)
      for (int i = 2 * c; i < 2 * c + 4 && i < 2 * a.chunks; i++)
        for (uint32_t it = 0; it < (WAIT_LIMIT >> 2) && !mbar_try_wait(half_bar(i), half_phase(i)); ++it) {}
    return;
  }
#pragma unroll
  for (int m = 0; m < MT; m++)
#pragma unroll
    for (int i = 0; i < NT; i++)
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const int col = e0 + 16 * m + g + 8 * (e >> 1), d = d0 + 8 * i + c2 + (e & 1);
        if (col < E && d < D) *state_at(col, d) = S[m][i][e];
      }
}

template <int DP, bool DELTA> int run(ChunkArgs a, cudaStream_t s) {
  typedef Item<DP> It;
  const size_t local = DELTA ? DeltaSmem<DP>::TOTAL : 8 * C * DP;
  const size_t x = DELTA ? It::X_BYTES : It::X_BYTES - It::Q;
  const auto scan = [&](int mt) { return 3 * std::max(x + (mt == 1 ? (size_t)C * 64 : 0), It::Y_BYTES) + (size_t)mt * (2 * 16 * DP * 2 + 2 * 16 * C * 2) + 64 + 128; };
  static PerDevice attr;
  const int dev = PerDevice::current();
  if (dev < 0 || !attr.done[dev]) {
    CUDA_TRY(cudaFuncSetAttribute(DELTA ? k_chunk_local_delta<DP> : k_chunk_local_sum<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)local));
    CUDA_TRY(cudaFuncSetAttribute(k_chunk_scan<DP, DELTA, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)scan(1)));
    CUDA_TRY(cudaFuncSetAttribute(k_chunk_scan<DP, DELTA, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)scan(2)));
    if (dev >= 0) attr.done[dev] = true;
  }
  a.item_bytes = (It::bytes(a.vdim) + 127) / 128 * 128;
  const int total = cdiv(a.T, C);
  const int most = (int)std::min<long long>(total, (long long)a.ws_bytes / ((long long)a.item_bytes * a.B * a.heads));
  // the local part runs one block per SM: of the segment lengths that fit, the one that needs the fewest waves in all
  int seg = most;
  long long best = -1;
  for (int n = most; n > most / 2; n--) {
    const auto waves = [&](int chunks) { return (long long)cdiv((long long)chunks * a.heads * a.B, device_sm_count()); };
    const long long w = total / n * waves(n) + (total % n ? waves(total % n) : 0);
    if (best < 0 || w < best) { best = w; seg = n; }
  }
  if (seg <= 0) return femto_fail(FEMTO_ERR_NOMEM, "chunked recurrence: workspace too small for %d columns of %d heads", a.B, a.heads);
  for (int c0 = 0; c0 < total; c0 += seg) {
    a.t0 = c0 * C; a.chunks = std::min(seg, total - c0);
    (DELTA ? k_chunk_local_delta<DP> : k_chunk_local_sum<DP>)<<<dim3(a.chunks, a.heads, a.B), LOCAL_THREADS, local, s>>>(a);
    KERNEL_CHECK();
    if (cdiv(a.vdim, 32) * a.heads * a.B >= device_sm_count())
      k_chunk_scan<DP, DELTA, 2><<<dim3(cdiv(a.vdim, 32), a.heads, a.B), SCAN_THREADS, scan(2), s>>>(a);
    else
      k_chunk_scan<DP, DELTA, 1><<<dim3(cdiv(a.vdim, 16), a.heads, a.B), SCAN_THREADS, scan(1), s>>>(a);
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
