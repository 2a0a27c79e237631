// A prompt's attention for the layer-listing decoders on the sm_100a tensor cores: causal from position `first` on, for any
// query/key and value sizes that are multiples of 8.  Each 64-channel slab of an operand is a TMA box of its own, and a slab
// that reaches past a head's channels is filled with zeros by the copy.
//
//   Latent attention: the unrotated part of K comes from the expanded keys of the head, the rotated part straight from the
//   cache rows that all heads share.
//   Windowed attention: the key tiles are those of the first `keep` tokens and then those of the window; groups of query
//   heads share a key/value head; a sink enters the sum at the end.  The softmax weights enter P V as the sum of two bf16
//   numbers (SPLIT), so they keep 32-bit accuracy: a tile's P takes the columns that held its S.
//
// One CTA per SM walks the items (128 queries of one head), latest queries first.  The steps of an item, 128 queries against
// 64 keys, alternate between two streams, each with two buffers for S / P and an accumulator O of its own in tensor memory and
// four softmax warps (one thread per query row): S of a stream's next step is there before the softmax of this one is
// done, and the exponentials of one stream run beside the loads and the row maxima of the other.  With two maps (differential
// attention) the streams are the maps, otherwise the even and the odd key tiles, whose partial results meet at the end.  One
// warp loads Q and K, one V (four stages of each), one issues S = Q K^T, another O += P V with P read back from tensor
// memory; all of them run ahead into the next item.  Sum of the streams, the head's own norm of differential attention and
// the output gate are applied as the result leaves.
#include <algorithm>

#include "decoder.cuh"
#include "sm100_ptx.cuh"

using namespace sm100;

namespace {

constexpr int BQ = 128, BKV = 64, THREADS = 128 + 2 * 128;
constexpr int STAGES = 4;                             // of K and of V
constexpr int SLAB_Q = BQ * 64 * 2, SLAB = BKV * 64 * 2;   // one box: 128 queries or 64 keys x 64 channels
constexpr int MAX_SLABS = 26;                         // 8 KB each: 2 maps + STAGES per query/key slab, STAGES per value slab
constexpr int MAX_V = 128;                            // value columns of one launch
constexpr float LOG2E = 1.4426950408889634f;
// registers per thread: 384 threads launch with 168 = (128 * 104 + 256 * 200) / 384
constexpr int REGS_ROLES = 104, REGS_SOFTMAX = 200;
struct SlabAttn {
  bf16* o; const bf16* gate; unsigned int* status;
  long long ld_gate;
  int T, first, N, heads, vdim, items, qtiles;
  int col0, cols;              // value columns of this launch
  int per;                     // query heads per key/value head
  int n_un, n_rot, n_v;        // slabs of the unrotated part, the rotated part, the values
  int k_un, k_rot;             // 16-channel steps of the two parts
  float c;                     // scale * log2(e)
  int window, keep, gate_mode;
  const float* sink;           // [heads] or null
  const float* lambda;         // two maps: o = a1 - lambda a2, then o / rms(o) * out_scale
  float out_scale, eps;
};

// One item: 128 queries of one head and the key tiles that they see: first those of the kept tokens before the window, then
// those from `lo`, the first token that any of the queries sees through the window.
struct Item {
  int h, b, q0, lo, kept, nkeep, ntile;
  __device__ __forceinline__ Item(const SlabAttn& p, int item) {
    const int per = p.items / p.qtiles;               // heads x columns
    const int rem = item % per;
    h = rem % p.heads;
    b = rem / p.heads;
    q0 = (p.qtiles - 1 - item / per) * BQ;
    const int last = min(p.first + q0 + BQ - 1, p.N - 1);
    lo = max(0, p.first + q0 - p.window + 1);
    kept = min(p.keep, lo);
    nkeep = (kept + BKV - 1) / BKV;
    ntile = nkeep + (last - lo) / BKV + 1;
  }
  __device__ __forceinline__ int key(int i) const { return i < nkeep ? i * BKV : lo + (i - nkeep) * BKV; }
};

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&h);
}
__device__ __forceinline__ float bf16_low(uint32_t v) { return __uint_as_float(v << 16); }
__device__ __forceinline__ float bf16_high(uint32_t v) { return __uint_as_float(v & 0xffff0000u); }

// S (+)= Q K^T over `steps` groups of 16 channels.  A descriptor counts in units of 16 bytes: 16 channels further are 2 of them.
__device__ __forceinline__ void issue_slabs(uint32_t tS, uint64_t qd, uint64_t kd, int steps, bool accumulate, uint32_t idesc) {
  for (; steps > 0; steps -= 4, qd += SLAB_Q >> 4, kd += SLAB >> 4) {
#pragma unroll
    for (int k = 0; k < 4; k++)
      if (k < steps) mma_ss(tS, qd + 2 * k, kd + 2 * k, idesc, k > 0 || accumulate);
    accumulate = true;
  }
}

template <int MAPS, bool SPLIT>
__global__ void __launch_bounds__(THREADS, 1)
slab_attn_kernel(const __grid_constant__ CUtensorMap tmQu, const __grid_constant__ CUtensorMap tmQr,
                 const __grid_constant__ CUtensorMap tmKu, const __grid_constant__ CUtensorMap tmKr,
                 const __grid_constant__ CUtensorMap tmV, const SlabAttn p) {
  grid_launch_dependents();
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const int q_bytes = (p.n_un + p.n_rot) * SLAB_Q, k_bytes = (p.n_un + p.n_rot) * SLAB, v_bytes = p.n_v * SLAB;
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + MAPS * q_bytes;
  uint8_t* sV = sK + STAGES * k_bytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(sV + STAGES * v_bytes);
  uint64_t* q_full = bars;
  uint64_t* q_free = bars + 1;    // the item's last S has been executed
  uint64_t* o_free = bars + 2;    // every softmax warp has read the item's O
  uint64_t* k_full = bars + 3;    // [STAGES]
  uint64_t* k_free = bars + 7;    // [STAGES]
  uint64_t* v_full = bars + 11;   // [STAGES]
  uint64_t* v_free = bars + 15;   // [STAGES]
  uint64_t* s_full = bars + 19;   // [2 streams][2 buffers]
  uint64_t* p_ready = bars + 23;  // [2 streams][2 buffers]
  uint64_t* pv_done = bars + 27;  // [2 streams][2 buffers] a step's P V has been accumulated; also frees its S / P buffer
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 31);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* xl = reinterpret_cast<float*>(bars + 32);     // [2 streams][128 rows] row sums, maxima, squares of the results
  float* xm = xl + 2 * 128;
  float* xs = xm + 2 * 128;

  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1); mbar_init(q_free, 1); mbar_init(o_free, 8);
    for (int i = 0; i < 4; i++) {
      mbar_init(&k_full[i], 1); mbar_init(&k_free[i], 1); mbar_init(&v_full[i], 1); mbar_init(&v_free[i], 1);
      mbar_init(&s_full[i], 1); mbar_init(&p_ready[i], 4); mbar_init(&pv_done[i], 1);
    }
    *abort_flag = 0;
    fence_barrier_init();
    tma_prefetch_desc(&tmQu); tma_prefetch_desc(&tmKu); tma_prefetch_desc(&tmKr); tma_prefetch_desc(&tmV);
  }
  if (warp == 1) { tmem_alloc(tmem_slot, 512); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  grid_dependency_wait();

  // Every role walks the same items in the same order and counts what it has seen: n items, kc key tiles, vc value tiles, cx[X]
  // steps of stream X (its turn t uses buffer t & 1).  The phase of a barrier is the count of its own turns, modulo two.
  if (warp < 4) {
    reg_dealloc<REGS_ROLES>();
    // let loads already in flight land before the CTA exits
    auto drain = [&](uint64_t* bar, int turn) { for (uint32_t t = 0; t < WAIT_LIMIT && !mbar_try_wait(bar, turn & 1); ++t) {} };
    if (warp == 0) {
      // ---------------- loads of Q and K ----------------
      int n = 0, kc = 0;
      bool ok = true;
      for (int item = blockIdx.x; item < p.items && ok; item += gridDim.x) {
        const Item it(p, item);
        const int hk = it.h / p.per;
        if (n >= 1 && !mbar_wait_warp(q_free, (n - 1) & 1, abort_flag, p.status)) break;
        if (elect_one()) {
          mbar_expect_tx(q_full, MAPS * q_bytes);
#pragma unroll
          for (int m = 0; m < MAPS; m++) {
            for (int j = 0; j < p.n_un; j++) tma_load_4d(sQ + m * q_bytes + j * SLAB_Q, &tmQu, q_full, j * 64, it.h * MAPS + m, it.q0, it.b);
            for (int j = 0; j < p.n_rot; j++) tma_load_4d(sQ + m * q_bytes + (p.n_un + j) * SLAB_Q, &tmQr, q_full, j * 64, it.h * MAPS + m, it.q0, it.b);
          }
        }
        n++;
        for (int i = 0; i < it.ntile && ok; i++) {
          const int key = it.key(i);
#pragma unroll
          for (int m = 0; m < MAPS; m++) {
            const int st = kc % STAGES;
            if (kc >= STAGES && !mbar_wait_warp(&k_free[st], (kc / STAGES - 1) & 1, abort_flag, p.status)) { ok = false; break; }
            if (elect_one()) {
              uint8_t* k = sK + st * k_bytes;
              mbar_expect_tx(&k_full[st], k_bytes);
              for (int j = 0; j < p.n_un; j++) tma_load_4d(k + j * SLAB, &tmKu, &k_full[st], j * 64, hk * MAPS + m, key, it.b);
              for (int j = 0; j < p.n_rot; j++) tma_load_3d(k + (p.n_un + j) * SLAB, &tmKr, &k_full[st], j * 64, key, it.b);
            }
            kc++;
          }
        }
      }
      if (*abort_flag) {
        if (n >= 1) drain(q_full, n - 1);
        for (int i = max(0, kc - STAGES); i < kc; i++) drain(&k_full[i % STAGES], i / STAGES);
      }
    } else if (warp == 3) {
      // ---------------- loads of V ----------------
      int vc = 0;
      bool ok = true;
      for (int item = blockIdx.x; item < p.items && ok; item += gridDim.x) {
        const Item it(p, item);
        const int hk = it.h / p.per;
        for (int i = 0; i < it.ntile; i++, vc++) {
          const int vt = vc % STAGES;
          if (vc >= STAGES && !mbar_wait_warp(&v_free[vt], (vc / STAGES - 1) & 1, abort_flag, p.status)) { ok = false; break; }
          if (elect_one()) {
            uint8_t* v = sV + vt * v_bytes;
            mbar_expect_tx(&v_full[vt], v_bytes);
            for (int j = 0; j < p.n_v; j++) tma_load_4d(v + j * SLAB, &tmV, &v_full[vt], p.col0 + j * 64, hk, it.key(i), it.b);
          }
        }
      }
      if (*abort_flag)
        for (int i = max(0, vc - STAGES); i < vc; i++) drain(&v_full[i % STAGES], i / STAGES);
    } else if (warp == 1) {
      // ---------------- S = Q K^T issuer ----------------
      constexpr uint32_t idesc_s = idesc_bf16(BQ, BKV, false, false);  // both operands K-major
      const uint64_t q_desc = smem_desc_sw128(smem_u32(sQ), 16, 1024), k_desc = smem_desc_sw128(smem_u32(sK), 16, 1024);
      int n = 0, kc = 0, cx[2] = {0, 0};
      bool ok = true;
      for (int item = blockIdx.x; item < p.items && ok; item += gridDim.x, n++) {
        const Item it(p, item);
        if (!mbar_wait_warp(q_full, n & 1, abort_flag, p.status)) break;
        for (int i = 0; i < it.ntile && ok; i++) {
#pragma unroll
          for (int m = 0; m < MAPS; m++, kc++) {
            const int X = MAPS == 2 ? m : i & 1, st = kc % STAGES;
            const int turn = X ? cx[1] : cx[0], xb = 2 * X + (turn & 1);
            // S overwrites the buffer that held P of the stream's last step but one: its P V must have been executed
            if (!mbar_wait_warp(&k_full[st], (kc / STAGES) & 1, abort_flag, p.status) ||
                (turn >= 2 && !mbar_wait_warp(&pv_done[xb], ((turn - 2) >> 1) & 1, abort_flag, p.status))) { ok = false; break; }
            tc_fence_after();
            const uint32_t tS = tmem_base + xb * BKV;
            const uint64_t qd = q_desc + (uint32_t)(m * q_bytes >> 4), kd = k_desc + (uint32_t)(st * k_bytes >> 4);
            if (elect_one()) {
              issue_slabs(tS, qd, kd, p.k_un, false, idesc_s);
              if (p.k_rot) issue_slabs(tS, qd + (uint32_t)(p.n_un * SLAB_Q >> 4), kd + (uint32_t)(p.n_un * SLAB >> 4), p.k_rot, true, idesc_s);
              tc_commit(&s_full[xb]);
              tc_commit(&k_free[st]);
              if (i == it.ntile - 1 && m == MAPS - 1) tc_commit(q_free);
            }
            if (X) cx[1]++; else cx[0]++;
          }
        }
      }
    } else if (warp == 2) {
      // ---------------- O += P V issuer ----------------
      const uint64_t v_desc = smem_desc_sw128(smem_u32(sV), SLAB, 1024);
      const uint32_t idesc_o = idesc_bf16(BQ, (p.cols + 15) / 16 * 16, false, true);    // V is N-contiguous
      int n = 0, vc = 0, cx[2] = {0, 0};
      bool ok = true;
      for (int item = blockIdx.x; item < p.items && ok; item += gridDim.x, n++) {
        const Item it(p, item);
        for (int i = 0; i < it.ntile && ok; i++, vc++) {
          const int vt = vc % STAGES;
          const uint64_t vd = v_desc + (uint32_t)(vt * v_bytes >> 4);
#pragma unroll
          for (int m = 0; m < MAPS; m++) {
            const int X = MAPS == 2 ? m : i & 1;
            const int turn = X ? cx[1] : cx[0], xb = 2 * X + (turn & 1);
            const bool fresh = MAPS == 2 ? i == 0 : i < 2;      // the stream's first step of the item overwrites O
            if (!mbar_wait_warp(&p_ready[xb], (turn >> 1) & 1, abort_flag, p.status) ||
                (m == 0 && !mbar_wait_warp(&v_full[vt], (vc / STAGES) & 1, abort_flag, p.status)) ||
                (i == 0 && m == 0 && n >= 1 && !mbar_wait_warp(o_free, (n - 1) & 1, abort_flag, p.status))) { ok = false; break; }
            tc_fence_after();
            const uint32_t tP = tmem_base + xb * BKV, tO = tmem_base + 256 + X * 128;
            if (elect_one()) {
#pragma unroll
              for (int k = 0; k < BKV / 16; k++) {
                // 32 keys: 16 columns of P and, with SPLIT, 16 columns of what rounding took from it; 16 keys of V are 2048 bytes
                mma_ts(tO, tP + (k >> 1) * 32 + (k & 1) * 8, vd + k * 128, idesc_o, (!fresh || k > 0) ? 1u : 0u);
                if (SPLIT) mma_ts(tO, tP + (k >> 1) * 32 + 16 + (k & 1) * 8, vd + k * 128, idesc_o, 1u);
              }
              tc_commit(&pv_done[xb]);
              if (m == MAPS - 1) tc_commit(&v_free[vt]);
            }
            if (X) cx[1]++; else cx[0]++;
          }
        }
      }
    }
  } else {
    // ---------------- softmax: stream X (four warps each), one thread per query row ----------------
    reg_alloc<REGS_SOFTMAX>();
    const int quad = warp & 3, X = (warp - 4) >> 2;
    const int r = quad * 32 + lane;
    const uint32_t lane_off = (uint32_t)(quad * 32) << 16;
    const uint32_t tO = tmem_base + 256 + lane_off;
    const int ochunks = (p.cols + 31) / 32;
    const float c = p.c;
    const uint64_t c2 = pack2(c, c);
    int cx[2] = {0, 0};
    bool ok = true;
    for (int item = blockIdx.x; item < p.items; item += gridDim.x) {
      const Item it(p, item);
      const int q = p.first + it.q0 + r;       // position of this row's query
      float m_used = -INFINITY, l = 0.f;
      const int steps = MAPS == 2 ? it.ntile : (it.ntile + 1 - X) / 2;
      const int before = X ? cx[1] : cx[0];
      for (int s = 0; s < steps && ok; s++) {
        const int turn = before + s, i = MAPS == 2 ? s : 2 * s + X, xb = 2 * X + (turn & 1);
        const uint32_t tS = tmem_base + xb * BKV + lane_off;
        const int k0 = it.key(i);
        // keys from k0 on that this row sees: [k0 + a0, k0 + a1), and below a0 the kept tokens
        const int a1 = i < it.nkeep ? it.kept - k0 : q + 1 - k0;
        const int a0 = i < it.nkeep ? 0 : q + 1 - p.window - k0;
        const int ak = p.keep - k0;
        ok = mbar_wait(&s_full[xb], (turn >> 1) & 1, abort_flag, p.status);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        tc_fence_after();
        // Per group of 32 keys the warp decides together: every lane sees all of it, no lane sees any of it, or mixed.
        bool mixed[2], empty[2];
#pragma unroll
        for (int u = 0; u < 2; u++) {
          mixed[u] = !__all_sync(0xffffffffu, a1 >= 32 * u + 32 && (a0 <= 32 * u || ak >= 32 * u + 32));
          empty[u] = mixed[u] && __all_sync(0xffffffffu, a1 <= 32 * u || (a0 >= 32 * u + 32 && ak <= 32 * u));
        }
        float x[2][32];
#pragma unroll
        for (int u = 0; u < 2; u++)
          if (!empty[u]) tmem_ld32(tS + u * 32, reinterpret_cast<uint32_t(&)[32]>(x[u]));
        tmem_ld_wait();
        float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
        for (int u = 0; u < 2; u++) {
          if (empty[u]) continue;
          if (mixed[u]) {
#pragma unroll
            for (int j = 0; j < 32; j++) x[u][j] = 32 * u + j < a1 && (32 * u + j >= a0 || 32 * u + j < ak) ? x[u][j] : -INFINITY;
          }
#pragma unroll
          for (int j = 0; j < 32; j += 8) {
            mx[0] = max3(mx[0], x[u][j], x[u][j + 1]); mx[1] = max3(mx[1], x[u][j + 2], x[u][j + 3]);
            mx[2] = max3(mx[2], x[u][j + 4], x[u][j + 5]); mx[3] = max3(mx[3], x[u][j + 6], x[u][j + 7]);
          }
        }
        const float mt = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * c;   // scaled units (c > 0 keeps the argmax)
        const bool grow = mt > m_used + 8.f || (m_used == -INFINITY && mt > -INFINITY);
        if (__any_sync(0xffffffffu, grow)) {
          const float m_new = fmaxf(m_used, mt);
          const float alpha = (m_used == -INFINITY) ? 0.f : fast_exp2(m_used - m_new);
          l *= alpha;
          m_used = m_new;
          if (s > 0) {
            // O is being accumulated by the tensor core: wait for the stream's previous P V
            ok = mbar_wait(&pv_done[xb ^ 1], ((turn - 1) >> 1) & 1, abort_flag, p.status);
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            tc_fence_after();
#pragma unroll 1
            for (int u = 0; u < ochunks; u++) {
              uint32_t rr[32];
              tmem_ld32(tO + X * 128 + u * 32, rr);
              tmem_ld_wait();
#pragma unroll
              for (int j = 0; j < 32; j++) rr[j] = __float_as_uint(__uint_as_float(rr[j]) * alpha);
              tmem_st32(tO + X * 128 + u * 32, rr);
            }
            tmem_st_wait();
          }
        }
        const float mm = (m_used == -INFINITY) ? 0.f : m_used;
        const uint64_t nm2 = pack2(-mm, -mm);
        uint64_t sm2[2] = {0ull, 0ull};   // (+0, +0)
#pragma unroll
        for (int u = 0; u < 2; u++) {
          uint32_t pk[16], pl[16];
          if (empty[u]) {
#pragma unroll
            for (int j = 0; j < 16; j++) pk[j] = pl[j] = 0u;
          } else {
#pragma unroll
            for (int j = 0; j < 16; j += 2) {
              float t0, t1, t2, t3;
              unpack2(fma2(pack2(x[u][2 * j], x[u][2 * j + 1]), c2, nm2), t0, t1);
              unpack2(fma2(pack2(x[u][2 * j + 2], x[u][2 * j + 3]), c2, nm2), t2, t3);
              const float p0 = fast_exp2(t0), p1 = fast_exp2(t1), p2 = fast_exp2(t2), p3 = fast_exp2(t3);
              sm2[0] = add2(sm2[0], pack2(p0, p1));
              sm2[1] = add2(sm2[1], pack2(p2, p3));
              pk[j] = pack_bf16(p0, p1);
              pk[j + 1] = pack_bf16(p2, p3);
              if (SPLIT) {
                pl[j] = pack_bf16(p0 - bf16_low(pk[j]), p1 - bf16_high(pk[j]));
                pl[j + 1] = pack_bf16(p2 - bf16_low(pk[j + 1]), p3 - bf16_high(pk[j + 1]));
              }
            }
          }
          tmem_st16(tS + u * 32, pk);      // over the S columns that this thread has loaded
          if (SPLIT) tmem_st16(tS + u * 32 + 16, pl);
        }
        {
          float s0, s1, s2, s3;
          unpack2(sm2[0], s0, s1);
          unpack2(sm2[1], s2, s3);
          l += (s0 + s1) + (s2 + s3);
        }
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&p_ready[xb]);
      }
      cx[0] += MAPS == 2 ? it.ntile : (it.ntile + 1) / 2;
      cx[1] += MAPS == 2 ? it.ntile : it.ntile / 2;
      // ---- the item's result = f[0] O_0 + f[1] O_1; the two warps of a quad take 64 columns each ----
      const bool row_ok = it.q0 + r < p.T;
      const long long row = (long long)it.b * p.T + it.q0 + r;
      const int col = X * 64;              // first column of this thread
      // what the result is multiplied by is on its way while the last products run
      float head_gate = 0.f;
      uint4 gate[8];
      if (row_ok) {
        if (p.gate_mode == FEMTO_GATE_HEAD) head_gate = __bfloat162float(p.gate[row * p.ld_gate + it.h]);
        if (p.gate_mode == FEMTO_GATE_ELEMENT) {
          const uint4* g = reinterpret_cast<const uint4*>(p.gate + row * p.ld_gate + (long long)it.h * p.vdim + p.col0 + col);
#pragma unroll
          for (int j = 0; j < 8; j++)
            if (col + j * 8 < p.cols) gate[j] = __ldg(g + j);
        }
      }
      xl[X * 128 + r] = l;
      xm[X * 128 + r] = m_used;
      asm volatile("bar.sync %0, %1;" ::"r"(2 + quad), "n"(64) : "memory");
      const bool second = MAPS == 2 || it.ntile > 1;      // O_1 holds something
      float f[2];
      {
        const float m0 = xm[r], m1 = xm[128 + r], l0 = xl[r], l1 = xl[128 + r];
        const float z = p.sink ? __ldg(p.sink + it.h) * LOG2E : -INFINITY;
        if constexpr (MAPS == 2) {
          const float t0 = fmaxf(m0, z), t1 = fmaxf(m1, z), e0 = fast_exp2(m0 - t0), e1 = fast_exp2(m1 - t1);
          f[0] = e0 / (l0 * e0 + fast_exp2(z - t0));
          f[1] = -__ldg(p.lambda) * e1 / (l1 * e1 + fast_exp2(z - t1));
        } else {
          const float top = fmaxf(fmaxf(m0, m1), z), e0 = fast_exp2(m0 - top), e1 = fast_exp2(m1 - top);
          const float inv = 1.f / (l0 * e0 + l1 * e1 + fast_exp2(z - top));
          f[0] = e0 * inv; f[1] = e1 * inv;
        }
      }
      ok = ok && mbar_wait(&pv_done[(cx[0] - 1) & 1], ((cx[0] - 1) >> 1) & 1, abort_flag, p.status);
      if (second) ok = ok && mbar_wait(&pv_done[2 + ((cx[1] - 1) & 1)], ((cx[1] - 1) >> 1) & 1, abort_flag, p.status);
      ok = __all_sync(0xffffffffu, ok);
      tc_fence_after();
      auto result = [&](int u, float (&v)[32]) {
        tmem_ld32(tO + col + u * 32, reinterpret_cast<uint32_t(&)[32]>(v));
        if (second) {
          uint32_t v1[32];
          tmem_ld32(tO + 128 + col + u * 32, v1);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 32; j++) v[j] = v[j] * f[0] + __uint_as_float(v1[j]) * f[1];
        } else {
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 32; j++) v[j] *= f[0];
        }
      };
      float mul = 1.f;
      if constexpr (MAPS == 2) {      // the head's own norm
        float ss = 0.f;
#pragma unroll 1
        for (int u = 0; u < 2; u++) {
          if (!ok || col + u * 32 >= p.cols) break;
          float v[32];
          result(u, v);
#pragma unroll
          for (int j = 0; j < 32; j++) ss += col + u * 32 + j < p.cols ? v[j] * v[j] : 0.f;
        }
        xs[X * 128 + r] = ss;
        asm volatile("bar.sync %0, %1;" ::"r"(2 + quad), "n"(64) : "memory");
        mul = p.out_scale / sqrtf((xs[r] + xs[128 + r]) / p.cols + p.eps);
      }
      if (p.gate_mode == FEMTO_GATE_HEAD) mul *= __fdividef(1.f, 1.f + __expf(-head_gate));
      bf16* o = p.o + (row * p.heads + it.h) * p.vdim + p.col0 + col;
#pragma unroll
      for (int u = 0; u < 2; u++) {
        if (!ok || col + u * 32 >= p.cols) continue;
        float v[32];
        result(u, v);
        __syncwarp();
#pragma unroll
        for (int j = 0; j < 4; j++) {
          if (row_ok && col + u * 32 + j * 8 < p.cols) {
            float w[8];
#pragma unroll
            for (int e = 0; e < 8; e++) w[e] = v[8 * j + e] * mul;
            if (p.gate_mode == FEMTO_GATE_ELEMENT) {
              const uint32_t* g = reinterpret_cast<const uint32_t*>(&gate[u * 4 + j]);
#pragma unroll
              for (int e = 0; e < 8; e += 2) {
                w[e] *= __fdividef(1.f, 1.f + __expf(-bf16_low(g[e / 2])));
                w[e + 1] *= __fdividef(1.f, 1.f + __expf(-bf16_high(g[e / 2])));
              }
            }
            store_vec<bf16, 8>(o + u * 32 + 8 * j, w);
          }
        }
        __syncwarp();
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(o_free);
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

int slabs(int n) { return (n + 63) / 64; }
size_t smem_bytes(int maps, int nqk, int nv) { return (size_t)SLAB * ((2 * maps + STAGES) * nqk + STAGES * nv) + 1024 + 256 + 6 * 128 * 4; }

template <int MAPS, bool SPLIT>
int launch(const CUtensorMap& tmQu, const CUtensorMap& tmQr, const CUtensorMap& tmKu, const CUtensorMap& tmKr, const CUtensorMap& tmV,
           SlabAttn p, int B, cudaStream_t s) {
  static PerDevice attr;
  const int dev = PerDevice::current();
  if (dev < 0 || !attr.done[dev]) {
    CUDA_TRY(cudaFuncSetAttribute(slab_attn_kernel<MAPS, SPLIT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    if (dev >= 0) attr.done[dev] = true;
  }
  p.qtiles = cdiv(p.T, BQ);
  p.items = p.qtiles * p.heads * B;
  const int grid = std::min(p.items, device_sm_count());
  for (p.col0 = 0; p.col0 < p.vdim; p.col0 += MAX_V) {      // wide values: the attention once per 128 columns
    p.cols = std::min(MAX_V, p.vdim - p.col0);
    p.n_v = slabs(p.cols);
    CUDA_TRY(launch_dependent(slab_attn_kernel<MAPS, SPLIT>, grid, THREADS, smem_bytes(MAPS, p.n_un + p.n_rot, p.n_v), s, tmQu, tmQr, tmKu, tmKr, tmV, p));
    KERNEL_CHECK();
  }
  return 0;
}

}  // namespace

bool latent_attention_tc_supported(const LatentArgs& a) {
  if ((a.dim | a.rot_dim | a.vdim) & 7 || a.vdim > 256 || !(a.scale > 0.f)) return false;
  if ((2 + STAGES) * (slabs(a.dim) + slabs(a.rot_dim)) + STAGES * slabs(std::min(a.vdim, MAX_V)) > MAX_SLABS) return false;
  return aligned16(a.q) && aligned16(a.kv) && aligned16(a.latent) && aligned16(a.o);
}

int latent_attention_tc(const LatentArgs& a, cudaStream_t s) {
  const uint64_t N = a.first + a.T, H = a.heads, hd = a.dim + a.rot_dim, wide = H * (a.dim + a.vdim);
  CUtensorMap tmQu, tmQr, tmKu, tmKr, tmV;
  const bf16 *q = (const bf16*)a.q, *kv = (const bf16*)a.kv;
  const uint32_t boxQ[4] = {64, 1, BQ, 1}, boxK[4] = {64, 1, BKV, 1}, box3[3] = {64, BKV, 1};
  {
    const uint64_t d[4] = {(uint64_t)a.dim, H, (uint64_t)a.T, (uint64_t)a.B}, st[3] = {hd, H * hd, H * hd * a.T};
    FEMTO_TRY(make_tmap_nd_bf16(&tmQu, q, 4, d, st, boxQ));
  }
  tmQr = tmQu;
  {
    const uint64_t d[4] = {(uint64_t)a.dim, H, N, (uint64_t)a.B}, st[3] = {(uint64_t)a.dim, wide, wide * a.maxT};
    FEMTO_TRY(make_tmap_nd_bf16(&tmKu, kv, 4, d, st, boxK));
  }
  tmKr = tmKu;
  if (a.rot_dim > 0) {
    const uint64_t d[4] = {(uint64_t)a.rot_dim, H, (uint64_t)a.T, (uint64_t)a.B}, st[3] = {hd, H * hd, H * hd * a.T};
    FEMTO_TRY(make_tmap_nd_bf16(&tmQr, q + a.dim, 4, d, st, boxQ));
    const uint64_t dk[3] = {(uint64_t)a.rot_dim, N, (uint64_t)a.B}, sk[2] = {(uint64_t)a.ld, (uint64_t)a.ld * a.maxT};
    FEMTO_TRY(make_tmap_nd_bf16(&tmKr, (const bf16*)a.latent + a.lp, 3, dk, sk, box3));
  }
  {
    const uint64_t d[4] = {(uint64_t)a.vdim, H, N, (uint64_t)a.B}, st[3] = {(uint64_t)a.vdim, wide, wide * a.maxT};
    FEMTO_TRY(make_tmap_nd_bf16(&tmV, kv + H * a.dim, 4, d, st, boxK));
  }
  SlabAttn p = {};
  p.o = (bf16*)a.o; p.gate = (const bf16*)a.gate; p.status = a.d->status; p.ld_gate = a.ld_gate; p.gate_mode = FEMTO_GATE_HEAD;
  p.T = a.T; p.first = a.first; p.N = (int)N; p.heads = a.heads; p.per = 1; p.vdim = a.vdim; p.window = 1 << 30;
  p.n_un = slabs(a.dim); p.n_rot = slabs(a.rot_dim);
  p.k_un = cdiv(a.dim, 16); p.k_rot = cdiv(a.rot_dim, 16); p.c = a.scale * LOG2E;
  return launch<1, false>(tmQu, tmQr, tmKu, tmKr, tmV, p, a.B, s);
}

bool window_attention_tc_supported(const WindowAttnArgs& a) {
  if ((a.dim | a.vdim) & 7 || a.vdim > (a.maps == 2 ? MAX_V : 256) || !(a.scale > 0.f)) return false;
  if ((2 * a.maps + STAGES) * slabs(a.dim) + STAGES * slabs(std::min(a.vdim, MAX_V)) > MAX_SLABS) return false;
  if ((a.ldq | a.ld | a.vo | a.ld_gate) & 7) return false;
  return aligned16(a.q) && aligned16(a.kv) && aligned16(a.o) && (a.gate_mode != FEMTO_GATE_ELEMENT || aligned16(a.gate));
}

int window_attention_tc(const WindowAttnArgs& a, cudaStream_t s) {
  const uint64_t N = a.first + a.T, H = a.heads, G = a.kv_heads, M = a.maps, D = a.dim, E = a.vdim;
  CUtensorMap tmQ, tmK, tmV;
  const bf16* kv = (const bf16*)a.kv;
  const uint32_t boxQ[4] = {64, 1, BQ, 1}, boxK[4] = {64, 1, BKV, 1};
  {
    const uint64_t d[4] = {D, H * M, (uint64_t)a.T, (uint64_t)a.B}, st[3] = {D, (uint64_t)a.ldq, (uint64_t)a.ldq * a.T};
    FEMTO_TRY(make_tmap_nd_bf16(&tmQ, a.q, 4, d, st, boxQ));
  }
  const uint64_t ld = a.ld, col = ld * a.maxT;
  {
    const uint64_t d[4] = {D, G * M, N, (uint64_t)a.B}, st[3] = {D, ld, col};
    FEMTO_TRY(make_tmap_nd_bf16(&tmK, kv, 4, d, st, boxK));
  }
  {
    const uint64_t d[4] = {E, G, N, (uint64_t)a.B}, st[3] = {E, ld, col};
    FEMTO_TRY(make_tmap_nd_bf16(&tmV, kv + a.vo, 4, d, st, boxK));
  }
  SlabAttn p = {};
  p.o = (bf16*)a.o; p.gate = (const bf16*)a.gate; p.status = a.status; p.ld_gate = a.ld_gate; p.gate_mode = a.gate_mode;
  p.T = a.T; p.first = a.first; p.N = (int)N; p.heads = a.heads; p.per = a.heads / a.kv_heads; p.vdim = a.vdim;
  p.window = a.window; p.keep = a.keep; p.sink = a.sink; p.lambda = a.lambda; p.out_scale = a.out_scale; p.eps = a.eps;
  p.n_un = slabs(a.dim); p.k_un = cdiv(a.dim, 16); p.c = a.scale * LOG2E;
  return a.maps == 2 ? launch<2, true>(tmQ, tmQ, tmK, tmK, tmV, p, a.B, s) : launch<1, true>(tmQ, tmQ, tmK, tmK, tmV, p, a.B, s);
}
