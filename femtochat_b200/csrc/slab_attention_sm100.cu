// A prompt's attention for the layer-listing decoders on the sm_100a tensor cores: causal from position `first` on, for any
// query/key and value sizes that are multiples of 8.  The structure is that of the GPT's forward kernel
// (attention_sm100.cu): one CTA owns 128 queries of one head, a TMA warp streams key and value tiles of 128 tokens, one
// thread issues S = Q K^T into one of two TMEM buffers, another O += P V with P read back from TMEM, and two threads per
// query row do the softmax.  What differs is how the operands arrive: each 64-channel slab is its own TMA box, and a slab
// that reaches past a head's channels is filled with zeros by the copy.
//
//   Latent attention: the unrotated part of K comes from the expanded keys of the head, the rotated part straight from the
//   cache rows that all heads share.
//   Windowed attention: the key tiles are those of the first `keep` tokens and then those of the window; groups of query
//   heads share a key/value head; a sink enters the sum at the end.  With two maps (differential attention) the steps of a
//   tile alternate between them: the two S buffers and two halves of O belong to one map each, the value tile to both.
//   The softmax weights enter P V as the sum of two bf16 numbers (SPLIT), so they keep 32-bit accuracy: a tile's P takes
//   the 128 columns that held its S.
//
// Normalisation, the head's own norm of differential attention and the output gate are applied as the result leaves.
#include <algorithm>

#include "decoder.cuh"
#include "sm100_ptx.cuh"

using namespace sm100;

namespace {

constexpr int BQ = 128, BKV = 128, NS = 2, CW = BKV / NS, THREADS = 128 + NS * 128;
constexpr int SLAB = 128 * 64 * 2;                    // one box: 128 tokens x 64 channels
constexpr int MAX_SLABS = 13;                         // 16 KB each: (maps + 2) per query/key slab (Q + two K stages), 2 per value slab
constexpr float LOG2E = 1.4426950408889634f;

struct SlabAttn {
  bf16* o; const bf16* gate; unsigned int* status;
  long long ld_gate;
  int T, first, N, heads, vdim;
  int per;                     // query heads per key/value head
  int n_un, n_rot, n_v;        // slabs of the unrotated part, the rotated part, the values
  int k_un, k_rot;             // 16-channel steps of the two parts
  float c;                     // scale * log2(e)
  int window, keep, gate_mode;
  const float* sink;           // [heads] or null
  const float* lambda;         // two maps: o = a1 - lambda a2, then o / rms(o) * out_scale
  float out_scale, eps;
};

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&h);
}
__device__ __forceinline__ float bf16_low(uint32_t v) { return __uint_as_float(v << 16); }
__device__ __forceinline__ float bf16_high(uint32_t v) { return __uint_as_float(v & 0xffff0000u); }

template <int MAPS, bool SPLIT>
__global__ void __launch_bounds__(THREADS, 1)
slab_attn_kernel(const __grid_constant__ CUtensorMap tmQu, const __grid_constant__ CUtensorMap tmQr,
                 const __grid_constant__ CUtensorMap tmKu, const __grid_constant__ CUtensorMap tmKr,
                 const __grid_constant__ CUtensorMap tmV, const SlabAttn p) {
  grid_launch_dependents();
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const int nqk = p.n_un + p.n_rot;
  const int q_bytes = nqk * SLAB, v_bytes = p.n_v * SLAB;
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + MAPS * q_bytes;     // 2 stages
  uint8_t* sV = sK + 2 * q_bytes;        // 2 stages
  uint64_t* bars = reinterpret_cast<uint64_t*>(sV + 2 * v_bytes);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;    // [2]
  uint64_t* v_full = bars + 3;    // [2]
  uint64_t* s_full = bars + 5;    // [2] S of a tile is in TMEM; also frees the tile's K stage
  uint64_t* p_ready = bars + 7;   // [2]
  uint64_t* pv_done = bars + 9;   // [2] P V of a step has been accumulated; also frees its S/P buffer
  uint64_t* v_free = bars + 11;   // [2] every map's P V of a tile has been accumulated
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 13);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* xmax = reinterpret_cast<float*>(bars + 32);   // [2 parities][NS][128 rows]
  float* xl = xmax + 2 * NS * 128;                     // [NS][128 rows]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int qt = gridDim.x - 1 - blockIdx.x;  // heavy (late) query tiles first
  const int h = blockIdx.y, b = blockIdx.z, hk = h / p.per;
  const int q0 = qt * BQ;
  // Key tiles: first those of the kept tokens before the window, then those from `lo`, the first token that any query of
  // this block sees through the window.  A step is one map of one tile.
  const int last = min(p.first + q0 + BQ - 1, p.N - 1);
  const int lo = max(0, p.first + q0 - p.window + 1), kept = min(p.keep, lo);
  const int nkeep = (kept + BKV - 1) / BKV, ntile = nkeep + (last - lo) / BKV + 1;
  const int nstep = ntile * MAPS;
  auto tile_key = [&](int i) { return i < nkeep ? i * BKV : lo + (i - nkeep) * BKV; };

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; i++) {
      mbar_init(&k_full[i], 1); mbar_init(&v_full[i], 1);
      mbar_init(&s_full[i], 1); mbar_init(&p_ready[i], NS * 4); mbar_init(&pv_done[i], 1); mbar_init(&v_free[i], 1);
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
  const uint32_t tS[2] = {tmem_base, tmem_base + 128};
  const uint32_t tO = tmem_base + 256;

  if (warp == 0) {
    if (lane == 0) {
      // ---------------- TMA producer ----------------
      mbar_expect_tx(q_full, MAPS * q_bytes);
#pragma unroll
      for (int m = 0; m < MAPS; m++) {
        for (int j = 0; j < p.n_un; j++) tma_load_4d(sQ + m * q_bytes + j * SLAB, &tmQu, q_full, j * 64, h * MAPS + m, q0, b);
        for (int j = 0; j < p.n_rot; j++) tma_load_4d(sQ + m * q_bytes + (p.n_un + j) * SLAB, &tmQr, q_full, j * 64, h * MAPS + m, q0, b);
      }
      bool ok = true;
      uint32_t k_issued = 0, v_issued = 0;
      for (int s = 0; s < nstep && ok; s++) {
        const int st = s & 1, i = s / MAPS, m = s % MAPS, vt = i & 1;
        const int key = tile_key(i);
        // the stage's previous user is step s-2, or tile i-2 for the values
        if (s >= 2 && !mbar_wait(&s_full[st], ((s - 2) >> 1) & 1, abort_flag, p.status)) { ok = false; break; }
        uint8_t* k = sK + st * q_bytes;
        mbar_expect_tx(&k_full[st], q_bytes);
        for (int j = 0; j < p.n_un; j++) tma_load_4d(k + j * SLAB, &tmKu, &k_full[st], j * 64, hk * MAPS + m, key, b);
        for (int j = 0; j < p.n_rot; j++) tma_load_3d(k + (p.n_un + j) * SLAB, &tmKr, &k_full[st], j * 64, key, b);
        k_issued = s + 1;
        if (m) continue;
        if (i >= 2 && !mbar_wait(&v_free[vt], ((i - 2) >> 1) & 1, abort_flag, p.status)) { ok = false; break; }
        uint8_t* v = sV + vt * v_bytes;
        mbar_expect_tx(&v_full[vt], v_bytes);
        for (int j = 0; j < p.n_v; j++) tma_load_4d(v + j * SLAB, &tmV, &v_full[vt], j * 64, hk, key, b);
        v_issued = i + 1;
      }
      if (*abort_flag) {
        // let loads already in flight land before the CTA exits
        auto drain = [&](uint64_t* bar, uint32_t ph) { for (uint32_t it = 0; it < WAIT_LIMIT && !mbar_try_wait(bar, ph); ++it) {} };
        drain(q_full, 0);
        for (int st = 0; st < 2; st++) {
          for (int i = (int)k_issued - 1; i >= 0 && i >= (int)k_issued - 2; i--) if ((i & 1) == st) drain(&k_full[st], (i >> 1) & 1);
          for (int i = (int)v_issued - 1; i >= 0 && i >= (int)v_issued - 2; i--) if ((i & 1) == st) drain(&v_full[st], (i >> 1) & 1);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      // ---------------- S = Q K^T issuer ----------------
      constexpr uint32_t idesc_s = idesc_bf16(BQ, BKV, false, false);  // both operands K-major
      const uint32_t q_addr = smem_u32(sQ);
      bool ok = mbar_wait(q_full, 0, abort_flag, p.status);
      for (int s = 0; s < nstep && ok; s++) {
        const int st = s & 1;
        if (!mbar_wait(&k_full[st], (s >> 1) & 1, abort_flag, p.status)) break;
        // S(s) overwrites the buffer that held P(s-2): its P V must have been executed
        if (s >= 2 && !mbar_wait(&pv_done[st], ((s - 2) >> 1) & 1, abort_flag, p.status)) break;
        tc_fence_after();
        const uint32_t k_addr = smem_u32(sK + st * q_bytes), qm_addr = q_addr + (s % MAPS) * q_bytes;
        for (int k = 0; k < p.k_un; k++) {
          const uint32_t off = (k >> 2) * SLAB + (k & 3) * 32;
          mma_ss(tS[st], smem_desc_sw128(qm_addr + off, 16, 1024), smem_desc_sw128(k_addr + off, 16, 1024), idesc_s, k > 0);
        }
        for (int k = 0; k < p.k_rot; k++) {
          const uint32_t off = (p.n_un + (k >> 2)) * SLAB + (k & 3) * 32;
          mma_ss(tS[st], smem_desc_sw128(qm_addr + off, 16, 1024), smem_desc_sw128(k_addr + off, 16, 1024), idesc_s, 1);
        }
        tc_commit(&s_full[st]);
      }
    }
  } else if (warp == 2) {
    if (lane == 0) {
      // ---------------- O += P V issuer ----------------
      const uint32_t idesc_o = idesc_bf16(BQ, (p.vdim + 15) / 16 * 16, false, true);    // V is N-contiguous
      for (int s = 0; s < nstep; s++) {
        const int st = s & 1, i = s / MAPS, m = s % MAPS, vt = i & 1;
        if (!mbar_wait(&p_ready[st], (s >> 1) & 1, abort_flag, p.status)) break;
        if (m == 0 && !mbar_wait(&v_full[vt], (i >> 1) & 1, abort_flag, p.status)) break;
        tc_fence_after();
        const uint32_t v_addr = smem_u32(sV + vt * v_bytes), tOm = tO + m * 128;
#pragma unroll
        for (int k = 0; k < BKV / 16; k++) {
          const uint64_t vd = smem_desc_sw128(v_addr + k * 2048, SLAB, 1024);
          mma_ts(tOm, tS[st] + k * 8, vd, idesc_o, (i > 0 || k > 0) ? 1u : 0u);
          if (SPLIT) mma_ts(tOm, tS[st] + BKV / 2 + k * 8, vd, idesc_o, 1u);
        }
        tc_commit(&pv_done[st]);
        if (m == MAPS - 1) tc_commit(&v_free[vt]);
      }
    }
  } else if (warp >= 4) {
    // ---------------- softmax: NS threads per query row, each owns CW = 128 / NS of the keys of a tile ----------------
    const int quad = warp & 3;
    const int hs = (warp - 4) >> 2;        // which CW keys of each tile; which 32-column chunks of O
    const int r = quad * 32 + lane;
    const int q = p.first + q0 + r;        // position of this row's query
    const bool row_ok = q0 + r < p.T;
    const uint32_t lane_off = (uint32_t)(quad * 32) << 16;
    const int ochunks = (p.vdim + 31) / 32;
    const float c = p.c;
    float m_row[MAPS], l_row[MAPS];      // l_row: this thread's share of the row sum (same m_row in all threads of a row)
#pragma unroll
    for (int m = 0; m < MAPS; m++) { m_row[m] = -INFINITY; l_row[m] = 0.f; }
    bool ok = true;
    for (int i = 0; i < ntile; i++) {
      const int k0 = tile_key(i) + hs * CW;
      // keys from k0 on that this row sees: [k0 + a0, k0 + a1)
      const int a1 = i < nkeep ? kept - k0 : q + 1 - k0;
      const int a0 = i < nkeep || k0 >= q + 1 - p.window ? 0 : q + 1 - p.window - k0;      // below a0 only kept tokens
#pragma unroll
      for (int m = 0; m < MAPS; m++) {
        const int s = i * MAPS + m, st = s & 1;
        float &m_used = m_row[m], &l = l_row[m];
        // After a timed-out wait the warp keeps walking the loop (skipping the work) so that it still
        // meets its partner warps at every row barrier.
        if (ok && !mbar_wait(&s_full[st], (s >> 1) & 1, abort_flag, p.status)) ok = false;
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) { asm volatile("bar.sync %0, %1;" ::"r"(2 + quad), "n"(NS * 32) : "memory"); continue; }
        tc_fence_after();
        float x[CW];
#pragma unroll
        for (int u = 0; u < CW / 32; u++)
          tmem_ld32(tS[st] + lane_off + hs * CW + u * 32, *reinterpret_cast<uint32_t(*)[32]>(&x[u * 32]));
        tmem_ld_wait();
        if (a1 < CW || a0 > 0) {
#pragma unroll
          for (int j = 0; j < CW; j++) x[j] = j < a1 && (j >= a0 || k0 + j < p.keep) ? x[j] : -INFINITY;
        }
        float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
        for (int j = 0; j < CW; j += 4) {
          mx[0] = fmaxf(mx[0], x[j]); mx[1] = fmaxf(mx[1], x[j + 1]);
          mx[2] = fmaxf(mx[2], x[j + 2]); mx[3] = fmaxf(mx[3], x[j + 3]);
        }
        float mt = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * c;   // scaled units (c > 0 keeps the argmax)
        // combine the partial row maxima; after this barrier every thread of the row holds its part of S in
        // registers, so P may overwrite S in TMEM
        xmax[st * (NS * 128) + hs * 128 + r] = mt;
        asm volatile("bar.sync %0, %1;" ::"r"(2 + quad), "n"(NS * 32) : "memory");
#pragma unroll
        for (int o = 1; o < NS; o++) mt = fmaxf(mt, xmax[st * (NS * 128) + ((hs + o) % NS) * 128 + r]);
        const bool grow = mt > m_used + 8.f || (m_used == -INFINITY && mt > -INFINITY);
        if (__any_sync(0xffffffffu, grow)) {
          const float m_new = fmaxf(m_used, mt);
          const float alpha = (m_used == -INFINITY) ? 0.f : fast_exp2(m_used - m_new);
          l *= alpha;
          m_used = m_new;
          if (i > 0) {
            // O lives in TMEM and is being accumulated by the tensor core: wait for this map's previous P V
            bool w = mbar_wait(&pv_done[(s - MAPS) & 1], ((s - MAPS) >> 1) & 1, abort_flag, p.status);
            w = __all_sync(0xffffffffu, w);
            if (!w) { ok = false; continue; }
            tc_fence_after();
            for (int u = hs; u < ochunks; u += NS) {
              uint32_t rr[32];
              tmem_ld32(tO + m * 128 + lane_off + u * 32, rr);
              tmem_ld_wait();
#pragma unroll
              for (int j = 0; j < 32; j++) rr[j] = __float_as_uint(__uint_as_float(rr[j]) * alpha);
              tmem_st32(tO + m * 128 + lane_off + u * 32, rr);
            }
            tmem_st_wait();
          }
        }
        const float mm = (m_used == -INFINITY) ? 0.f : m_used;
        float sm[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int u = 0; u < CW / 32; u++) {
          uint32_t pk[16], pl[16];
#pragma unroll
          for (int j = 0; j < 16; j += 2) {
            const float p0 = fast_exp2(fmaf(x[u * 32 + 2 * j], c, -mm)), p1 = fast_exp2(fmaf(x[u * 32 + 2 * j + 1], c, -mm));
            const float p2 = fast_exp2(fmaf(x[u * 32 + 2 * j + 2], c, -mm)), p3 = fast_exp2(fmaf(x[u * 32 + 2 * j + 3], c, -mm));
            sm[0] += p0; sm[1] += p1; sm[2] += p2; sm[3] += p3;
            pk[j] = pack_bf16(p0, p1);
            pk[j + 1] = pack_bf16(p2, p3);
            if (SPLIT) {
              pl[j] = pack_bf16(p0 - bf16_low(pk[j]), p1 - bf16_high(pk[j]));
              pl[j + 1] = pack_bf16(p2 - bf16_low(pk[j + 1]), p3 - bf16_high(pk[j + 1]));
            }
          }
          tmem_st16(tS[st] + lane_off + hs * (CW / 2) + u * 16, pk);
          if (SPLIT) tmem_st16(tS[st] + BKV / 2 + lane_off + hs * (CW / 2) + u * 16, pl);
        }
        l += (sm[0] + sm[1]) + (sm[2] + sm[3]);
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&p_ready[st]);
      }
    }
    // 1 / (row sum), the sink's term included
    float inv[MAPS];
#pragma unroll
    for (int m = 0; m < MAPS; m++) {
      float l = l_row[m];
      xl[hs * 128 + r] = l;
      asm volatile("bar.sync %0, %1;" ::"r"(2 + quad), "n"(NS * 32) : "memory");
#pragma unroll
      for (int o = 1; o < NS; o++) l += xl[((hs + o) % NS) * 128 + r];
      asm volatile("bar.sync %0, %1;" ::"r"(2 + quad), "n"(NS * 32) : "memory");
      if (p.sink) {
        const float z = __ldg(p.sink + h) * LOG2E, top = fmaxf(z, m_row[m]), f = fast_exp2(m_row[m] - top);
        inv[m] = f / (l * f + fast_exp2(z - top));
      } else {
        inv[m] = 1.f / l;
      }
      const int s = (ntile - 1) * MAPS + m;
      ok = ok && mbar_wait(&pv_done[s & 1], (s >> 1) & 1, abort_flag, p.status);
    }
    ok = __all_sync(0xffffffffu, ok);
    if (ok) tc_fence_after();
    const long long row = (long long)b * p.T + q0 + r;
    float lam = 0.f, rms = 1.f;
    if constexpr (MAPS == 2) {
      // the head's own norm: mean square of a1 - lambda a2 over both threads of the row
      lam = __ldg(p.lambda) * inv[1];
      float ss = 0.f;
      if (ok) {
        for (int u = hs; u < ochunks; u += NS) {
          uint32_t r1[32], r2[32];
          tmem_ld32(tO + lane_off + u * 32, r1);
          tmem_ld32(tO + 128 + lane_off + u * 32, r2);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 32; j++) {
            const float v = __uint_as_float(r1[j]) * inv[0] - __uint_as_float(r2[j]) * lam;
            ss += u * 32 + j < p.vdim ? v * v : 0.f;
          }
        }
      }
      xl[hs * 128 + r] = ss;
      asm volatile("bar.sync %0, %1;" ::"r"(2 + quad), "n"(NS * 32) : "memory");
#pragma unroll
      for (int o = 1; o < NS; o++) ss += xl[((hs + o) % NS) * 128 + r];
      rms = p.out_scale / sqrtf(ss / p.vdim + p.eps);
    }
    if (ok) {
      if (p.gate_mode == FEMTO_GATE_HEAD && row_ok) rms *= 1.f / (1.f + expf(-__bfloat162float(p.gate[row * p.ld_gate + h])));
      const bf16* gate = p.gate_mode == FEMTO_GATE_ELEMENT ? p.gate + row * p.ld_gate + (long long)h * p.vdim : nullptr;
      bf16* o = p.o + (row * p.heads + h) * p.vdim;
      for (int u = hs; u < ochunks; u += NS) {
        uint32_t r1[32], r2[32];
        tmem_ld32(tO + lane_off + u * 32, r1);
        if constexpr (MAPS == 2) tmem_ld32(tO + 128 + lane_off + u * 32, r2);
        tmem_ld_wait();
        if (row_ok) {
#pragma unroll
          for (int j = 0; j < 32; j += 8) {
            if (u * 32 + j < p.vdim) {
              float v[8];
#pragma unroll
              for (int e = 0; e < 8; e++) {
                v[e] = __uint_as_float(r1[j + e]) * inv[0];
                if constexpr (MAPS == 2) v[e] -= __uint_as_float(r2[j + e]) * lam;
                v[e] *= rms;
              }
              if (gate) {
                float z[8];
                load_vec<bf16, 8>(gate + u * 32 + j, z);
#pragma unroll
                for (int e = 0; e < 8; e++) v[e] *= __fdividef(1.f, 1.f + __expf(-z[e]));
              }
              store_vec<bf16, 8>(o + u * 32 + j, v);
            }
          }
        }
      }
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
size_t smem_bytes(int maps, int nqk, int nv) { return (size_t)SLAB * ((maps + 2) * nqk + 2 * nv) + 1024 + 256 + 3 * NS * 128 * 4; }

template <int MAPS, bool SPLIT>
int launch(const CUtensorMap& tmQu, const CUtensorMap& tmQr, const CUtensorMap& tmKu, const CUtensorMap& tmKr, const CUtensorMap& tmV,
           const SlabAttn& p, int B, cudaStream_t s) {
  static PerDevice attr;
  const int dev = PerDevice::current();
  if (dev < 0 || !attr.done[dev]) {
    CUDA_TRY(cudaFuncSetAttribute(slab_attn_kernel<MAPS, SPLIT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    if (dev >= 0) attr.done[dev] = true;
  }
  slab_attn_kernel<MAPS, SPLIT><<<dim3(cdiv(p.T, BQ), p.heads, B), THREADS, smem_bytes(MAPS, p.n_un + p.n_rot, p.n_v), s>>>(tmQu, tmQr, tmKu, tmKr, tmV, p);
  KERNEL_CHECK();
  return 0;
}

}  // namespace

bool latent_attention_tc_supported(const LatentArgs& a) {
  if ((a.dim | a.rot_dim | a.vdim) & 7 || a.vdim > 256 || !(a.scale > 0.f)) return false;
  if (3 * (slabs(a.dim) + slabs(a.rot_dim)) + 2 * slabs(a.vdim) > MAX_SLABS) return false;
  return aligned16(a.q) && aligned16(a.kv) && aligned16(a.latent) && aligned16(a.o);
}

int latent_attention_tc(const LatentArgs& a, cudaStream_t s) {
  const uint64_t N = a.first + a.T, H = a.heads, hd = a.dim + a.rot_dim, wide = H * (a.dim + a.vdim);
  CUtensorMap tmQu, tmQr, tmKu, tmKr, tmV;
  const bf16 *q = (const bf16*)a.q, *kv = (const bf16*)a.kv;
  const uint32_t box4[4] = {64, 1, 128, 1}, box3[3] = {64, 128, 1};
  {
    const uint64_t d[4] = {(uint64_t)a.dim, H, (uint64_t)a.T, (uint64_t)a.B}, st[3] = {hd, H * hd, H * hd * a.T};
    FEMTO_TRY(make_tmap_nd_bf16(&tmQu, q, 4, d, st, box4));
  }
  tmQr = tmQu;
  {
    const uint64_t d[4] = {(uint64_t)a.dim, H, N, (uint64_t)a.B}, st[3] = {(uint64_t)a.dim, wide, wide * a.maxT};
    FEMTO_TRY(make_tmap_nd_bf16(&tmKu, kv, 4, d, st, box4));
  }
  tmKr = tmKu;
  if (a.rot_dim > 0) {
    const uint64_t d[4] = {(uint64_t)a.rot_dim, H, (uint64_t)a.T, (uint64_t)a.B}, st[3] = {hd, H * hd, H * hd * a.T};
    FEMTO_TRY(make_tmap_nd_bf16(&tmQr, q + a.dim, 4, d, st, box4));
    const uint64_t dk[3] = {(uint64_t)a.rot_dim, N, (uint64_t)a.B}, sk[2] = {(uint64_t)a.ld, (uint64_t)a.ld * a.maxT};
    FEMTO_TRY(make_tmap_nd_bf16(&tmKr, (const bf16*)a.latent + a.lp, 3, dk, sk, box3));
  }
  {
    const uint64_t d[4] = {(uint64_t)a.vdim, H, N, (uint64_t)a.B}, st[3] = {(uint64_t)a.vdim, wide, wide * a.maxT};
    FEMTO_TRY(make_tmap_nd_bf16(&tmV, kv + H * a.dim, 4, d, st, box4));
  }
  SlabAttn p = {};
  p.o = (bf16*)a.o; p.gate = (const bf16*)a.gate; p.status = a.d->status; p.ld_gate = a.ld_gate; p.gate_mode = FEMTO_GATE_HEAD;
  p.T = a.T; p.first = a.first; p.N = (int)N; p.heads = a.heads; p.per = 1; p.vdim = a.vdim; p.window = 1 << 30;
  p.n_un = slabs(a.dim); p.n_rot = slabs(a.rot_dim); p.n_v = slabs(a.vdim);
  p.k_un = cdiv(a.dim, 16); p.k_rot = cdiv(a.rot_dim, 16); p.c = a.scale * LOG2E;
  return launch<1, false>(tmQu, tmQr, tmKu, tmKr, tmV, p, a.B, s);
}

bool window_attention_tc_supported(const WindowAttnArgs& a) {
  if ((a.dim | a.vdim) & 7 || a.vdim > (a.maps == 2 ? 128 : 256) || !(a.scale > 0.f)) return false;
  if ((a.maps + 2) * slabs(a.dim) + 2 * slabs(a.vdim) > MAX_SLABS) return false;
  if ((a.ldq | a.ld | a.vo | a.ld_gate) & 7) return false;
  return aligned16(a.q) && aligned16(a.kv) && aligned16(a.o) && (a.gate_mode != FEMTO_GATE_ELEMENT || aligned16(a.gate));
}

int window_attention_tc(const WindowAttnArgs& a, cudaStream_t s) {
  const uint64_t N = a.first + a.T, H = a.heads, G = a.kv_heads, M = a.maps, D = a.dim, E = a.vdim;
  CUtensorMap tmQ, tmK, tmV;
  const bf16* kv = (const bf16*)a.kv;
  const uint32_t box[4] = {64, 1, 128, 1};
  {
    const uint64_t d[4] = {D, H * M, (uint64_t)a.T, (uint64_t)a.B}, st[3] = {D, (uint64_t)a.ldq, (uint64_t)a.ldq * a.T};
    FEMTO_TRY(make_tmap_nd_bf16(&tmQ, a.q, 4, d, st, box));
  }
  const uint64_t ld = a.ld, col = ld * a.maxT;
  {
    const uint64_t d[4] = {D, G * M, N, (uint64_t)a.B}, st[3] = {D, ld, col};
    FEMTO_TRY(make_tmap_nd_bf16(&tmK, kv, 4, d, st, box));
  }
  {
    const uint64_t d[4] = {E, G, N, (uint64_t)a.B}, st[3] = {E, ld, col};
    FEMTO_TRY(make_tmap_nd_bf16(&tmV, kv + a.vo, 4, d, st, box));
  }
  SlabAttn p = {};
  p.o = (bf16*)a.o; p.gate = (const bf16*)a.gate; p.status = a.status; p.ld_gate = a.ld_gate; p.gate_mode = a.gate_mode;
  p.T = a.T; p.first = a.first; p.N = (int)N; p.heads = a.heads; p.per = a.heads / a.kv_heads; p.vdim = a.vdim;
  p.window = a.window; p.keep = a.keep; p.sink = a.sink; p.lambda = a.lambda; p.out_scale = a.out_scale; p.eps = a.eps;
  p.n_un = slabs(a.dim); p.n_v = slabs(a.vdim); p.k_un = cdiv(a.dim, 16); p.c = a.scale * LOG2E;
  return a.maps == 2 ? launch<2, true>(tmQ, tmQ, tmK, tmK, tmV, p, a.B, s) : launch<1, true>(tmQ, tmQ, tmK, tmK, tmV, p, a.B, s);
}
