// HBM-streaming kernels of the layer-listing decoders: embedding, norms around each sublayer with the fp32 residual
// sum, gated norms, the feed-forward's gate, weight packing, and the product of a few rows with a [out][in] weight.
#include "decoder.cuh"
#include "streaming.cuh"

namespace {

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }

// Sum over the 256 threads of a block; every thread gets it.
__device__ __forceinline__ float block_sum(float v) {
  __shared__ float red[8];
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < 8; i++) t += red[i];
  return t;
}

constexpr int RT = 256;   // threads of a row kernel: one row per block

template <typename T>
__global__ void __launch_bounds__(RT) k_dec_embed(const T* __restrict__ table, const int* __restrict__ tokens, int ld_tok, int T_,
                                                  int base, int vocab, float scale, float* __restrict__ x, const NextNorms<T> nn, int d,
                                                  float eps, unsigned int* status) {
  pdl_trigger();
  pdl_wait();
  const int row = blockIdx.x;
  int tk = tokens[(long long)(row / T_) * ld_tok + row % T_] - base;
  if (tk < 0 || tk >= vocab) { if (threadIdx.x == 0) atomicOr(status, ST_BAD_TOKEN); tk = min(max(tk, 0), vocab - 1); }
  const T* src = table + (long long)tk * d;
  float ss = 0.f;
  for (int c = threadIdx.x; c < d; c += RT) { const float f = to_f<T>(src[c]) * scale; ss += f * f; }
  const float inv = 1.f / sqrtf(block_sum(ss) / d + eps);
  for (int c = threadIdx.x; c < d; c += RT) {
    const float f = to_f<T>(src[c]) * scale;
    const long long at = (long long)row * d + c;
    x[at] = f;
    nn.h[at] = from_f<T>(f * inv * nn.w[c]);
    if (nn.h2) nn.h2[at] = from_f<T>(f * inv * nn.w2[c]);
  }
}

template <typename T> __device__ __forceinline__ void load4(const T* p, float (&f)[4]) {
  if constexpr (sizeof(T) == 4) {
    const float4 q = *reinterpret_cast<const float4*>(p);
    f[0] = q.x; f[1] = q.y; f[2] = q.z; f[3] = q.w;
  } else {
    const uint2 q = *reinterpret_cast<const uint2*>(p);
    const bf16* h = reinterpret_cast<const bf16*>(&q);
#pragma unroll
    for (int e = 0; e < 4; e++) f[e] = __bfloat162float(h[e]);
  }
}
template <typename T> __device__ __forceinline__ void store4(T* p, float a, float b, float c, float d) {
  if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
  } else {
    uint2 q;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&q);
    h[0] = __floats2bfloat162_rn(a, b); h[1] = __floats2bfloat162_rn(c, d);
    *reinterpret_cast<uint2*>(p) = q;
  }
}

// NV 4-element vectors per thread stay in registers between the sum and the norms (NV = 0: any width, through memory).
template <typename T, int NV>
__global__ void __launch_bounds__(RT) k_parallel_resid(float* __restrict__ x, const T* __restrict__ y, const T* __restrict__ y2, const MoeRows m,
                                                       const NextNorms<T> nn, int d, float eps) {
  pdl_trigger();
  pdl_wait();
  const long long row = blockIdx.x, base = row * d;
  auto expert_row = [&](int k, float& w) {
    const long long p = row * m.top + k;
    w = m.weight[p];
    return reinterpret_cast<const T*>(m.out) + (m.slot ? m.slot[p] : p) * (long long)d;
  };
  float ss = 0.f;
  if constexpr (NV > 0) {
    float r[NV][4], f[4];
#pragma unroll
    for (int i = 0; i < NV; i++) {
      const int c = (i * RT + threadIdx.x) * 4;
      if (c >= d) continue;
      load4<T>(y + base + c, r[i]);
      if (y2) {
        load4<T>(y2 + base + c, f);
#pragma unroll
        for (int e = 0; e < 4; e++) r[i][e] += f[e];
      }
    }
#pragma unroll 4
    for (int k = 0; k < m.top; k++) {
      float w;
      const T* o = expert_row(k, w);
#pragma unroll
      for (int i = 0; i < NV; i++) {
        const int c = (i * RT + threadIdx.x) * 4;
        if (c >= d) continue;
        load4<T>(o + c, f);
#pragma unroll
        for (int e = 0; e < 4; e++) r[i][e] = fmaf(w, f[e], r[i][e]);
      }
    }
#pragma unroll
    for (int i = 0; i < NV; i++) {
      const int c = (i * RT + threadIdx.x) * 4;
      if (c >= d) continue;
      load4<float>(x + base + c, f);
#pragma unroll
      for (int e = 0; e < 4; e++) { r[i][e] += f[e]; ss += r[i][e] * r[i][e]; }
      store4<float>(x + base + c, r[i][0], r[i][1], r[i][2], r[i][3]);
    }
    if (!nn.h) return;
    const float inv = 1.f / sqrtf(block_sum(ss) / d + eps);
#pragma unroll
    for (int i = 0; i < NV; i++) {
      const int c = (i * RT + threadIdx.x) * 4;
      if (c >= d) continue;
      load4<float>(nn.w + c, f);
      store4<T>(nn.h + base + c, r[i][0] * inv * f[0], r[i][1] * inv * f[1], r[i][2] * inv * f[2], r[i][3] * inv * f[3]);
      if (!nn.h2) continue;
      load4<float>(nn.w2 + c, f);
      store4<T>(nn.h2 + base + c, r[i][0] * inv * f[0], r[i][1] * inv * f[1], r[i][2] * inv * f[2], r[i][3] * inv * f[3]);
    }
  } else {
    for (int c = threadIdx.x; c < d; c += RT) {
      float r = to_f<T>(y[base + c]) + (y2 ? to_f<T>(y2[base + c]) : 0.f);
      for (int k = 0; k < m.top; k++) {
        float w;
        const T* o = expert_row(k, w);
        r = fmaf(w, to_f<T>(o[c]), r);
      }
      r += x[base + c];
      x[base + c] = r;
      ss += r * r;
    }
    if (!nn.h) return;
    const float inv = 1.f / sqrtf(block_sum(ss) / d + eps);
    for (int c = threadIdx.x; c < d; c += RT) {
      const float r = x[base + c] * inv;
      nn.h[base + c] = from_f<T>(r * nn.w[c]);
      if (nn.h2) nn.h2[base + c] = from_f<T>(r * nn.w2[c]);
    }
  }
}

// NV 4-element vectors per thread stay in registers between the two norms (NV = 0: any width, through memory).
template <typename T, int NV>
__global__ void __launch_bounds__(RT) k_resid_norm(float* __restrict__ x, const T* __restrict__ y, const float* __restrict__ w_post,
                                                   float m, const float* __restrict__ w_pre, T* __restrict__ h, int d, float eps) {
  pdl_trigger();
  pdl_wait();
  const long long base = (long long)blockIdx.x * d;
  if constexpr (NV > 0) {
    float f[NV][4], r[NV][4];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; i++) {
      const int c = (i * RT + threadIdx.x) * 4;
      if (c < d) {
        if constexpr (sizeof(T) == 4) {
          const float4 q = *reinterpret_cast<const float4*>(y + base + c);
          f[i][0] = q.x; f[i][1] = q.y; f[i][2] = q.z; f[i][3] = q.w;
        } else {
          const uint2 q = *reinterpret_cast<const uint2*>(y + base + c);
          const bf16* hq = reinterpret_cast<const bf16*>(&q);
#pragma unroll
          for (int e = 0; e < 4; e++) f[i][e] = __bfloat162float(hq[e]);
        }
        const float4 q = *reinterpret_cast<const float4*>(x + base + c);
        r[i][0] = q.x; r[i][1] = q.y; r[i][2] = q.z; r[i][3] = q.w;
#pragma unroll
        for (int e = 0; e < 4; e++) ss += f[i][e] * f[i][e];
      }
    }
    float inv = 1.f / sqrtf(block_sum(ss) / d + eps);
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; i++) {
      const int c = (i * RT + threadIdx.x) * 4;
      if (c < d) {
        const float4 w = *reinterpret_cast<const float4*>(w_post + c);
        r[i][0] += m * (f[i][0] * inv * w.x); r[i][1] += m * (f[i][1] * inv * w.y);
        r[i][2] += m * (f[i][2] * inv * w.z); r[i][3] += m * (f[i][3] * inv * w.w);
        *reinterpret_cast<float4*>(x + base + c) = make_float4(r[i][0], r[i][1], r[i][2], r[i][3]);
#pragma unroll
        for (int e = 0; e < 4; e++) ss += r[i][e] * r[i][e];
      }
    }
    if (!h) return;
    inv = 1.f / sqrtf(block_sum(ss) / d + eps);
#pragma unroll
    for (int i = 0; i < NV; i++) {
      const int c = (i * RT + threadIdx.x) * 4;
      if (c < d) {
        const float4 w = *reinterpret_cast<const float4*>(w_pre + c);
        const float o[4] = {r[i][0] * inv * w.x, r[i][1] * inv * w.y, r[i][2] * inv * w.z, r[i][3] * inv * w.w};
        if constexpr (sizeof(T) == 4) {
          *reinterpret_cast<float4*>(h + base + c) = make_float4(o[0], o[1], o[2], o[3]);
        } else {
          uint2 q;
          __nv_bfloat162* hq = reinterpret_cast<__nv_bfloat162*>(&q);
          hq[0] = __floats2bfloat162_rn(o[0], o[1]); hq[1] = __floats2bfloat162_rn(o[2], o[3]);
          *reinterpret_cast<uint2*>(h + base + c) = q;
        }
      }
    }
  } else {
    float ss = 0.f;
    for (int c = threadIdx.x; c < d; c += RT) { const float f = to_f<T>(y[base + c]); ss += f * f; }
    float inv = 1.f / sqrtf(block_sum(ss) / d + eps);
    ss = 0.f;
    for (int c = threadIdx.x; c < d; c += RT) {
      const float r = x[base + c] + m * (to_f<T>(y[base + c]) * inv * w_post[c]);
      x[base + c] = r;
      ss += r * r;
    }
    if (!h) return;
    inv = 1.f / sqrtf(block_sum(ss) / d + eps);
    for (int c = threadIdx.x; c < d; c += RT) h[base + c] = from_f<T>(x[base + c] * inv * w_pre[c]);
  }
}

template <typename T>
__global__ void __launch_bounds__(RT) k_gather_norm(const float* __restrict__ x, const int* __restrict__ want, int stride,
                                                    const float* __restrict__ w, T* __restrict__ h, int d, float eps) {
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.x;
  const float* src = x + (long long)(want ? want[i] : (i + 1) * stride - 1) * d;
  float ss = 0.f;
  for (int c = threadIdx.x; c < d; c += RT) ss += src[c] * src[c];
  const float inv = 1.f / sqrtf(block_sum(ss) / d + eps);
  for (int c = threadIdx.x; c < d; c += RT) h[(long long)i * d + c] = from_f<T>(src[c] * inv * w[c]);
}

// LG lanes per (row, group).
template <typename T, int V, int LG>
__global__ void __launch_bounds__(256) k_gated_norm(const T* __restrict__ in, const float* __restrict__ w, int w_all,
                                                    const T* __restrict__ gate, long long ldg, T* __restrict__ out, long long n,
                                                    int groups, int size, float eps) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & (LG - 1);
  long long it = (long long)blockIdx.x * (256 / LG) + threadIdx.x / LG;
  const bool live = it < n;
  if (!live) it = n - 1;
  const int g = (int)(it % groups);
  const long long row = it / groups;
  const T* a = in + it * size;
  const T* gt = gate + row * ldg + (long long)g * size;
  const float* wg = w + (w_all ? (long long)g * size : 0);
  float ss = 0.f;
#pragma unroll 4
  for (int c = lane * V; c < size; c += LG * V) {
    float f[V];
    load_vec<T, V>(a + c, f);
#pragma unroll
    for (int e = 0; e < V; e++) ss += f[e] * f[e];
  }
#pragma unroll
  for (int o = LG / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const float inv = 1.f / sqrtf(ss / size + eps);
  if (!live) return;
#pragma unroll 4
  for (int c = lane * V; c < size; c += LG * V) {
    float f[V], z[V];
    load_vec<T, V>(a + c, f);
    load_vec<T, V>(gt + c, z);
#pragma unroll
    for (int e = 0; e < V; e++) f[e] = f[e] * inv * wg[c + e] * (sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-z[e])) : sigmoid_f(z[e]));
    store_vec<T, V>(out + it * size + c, f);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) k_gated_mlp(const T* __restrict__ gu, T* __restrict__ act, long long n, int ffp) {
  pdl_trigger();
  pdl_wait();
  constexpr int V = VecN<T>::n;
  const long long i = ((long long)blockIdx.x * 256 + threadIdx.x) * V;
  if (i >= n) return;
  const long long row = i / ffp;
  const int j = (int)(i % ffp);
  const T* src = gu + row * 2 * ffp + (j >> 5) * 64 + (j & 31);
  float a[V], b[V];
  load_vec<T, V>(src, a);
  load_vec<T, V>(src + 32, b);
#pragma unroll
  for (int e = 0; e < V; e++) a[e] = a[e] * sigmoid_f(a[e]) * b[e];
  store_vec<T, V>(act + i, a);
}

template <typename T>
__global__ void __launch_bounds__(256) k_pack_rows(const float* __restrict__ src, long long n, int cols, T* __restrict__ dst, long long ldd,
                                                   int dst_row, int group, int step) {
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= n) return;
  const int r = (int)(i / cols), c = (int)(i % cols);
  dst[(long long)(dst_row + (r / group) * step + r % group) * ldd + c] = from_f<T>(src[i]);
}

template <typename T>
__global__ void __launch_bounds__(256) k_pack_transposed(const float* __restrict__ src, long long n, int rows, int cols, T* __restrict__ dst,
                                                         int ld_rows, int ld_cols) {
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= n) return;
  const int c = (int)(i % cols), r = (int)(i / cols % rows);
  const long long b = i / cols / rows;
  dst[(b * ld_cols + c) * ld_rows + r] = from_f<T>(src[i]);
}

// C[m][n] = sum_k X[m][k] W[n][k] for a few rows, any size: one warp per output column.  GATED: column n is
// silu(row n of the gate weights) * row n of the up weights, which alternate in groups of 32 rows.
constexpr int RL_ROWS = 8;
template <typename T, bool GATED>
__global__ void __launch_bounds__(256) k_rows_linear(const T* __restrict__ X, long long ldx, const T* __restrict__ W, long long ldw,
                                                     void* __restrict__ C, long long ldc, int M, int N, int K, int f32_out, const RowsOut out) {
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n = blockIdx.x * 8 + warp;
  if (n >= N) return;
  const T* wr = W + (long long)(GATED ? (n >> 5) * 64 + (n & 31) : n) * ldw;
  float acc[RL_ROWS] = {}, up[RL_ROWS] = {};
  for (int k = lane; k < K; k += 32) {
    const float w = to_f<T>(wr[k]), u = GATED ? to_f<T>(wr[32 * ldw + k]) : 0.f;
#pragma unroll
    for (int m = 0; m < RL_ROWS; m++)
      if (m < M) {
        const float x = to_f<T>(X[m * ldx + k]);
        acc[m] = fmaf(x, w, acc[m]);
        if (GATED) up[m] = fmaf(x, u, up[m]);
      }
  }
#pragma unroll
  for (int m = 0; m < RL_ROWS; m++) {
    if (m >= M) break;
    float v = warp_sum(acc[m]);
    if (GATED) v = v * sigmoid_f(v) * warp_sum(up[m]);
    if (lane == 0) {
      if (out.bias) v += out.bias[n];
      if (out.softcap != 0.f) v = out.softcap * tanhf(v / out.softcap);
      if (out.n2 && n >= out.n2) reinterpret_cast<T*>(out.C2)[(m / out.T2) * out.stride2 + (m % out.T2) * out.ld2 + n - out.n2] = from_f<T>(v);
      else if (f32_out) reinterpret_cast<float*>(C)[m * ldc + n] = v;
      else reinterpret_cast<T*>(C)[m * ldc + n] = from_f<T>(v);
    }
  }
}

// The same in bf16 as a stream of the weights through the tensor cores: a block owns 16 output columns (32 weight rows when
// GATED), its eight warps share K.  The weights are the 16-row operand, the rows of X the 8-column operand, so every
// weight is loaded once, straight into the fragment that uses it: a lane takes 16 consecutive bytes of a row, and since X
// is read in the same order the permutation of K inside a step does not matter.  The first weights are on their way
// before the kernel waits for its predecessor.  LISTS: the rows of a block are one list of k_moe_choose_few, its weights those
// of the list's expert.
template <int NT, bool GATED, bool LISTS>
__global__ void __launch_bounds__(256) k_rows_mma(const bf16* __restrict__ X, long long ldx, const bf16* __restrict__ W, long long ldw,
                                                  void* __restrict__ C, long long ldc, int M, int N, int K, int epi, const RowsBatch bt) {
  pdl_trigger();
  const int* list = nullptr;
  if constexpr (LISTS) {
    pdl_wait();
    if ((int)blockIdx.y >= bt.lists[0]) return;
    const int* g = bt.lists + 1 + 3 * blockIdx.y;
    W += g[0] * bt.w;
    list = bt.lists + 1 + 3 * bt.max_lists + g[1];
    M = g[2];
  } else {
    X += blockIdx.y * bt.x;
    W += blockIdx.y * bt.w;
  }
  constexpr int RT = GATED ? 2 : 1, U = 4;      // U steps of 256 k are loaded ahead
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c8 = (lane & 3) * 8;
  const int n0 = blockIdx.x * 16;
  const bf16* wp[2 * RT];
#pragma unroll
  for (int i = 0; i < 2; i++) {
    const int n = min(n0 + g + 8 * i, N - 1), r = GATED ? (n >> 5) * 64 + (n & 31) : n;
    wp[i] = W + (long long)r * ldw;
    if (GATED) wp[2 + i] = W + (long long)(r + 32) * ldw;
  }
  const uint4 zero = make_uint4(0, 0, 0, 0);
  uint4 w[U][2 * RT];
  auto fetch = [&](int u, int k) {
#pragma unroll
    for (int i = 0; i < 2 * RT; i++) w[u][i] = k < K ? __ldg(reinterpret_cast<const uint4*>(wp[i] + k)) : zero;
  };
  const int kb = warp * 32 + c8;
#pragma unroll
  for (int u = 0; u < U; u++) fetch(u, kb + u * 256);
  if (!LISTS) pdl_wait();
  const bf16* xp[NT];          // this lane's rows of X
#pragma unroll
  for (int t = 0; t < NT; t++) {
    const int m = 8 * t + g;
    xp[t] = X + (m < M ? (LISTS ? list[m] / bt.x_div : m) : 0) * ldx;
  }
  float acc[RT][NT][4] = {};
  for (int k0 = kb; k0 < K + c8; k0 += U * 256) {       // the four lanes of a row leave together
#pragma unroll
    for (int u = 0; u < U; u++) {
      const int k = k0 + u * 256;
      uint4 x[NT];
#pragma unroll
      for (int t = 0; t < NT; t++) x[t] = k < K && 8 * t + g < M ? *reinterpret_cast<const uint4*>(xp[t] + k) : zero;
#pragma unroll
      for (int i = 0; i < RT; i++)
#pragma unroll
        for (int t = 0; t < NT; t++) {
          float* d = acc[i][t];
          const uint4 a = w[u][2 * i], b = w[u][2 * i + 1];
          asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                       : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a.x), "r"(b.x), "r"(a.y), "r"(b.y), "r"(x[t].x), "r"(x[t].y));
          asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                       : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a.z), "r"(b.z), "r"(a.w), "r"(b.w), "r"(x[t].z), "r"(x[t].w));
        }
      fetch(u, k + U * 256);
    }
  }
  // sum over the warps in order
  __shared__ float red[8][RT][8 * NT][16 + 1];
#pragma unroll
  for (int i = 0; i < RT; i++)
#pragma unroll
    for (int t = 0; t < NT; t++)
#pragma unroll
      for (int e = 0; e < 4; e++) red[warp][i][8 * t + 2 * (lane & 3) + (e & 1)][g + 8 * (e >> 1)] = acc[i][t][e];
  __syncthreads();
  for (int o = threadIdx.x; o < 16 * 8 * NT; o += 256) {
    const int m = o >> 4, j = o & 15;
    if (m >= M || n0 + j >= N) continue;
    float v = 0.f, up = 0.f;
#pragma unroll
    for (int i = 0; i < 8; i++) { v += red[i][0][m][j]; if (GATED) up += red[i][RT - 1][m][j]; }
    if (GATED) v = v * sigmoid_f(v) * up;
    if (bt.gate) v *= sigmoid_f(__bfloat162float(bt.gate[m * bt.ld_gate + blockIdx.y]));
    const int n = n0 + j;
    const RowsOut& out = bt.out;
    if (out.bias) v += out.bias[n];
    if (out.softcap != 0.f) v = out.softcap * tanhf(v / out.softcap);
    if (epi == EPI_RELU2) { v = fmaxf(v, 0.f); v *= v; }
    if (out.n2 && n >= out.n2) {
      reinterpret_cast<bf16*>(out.C2)[(m / out.T2) * out.stride2 + (m % out.T2) * out.ld2 + n - out.n2] = __float2bfloat16_rn(v);
      continue;
    }
    const long long at = LISTS ? list[m] * ldc + n : m * ldc + blockIdx.y * bt.c + n;
    if (epi == EPI_F32) reinterpret_cast<float*>(C)[at] = v;
    else reinterpret_cast<bf16*>(C)[at] = __float2bfloat16_rn(v);
  }
}

}  // namespace

template <typename T>
int DecStream<T>::embed(const T* table, const int* tokens, int ld_tok, int B, int T_, int base, int vocab, float scale, float* x,
                        const NextNorms<T>& n, int d, float eps, unsigned int* status, cudaStream_t s) {
  CUDA_TRY(launch_dependent(k_dec_embed<T>, B * T_, RT, 0, s, table, tokens, ld_tok, T_, base, vocab, scale, x, n, d, eps, status));
  KERNEL_CHECK();
  return 0;
}
template <typename T>
int DecStream<T>::parallel_resid(float* x, const T* y, const T* y2, const MoeRows& m, const NextNorms<T>& n, int rows, int d, float eps,
                                 cudaStream_t s) {
  bool vec = (d & 3) == 0;
  for (const void* p : {(const void*)x, (const void*)y, (const void*)y2, m.out, (const void*)n.w, (const void*)n.h, (const void*)n.w2, (const void*)n.h2})
    vec = vec && aligned16(p);
  const int nv = vec ? cdiv(d, RT * 4) : 0;
#define LAUNCH(NV) CUDA_TRY(launch_dependent(k_parallel_resid<T, NV>, rows, RT, 0, s, x, y, y2, m, n, d, eps))
  if (nv == 1) LAUNCH(1);
  else if (nv == 2) LAUNCH(2);
  else if (nv == 3 || nv == 4) LAUNCH(4);
  else LAUNCH(0);
#undef LAUNCH
  KERNEL_CHECK();
  return 0;
}
template <typename T>
int DecStream<T>::resid_norm(float* x, const T* y, const float* w_post, float m, const float* w_pre, T* h, int rows, int d, float eps,
                             cudaStream_t s) {
  const bool vec = (d & 3) == 0 && aligned16(x) && aligned16(y) && aligned16(w_post) && (!h || (aligned16(w_pre) && aligned16(h)));
  const int nv = vec ? cdiv(d, RT * 4) : 0;
  if (nv == 1) CUDA_TRY(launch_dependent(k_resid_norm<T, 1>, rows, RT, 0, s, x, y, w_post, m, w_pre, h, d, eps));
  else if (nv == 2) CUDA_TRY(launch_dependent(k_resid_norm<T, 2>, rows, RT, 0, s, x, y, w_post, m, w_pre, h, d, eps));
  else if (nv == 3 || nv == 4) CUDA_TRY(launch_dependent(k_resid_norm<T, 4>, rows, RT, 0, s, x, y, w_post, m, w_pre, h, d, eps));
  else CUDA_TRY(launch_dependent(k_resid_norm<T, 0>, rows, RT, 0, s, x, y, w_post, m, w_pre, h, d, eps));
  KERNEL_CHECK();
  return 0;
}
template <typename T>
int DecStream<T>::gather_norm(const float* x, const int* want, int stride, const float* w, T* h, int n, int d, float eps, cudaStream_t s) {
  CUDA_TRY(launch_dependent(k_gather_norm<T>, n, RT, 0, s, x, want, stride, w, h, d, eps));
  KERNEL_CHECK();
  return 0;
}
template <typename T>
int DecStream<T>::gated_norm(const T* in, const float* w, bool w_all, const T* gate, long long ldg, T* out, int rows, int groups, int size,
                             float eps, cudaStream_t s) {
  const long long n = (long long)rows * groups;
  constexpr int V = VecN<T>::n;
  const bool vec = size % V == 0 && ldg % V == 0 && aligned16(in) && aligned16(gate) && aligned16(out);
#define LAUNCH(VV, LG) CUDA_TRY(launch_dependent(k_gated_norm<T, VV, LG>, cdiv(n, 256 / LG), 256, 0, s, in, w, (int)w_all, gate, ldg, out, n, groups, size, eps))
  if (!vec) LAUNCH(1, 32);
  else if (size <= 8 * V) LAUNCH(V, 8);
  else if (size <= 16 * V) LAUNCH(V, 16);
  else LAUNCH(V, 32);
#undef LAUNCH
  KERNEL_CHECK();
  return 0;
}
template <typename T> int DecStream<T>::gated_mlp(const T* gu, T* act, int rows, int ffp, cudaStream_t s) {
  const long long n = (long long)rows * ffp;
  CUDA_TRY(launch_dependent(k_gated_mlp<T>, cdiv(n, 256 * VecN<T>::n), 256, 0, s, gu, act, n, ffp));
  KERNEL_CHECK();
  return 0;
}
template struct DecStream<float>;
template struct DecStream<bf16>;

template <typename T>
int pack_rows(const float* src, int rows, int cols, T* dst, long long ldd, int dst_row, int group, int step, cudaStream_t s) {
  const long long n = (long long)rows * cols;
  k_pack_rows<T><<<cdiv(n, 256), 256, 0, s>>>(src, n, cols, dst, ldd, dst_row, group, step);
  KERNEL_CHECK();
  return 0;
}
template int pack_rows<float>(const float*, int, int, float*, long long, int, int, int, cudaStream_t);
template int pack_rows<bf16>(const float*, int, int, bf16*, long long, int, int, int, cudaStream_t);

// Up to ROWS_STREAM rows in bf16 with aligned operands (RL_ROWS otherwise) stream the weights; more rows are a GEMM.
int rows_stream(const bf16* X, long long ldx, const bf16* W, long long ldw, void* C, long long ldc, int M, int N, int K, int epi, int batch,
                const RowsBatch& bt, cudaStream_t s) {
  const dim3 grid(cdiv(N, 16), batch);
#define LAUNCH(NT) CUDA_TRY(bt.lists          ? launch_dependent(k_rows_mma<NT, false, true>, grid, 256, 0, s, X, ldx, W, ldw, C, ldc, M, N, K, epi, bt) \
                            : epi == EPI_SWIGLU ? launch_dependent(k_rows_mma<NT, true, false>, grid, 256, 0, s, X, ldx, W, ldw, C, ldc, M, N, K, epi, bt) \
                                                : launch_dependent(k_rows_mma<NT, false, false>, grid, 256, 0, s, X, ldx, W, ldw, C, ldc, M, N, K, epi, bt))
  if (M <= 8) LAUNCH(1);
  else if (M <= 16) LAUNCH(2);
  else LAUNCH(4);
#undef LAUNCH
  KERNEL_CHECK();
  return 0;
}

template <typename T>
int pack_transposed(const float* src, int batch, int rows, int cols, T* dst, int ld_rows, int ld_cols, cudaStream_t s) {
  const long long n = (long long)batch * rows * cols;
  k_pack_transposed<T><<<cdiv(n, 256), 256, 0, s>>>(src, n, rows, cols, dst, ld_rows, ld_cols);
  KERNEL_CHECK();
  return 0;
}
template int pack_transposed<float>(const float*, int, int, int, float*, int, int, cudaStream_t);
template int pack_transposed<bf16>(const float*, int, int, int, bf16*, int, int, cudaStream_t);

template <typename T>
int rows_linear(DecoderStack* d, const void* X, long long ldx, const void* W, long long ldw, void* C, long long ldc, int M, int N, int K,
                int epi, cudaStream_t s, const RowsOut& out) {
  const int f32 = epi == EPI_F32;
  if constexpr (sizeof(T) == 2)
    if (M <= ROWS_STREAM && ((K | ldx | ldw) & 7) == 0 && aligned16(X) && aligned16(W)) {
      RowsBatch bt;
      bt.out = out;
      return rows_stream((const bf16*)X, ldx, (const bf16*)W, ldw, C, ldc, M, N, K, epi, 1, bt, s);
    }
  if (M <= RL_ROWS) {
    if (epi == EPI_SWIGLU) CUDA_TRY(launch_dependent(k_rows_linear<T, true>, cdiv(N, 8), 256, 0, s, (const T*)X, ldx, (const T*)W, ldw, C, ldc, M, N, K, f32, out));
    else CUDA_TRY(launch_dependent(k_rows_linear<T, false>, cdiv(N, 8), 256, 0, s, (const T*)X, ldx, (const T*)W, ldw, C, ldc, M, N, K, f32, out));
    KERNEL_CHECK();
    return 0;
  }
  GemmArgs g;
  g.ws = d->gemm_ws; g.ws_bytes = d->gemm_ws_bytes; g.status = d->status;
  g.A = X; g.lda = ldx; g.a_kmajor = true; g.B = W; g.ldb = ldw; g.b_kmajor = true;
  g.C = C; g.ldc = ldc; g.M = M; g.N = N; g.K = K; g.epi = epi; g.beta = 0.f; g.any_size = true; g.bias = out.bias;
  if (out.n2) {      // two products: this part, and the rest as a batch over the columns of tokens
    g.N = out.n2;
    FEMTO_TRY(gemm<T>(g, s));
    g.B = (const T*)W + out.n2 * ldw; g.N = N - out.n2; g.M = out.T2; g.batch = M / out.T2; g.strideA = out.T2 * ldx;
    g.C = out.C2; g.ldc = out.ld2; g.strideC = out.stride2;
    if (g.bias) g.bias += out.n2;
    return gemm<T>(g, s);
  }
  if (epi != EPI_SWIGLU) {
    FEMTO_TRY(gemm<T>(g, s));
    return out.softcap != 0.f ? softcap_inplace((float*)C, (long long)M * ldc, s, out.softcap) : 0;
  }
  // g.N counts the weight rows, gate and up together; the result is half as wide
  g.N = 2 * N;
  if (sizeof(T) == 2 && gemm_tc_supported(g)) return gemm<T>(g, s);
  g.epi = EPI_STORE; g.C = d->gu; g.ldc = 2 * N;
  FEMTO_TRY(gemm<T>(g, s));
  return DecStream<T>::gated_mlp((const T*)d->gu, (T*)C, M, N, s);
}
template int rows_linear<float>(DecoderStack*, const void*, long long, const void*, long long, void*, long long, int, int, int, int, cudaStream_t, const RowsOut&);
template int rows_linear<bf16>(DecoderStack*, const void*, long long, const void*, long long, void*, long long, int, int, int, int, cudaStream_t, const RowsOut&);
