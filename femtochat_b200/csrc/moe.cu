// Mixture-of-experts feed-forward: every token goes to the `top` experts with the largest router logits, weighted by the
// softmax over those logits.  Many tokens: the rows are sorted by expert into runs of whole GEMM tiles, and each of the two
// products is one grouped GEMM.  A few tokens: one launch per product streams the weights of the experts that were chosen.
// A result row never depends on the order of the rows beside it, so the order inside a run does not matter.
#include <algorithm>

#include <limits.h>

#include "decoder.cuh"
#include "streaming.cuh"
#include "warp_mma.cuh"

namespace {

constexpr int MAX_EXPERTS = 1024, MAX_TOP = 32;

// By one warp: the k-th largest logit of a row (ties: the lower index) ends up in lane k, as index and softmax weight.
template <int PER>
__device__ __forceinline__ void choose(const float* __restrict__ z, const float* __restrict__ bias, int experts, int top, int lane, int& id,
                                       float& weight) {
  float v[PER];
#pragma unroll
  for (int i = 0; i < PER; i++) {
    const int e = lane + 32 * i;
    v[i] = e < experts ? z[e] + bias[e] : -INFINITY;
  }
  float mine = -INFINITY, first = 0.f;
  id = 0;
  for (int k = 0; k < top; k++) {
    float best = -INFINITY;
    int at = INT_MAX;
#pragma unroll
    for (int i = 0; i < PER; i++)
      if (v[i] > best) { best = v[i]; at = lane + 32 * i; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oa = __shfl_xor_sync(0xffffffffu, at, o);
      if (ov > best || (ov == best && oa < at)) { best = ov; at = oa; }
    }
    if (at == INT_MAX) at = k;       // only when logits are not finite
    if (k == 0) first = best;
    if (lane == k) { mine = best; id = at; }
#pragma unroll
    for (int i = 0; i < PER; i++) if (at == lane + 32 * i) v[i] = -INFINITY;
  }
  const float p = lane < top ? expf(mine - first) : 0.f;
  weight = p / warp_sum(p);
}

// The choices of a block's TOPK_ROWS rows (logits z with pitch ldz, of these rows): weights, experts, and every choice's place
// among the rows of its expert.  By 256 threads.
constexpr int TOPK_ROWS = 32;
template <int PER>
__device__ __forceinline__ void choose_rows(const MoeArgs& a, const float* z, long long ldz) {
  __shared__ int count[32 * PER];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int e = threadIdx.x; e < a.experts; e += 256) count[e] = 0;
  __syncthreads();
  int id[TOPK_ROWS / 8], at[TOPK_ROWS / 8];
#pragma unroll
  for (int i = 0; i < TOPK_ROWS / 8; i++) {
    const long long row = (long long)blockIdx.x * TOPK_ROWS + i * 8 + warp;
    id[i] = -1;
    if (row >= a.rows) continue;
    float w;
    int e;
    choose<PER>(z + (i * 8 + warp) * ldz, a.bias, a.experts, a.top, lane, e, w);
    if (lane < a.top) {
      a.weight[row * a.top + lane] = w;
      id[i] = e;
      at[i] = atomicAdd(&count[e], 1);
    }
  }
  __syncthreads();
  for (int e = threadIdx.x; e < a.experts; e += 256) { const int n = count[e]; count[e] = n ? atomicAdd(&a.counts[e], n) : 0; }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < TOPK_ROWS / 8; i++) {
    if (id[i] < 0) continue;
    const long long pair = ((long long)blockIdx.x * TOPK_ROWS + i * 8 + warp) * a.top + lane;
    a.expert[pair] = id[i];
    a.slot[pair] = count[id[i]] + at[i];      // place among the expert's rows
  }
}

template <int PER>
__global__ void __launch_bounds__(256) k_moe_choose(const MoeArgs a) {
  pdl_trigger();
  pdl_wait();
  choose_rows<PER>(a, a.z + (long long)blockIdx.x * TOPK_ROWS * a.ldz, a.ldz);
}

// Router and choice in one launch, bf16 rows and at most 8 NT experts: 32 rows per block, two tiles of 16 rows by four parts of
// the channels.  Rows and weights go straight from global memory into the fragments: a lane takes 16 consecutive bytes of
// each, and since both are read in the same order the permutation of the channels inside a step does not matter.
template <int NT>
__global__ void __launch_bounds__(256) k_moe_route(const MoeArgs a) {
  pdl_trigger();
  constexpr int ZP = 8 * NT + 1;
  __shared__ float z[4][TOPK_ROWS][ZP];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c2 = 2 * (lane & 3);
  const int rt = warp & 1, part = warp >> 1, K = a.width;
  const long long row = (long long)blockIdx.x * TOPK_ROWS + rt * 16 + g;
  const bf16* h = reinterpret_cast<const bf16*>(a.h);
  const bf16 *x0 = h + min(row, (long long)a.rows - 1) * K, *x1 = h + min(row + 8, (long long)a.rows - 1) * K;
  const bf16* w = reinterpret_cast<const bf16*>(a.router);
  const uint4 zero = make_uint4(0, 0, 0, 0);
  pdl_wait();
  float acc[NT][4] = {};
#pragma unroll 4
  for (int k0 = part * 32; k0 < K; k0 += 128) {
    const int k = k0 + (lane & 3) * 8;
    const uint4 p = k < K ? *reinterpret_cast<const uint4*>(x0 + k) : zero, q = k < K ? *reinterpret_cast<const uint4*>(x1 + k) : zero;
    const uint32_t lo[4] = {p.x, q.x, p.y, q.y}, hi[4] = {p.z, q.z, p.w, q.w};
#pragma unroll
    for (int t = 0; t < NT; t++) {
      const uint4 b = k < K && 8 * t + g < a.experts ? __ldg(reinterpret_cast<const uint4*>(w + (long long)(8 * t + g) * K + k)) : zero;
      mma16816(acc[t], lo, b.x, b.y);
      mma16816(acc[t], hi, b.z, b.w);
    }
  }
#pragma unroll
  for (int t = 0; t < NT; t++)
#pragma unroll
    for (int e = 0; e < 4; e++) z[part][rt * 16 + g + 8 * (e >> 1)][8 * t + c2 + (e & 1)] = acc[t][e];
  __syncthreads();
  for (int i = threadIdx.x; i < TOPK_ROWS * 8 * NT; i += 256) {
    const int r = i / (8 * NT), c = i % (8 * NT);
    z[0][r][c] = (z[0][r][c] + z[1][r][c]) + (z[2][r][c] + z[3][r][c]);
  }
  __syncthreads();
  choose_rows<(NT + 3) / 4>(a, &z[0][0][0], ZP);
}

// Places every (row, choice) pair: slot = start of its expert's run + place, and the row's input is copied there.  Every block
// works out the starts from the counts; block 0 writes the list of runs for the GEMM.
constexpr int PLACE_PAIRS = 64;
template <typename T, int V>
__global__ void __launch_bounds__(256) k_moe_place(const MoeArgs a) {
  pdl_trigger();
  pdl_wait();
  __shared__ int start[MAX_EXPERTS];
  __shared__ int sums[8];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  int runs[4], mine = 0;
#pragma unroll
  for (int i = 0; i < 4; i++) {
    const int e = tid * 4 + i;
    runs[i] = e < a.experts ? (a.counts[e] + a.group_rows - 1) / a.group_rows : 0;
    mine += runs[i];
  }
  int inc = mine;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) { const int up = __shfl_up_sync(0xffffffffu, inc, o); if (lane >= o) inc += up; }
  if (lane == 31) sums[warp] = inc;
  __syncthreads();
  int at = inc - mine, total = 0;
#pragma unroll
  for (int i = 0; i < 8; i++) { if (i < warp) at += sums[i]; total += sums[i]; }
#pragma unroll
  for (int i = 0; i < 4; i++) {
    const int e = tid * 4 + i;
    if (e >= a.experts) break;
    start[e] = at * a.group_rows;
    if (blockIdx.x == 0) for (int r = 0; r < runs[i]; r++) a.groups[1 + at + r] = e;
    at += runs[i];
  }
  if (blockIdx.x == 0 && tid == 0) a.groups[0] = total;
  __syncthreads();
  const long long pairs = (long long)a.rows * a.top;
  for (int i = warp; i < PLACE_PAIRS; i += 8) {
    const long long pair = (long long)blockIdx.x * PLACE_PAIRS + i;
    if (pair >= pairs) break;
    const int slot = start[a.expert[pair]] + a.slot[pair];
    __syncwarp();
    if (lane == 0) a.slot[pair] = slot;
    const T* src = reinterpret_cast<const T*>(a.h) + pair / a.top * a.width;
    T* dst = reinterpret_cast<T*>(a.xs) + (long long)slot * a.width;
    if constexpr (V > 1) {
#pragma unroll 4
      for (int c = lane * V; c < a.width; c += 32 * V) *reinterpret_cast<uint4*>(dst + c) = *reinterpret_cast<const uint4*>(src + c);
    } else {
      for (int c = lane; c < a.width; c += 32) dst[c] = src[c];
    }
  }
}

// A few rows, one block: the choices, and for every expert that was chosen the list of its pairs.
template <int PER>
__global__ void __launch_bounds__(1024) k_moe_choose_few(const MoeArgs a) {
  pdl_trigger();
  __shared__ int id[ROWS_STREAM * MAX_TOP];
  __shared__ int cursor[2];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, pairs = a.rows * a.top;
  if (tid < 2) cursor[tid] = 0;
  pdl_wait();
  if (warp < a.rows) {
    float w;
    int e;
    choose<PER>(a.z + (long long)warp * a.ldz, a.bias, a.experts, a.top, lane, e, w);
    if (lane < a.top) { a.weight[warp * a.top + lane] = w; id[warp * a.top + lane] = e; }
  }
  __syncthreads();
  if (tid < a.experts) {
    int n = 0;
    for (int p = 0; p < pairs; p++) n += id[p] == tid;
    if (n) {
      const int y = atomicAdd(&cursor[0], 1);
      int at = atomicAdd(&cursor[1], n);
      int* g = a.lists + 1 + 3 * y;
      g[0] = tid; g[1] = at; g[2] = n;
      int* list = a.lists + 1 + 3 * a.max_lists;
      for (int p = 0; p < pairs; p++) if (id[p] == tid) list[at++] = p;
    }
  }
  __syncthreads();
  if (tid == 0) a.lists[0] = cursor[0];
}

// y[row] = sum over its choices of weight * result
template <typename T>
__global__ void __launch_bounds__(256) k_moe_combine(const MoeRows m, T* __restrict__ y, int d) {
  pdl_trigger();
  pdl_wait();
  const long long row = blockIdx.x;
  for (int c = threadIdx.x; c < d; c += 256) {
    float v = 0.f;
    for (int k = 0; k < m.top; k++) {
      const long long p = row * m.top + k;
      v = fmaf(m.weight[p], to_f<T>(reinterpret_cast<const T*>(m.out)[(m.slot ? m.slot[p] : p) * (long long)d + c]), v);
    }
    y[row * d + c] = from_f<T>(v);
  }
}

}  // namespace

bool moe_supported(int experts, int top) { return experts > 0 && experts <= MAX_EXPERTS && top > 0 && top <= experts && top <= MAX_TOP; }
int moe_group_rows(long long rows, int experts, int top) { return rows * top >= 192LL * experts ? 256 : 128; }
long long moe_max_slots(long long rows, int experts, int top, int group_rows) {
  return ((rows * top + group_rows - 1) / group_rows + std::min<long long>(experts, rows * top)) * group_rows;
}

#define DISPATCH_PER(experts, LAUNCH) \
  if (experts <= 32) LAUNCH(1); \
  else if (experts <= 64) LAUNCH(2); \
  else if (experts <= 128) LAUNCH(4); \
  else if (experts <= 256) LAUNCH(8); \
  else LAUNCH(32)

template <typename T> int moe_sort(const MoeArgs& a, cudaStream_t s) {
  constexpr int V = VecN<T>::n;
  FEMTO_TRY(fill_zero(a.counts, 4 * (size_t)a.experts, s));
  const int choosers = cdiv(a.rows, TOPK_ROWS);
  if (a.router) {
#define LAUNCH(NT) CUDA_TRY(launch_dependent(k_moe_route<NT>, choosers, 256, 0, s, a))
    if (a.experts <= 8) LAUNCH(1);
    else if (a.experts <= 16) LAUNCH(2);
    else if (a.experts <= 32) LAUNCH(4);
    else LAUNCH(8);
#undef LAUNCH
  } else {
#define LAUNCH(PER) CUDA_TRY(launch_dependent(k_moe_choose<PER>, choosers, 256, 0, s, a))
    DISPATCH_PER(a.experts, LAUNCH);
#undef LAUNCH
  }
  KERNEL_CHECK();
  const int blocks = cdiv((long long)a.rows * a.top, PLACE_PAIRS);
  if (a.width % V == 0 && aligned16(a.h) && aligned16(a.xs)) CUDA_TRY(launch_dependent(k_moe_place<T, V>, blocks, 256, 0, s, a));
  else CUDA_TRY(launch_dependent(k_moe_place<T, 1>, blocks, 256, 0, s, a));
  KERNEL_CHECK();
  return 0;
}
template int moe_sort<float>(const MoeArgs&, cudaStream_t);
template int moe_sort<bf16>(const MoeArgs&, cudaStream_t);

int moe_choose_few(const MoeArgs& a, cudaStream_t s) {
#define LAUNCH(PER) CUDA_TRY(launch_dependent(k_moe_choose_few<PER>, 1, 1024, 0, s, a))
  DISPATCH_PER(a.experts, LAUNCH);
#undef LAUNCH
  KERNEL_CHECK();
  return 0;
}

template <typename T> int moe_combine(const MoeRows& m, T* y, int rows, int d, cudaStream_t s) {
  CUDA_TRY(launch_dependent(k_moe_combine<T>, rows, 256, 0, s, m, y, d));
  KERNEL_CHECK();
  return 0;
}
template int moe_combine<float>(const MoeRows&, float*, int, int, cudaStream_t);
template int moe_combine<bf16>(const MoeRows&, bf16*, int, int, cudaStream_t);
