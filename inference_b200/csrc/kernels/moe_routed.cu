// Mixture-of-experts feed-forward: routing plans, from a table or from router logits, and the small-batch grouped GEMM.
//
// moe_route_kernel / moe_layout_kernel: softmax over a token's router logits (fp32), the `top` largest (as they are, or divided by their sum), and their places in an
// expert-sorted buffer of the same two layouts as below. Small steps do it in one launch (the last CTA to finish lays the pairs
// out); large ones lay out in a second, which also copies the rows to their places. The counters clean up after themselves.
//
// moe_table_plan_kernel: a router without arithmetic. A table [vocab, top] names each token id's experts, so the token ids
// of a step fix the routing of every layer before the first one starts: one launch plans all layers (one CTA each).
// Per layer the (token, slot) pairs are counted and laid out expert by expert; with `pad` = 128 every expert's segment is
// padded to the row tile of the tcgen05 grouped GEMM and tile_group[] names each tile's expert, with `pad` = 1 the
// segments are dense and the active experts are listed for the kernel below.
//
// grouped_rows_kernel: out[r] = act(x[src[r]] W[e]^T) for the rows r of expert e's segment, few rows per expert: weight
// streaming, so every weight row is read once per 8 * NT tokens with 16-byte loads straight into mma.sync fragments.
// The reduction index may be visited in any order as long as both operands agree: lane t4 of a row takes the eight
// consecutive elements 8 t4 .. 8 t4 + 7 of each 32-wide slab and feeds them to two MMAs as if they were the fragment
// columns, for weights and tokens alike. Eight warps take slabs in turn; partial sums meet in shared memory.
#include "common.cuh"
#include "gemm_tcgen05.cuh"

namespace swb {

SWB_REGISTER_STATUS_UNIT(moe_routed);

namespace {

__global__ void __launch_bounds__(1024) moe_table_plan_kernel(const long long* __restrict__ ids, int T,
                                                              const int* __restrict__ tables, int vocab, int top, int E,
                                                              int pad, int* dest, int* src, int* offsets, int* active,
                                                              int* tile_group, int rows_cap) {
  // No early trigger here: the kernels of the step start after this grid has finished, so the grouped kernels may read the
  // plan before they wait for the rows they multiply. (Prefetching the weight rows into L2 there as well was slower.)
  pdl_wait();
  extern __shared__ int sm[];
  int* count = sm;          // [E] pairs per expert, then the write cursor
  int* start = sm + E;      // [E + 1] first row of each expert's segment
  __shared__ int n_active;
  const int layer = blockIdx.x, pairs = T * top;
  const int* table = tables + (size_t)layer * vocab * top;
  dest += (size_t)layer * pairs;
  if (src) src += (size_t)layer * rows_cap;
  offsets += (size_t)layer * (E + 1);
  const int n_act_cap = min(E, pairs), n_tiles = rows_cap / 128;
  if (active) active += (size_t)layer * n_act_cap;
  if (tile_group) tile_group += (size_t)layer * n_tiles;
  for (int e = threadIdx.x; e < E; e += blockDim.x) count[e] = 0;
  if (threadIdx.x == 0) n_active = 0;
  __syncthreads();
  const int lane = threadIdx.x & 31;
  auto expert_of = [&](int pair) {
    const long long id = ids[pair / top];
    const long long row = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
    return min(max(__ldg(table + row * top + pair % top), 0), E - 1);
  };
  // equal experts of a warp are added with one shared-memory atomic
  const int rounds = (pairs + blockDim.x - 1) / blockDim.x;
  for (int r = 0; r < rounds; ++r) {
    const int pair = r * blockDim.x + threadIdx.x;
    const int e = pair < pairs ? expert_of(pair) : -1;
    const unsigned same = __match_any_sync(0xffffffffu, e);
    if (e >= 0 && lane == __ffs(same) - 1) atomicAdd(&count[e], __popc(same));
  }
  __syncthreads();
  if (threadIdx.x < 32) {   // exclusive scan of the (padded) counts by one warp
    int carry = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + lane;
      const int n = e < E ? (count[e] + pad - 1) / pad * pad : 0;
      int s = n;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int y = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s += y;
      }
      if (e < E) start[e] = carry + s - n;
      carry += __shfl_sync(0xffffffffu, s, 31);
    }
    if (lane == 0) start[E] = carry;
  }
  __syncthreads();
  for (int e = threadIdx.x; e <= E; e += blockDim.x) offsets[e] = start[e];
  if (tile_group) {
    for (int i = threadIdx.x; i < n_tiles; i += blockDim.x) {
      int lo = 0, hi = E;   // the expert whose segment holds row 128 i
      while (lo < hi) {
        const int mid = (lo + hi) >> 1;
        if (start[mid + 1] <= i * 128) lo = mid + 1;
        else hi = mid;
      }
      tile_group[i] = lo < E ? lo : -1;
    }
  }
  if (active) {
    for (int e = threadIdx.x; e < E; e += blockDim.x)
      if (count[e] > 0) active[atomicAdd(&n_active, 1)] = e;
    __syncthreads();
    for (int i = n_active + threadIdx.x; i < n_act_cap; i += blockDim.x) active[i] = -1;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) count[e] = start[e];
  __syncthreads();
  for (int r = 0; r < rounds; ++r) {
    const int pair = r * blockDim.x + threadIdx.x;
    const int e = pair < pairs ? expert_of(pair) : -1;
    const unsigned same = __match_any_sync(0xffffffffu, e);
    int base = 0;
    const int leader = __ffs(same) - 1;
    if (e >= 0 && lane == leader) base = atomicAdd(&count[e], __popc(same));
    base = __shfl_sync(0xffffffffu, base, leader);
    if (e >= 0) {
      const int row = base + __popc(same & ((1u << lane) - 1));
      dest[pair] = row;
      if (src) src[row] = pair / top;
    }
  }
}

struct RouteParams {
  const float* logits;       // [T, ld]
  int ld, T, E, top, pad;
  int* expert;               // [T * top]
  int* rank;                 // [T * top] place of the pair among those of its expert
  float* weights;            // [T * top] softmax scores
  int renorm;                // 1: divided by the sum of the chosen ones
  int* counters;             // [E + 2] pairs per expert, two tickets; zero between launches
  int* dest;                 // [T * top]
  int* src;                  // optional [rows_cap]
  int* offsets;              // [E + 1]
  int* active;               // optional [min(E, T * top)]
  int* tile_group;           // optional [rows_cap / 128]
  int rows_cap;
  const uint4* rows_in;      // optional: row t goes to row dest[t, k] of rows_out, 16-byte pieces
  uint4* rows_out;
  long long ld_in, ld_out;
  int pieces;
};

// First row of every expert's (padded) segment from the counts, by the whole block; start [E + 1] in shared memory.
__device__ __forceinline__ void segment_starts(const RouteParams& p, int* start) {
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    int carry = 0;
    for (int e0 = 0; e0 < p.E; e0 += 32) {
      const int e = e0 + lane;
      const int n = e < p.E ? (__ldcg(p.counters + e) + p.pad - 1) / p.pad * p.pad : 0;
      int s = n;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int y = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s += y;
      }
      if (e < p.E) start[e] = carry + s - n;
      carry += __shfl_sync(0xffffffffu, s, 31);
    }
    if (lane == 0) start[p.E] = carry;
  }
  __syncthreads();
}

// What one block writes about the segments as a whole.
__device__ __forceinline__ void describe_segments(const RouteParams& p, const int* start) {
  for (int e = threadIdx.x; e <= p.E; e += blockDim.x) p.offsets[e] = start[e];
  if (p.tile_group) {
    for (int i = threadIdx.x; i < p.rows_cap / 128; i += blockDim.x) {
      int lo = 0, hi = p.E;
      while (lo < hi) {
        const int mid = (lo + hi) >> 1;
        if (start[mid + 1] <= i * 128) lo = mid + 1;
        else hi = mid;
      }
      p.tile_group[i] = lo < p.E ? lo : -1;
    }
  }
  if (p.active) {
    __shared__ int n_active;
    if (threadIdx.x == 0) n_active = 0;
    __syncthreads();
    for (int e = threadIdx.x; e < p.E; e += blockDim.x)
      if (__ldcg(p.counters + e) > 0) p.active[atomicAdd(&n_active, 1)] = e;
    __syncthreads();
    for (int i = n_active + threadIdx.x; i < min(p.E, p.T * p.top); i += blockDim.x) p.active[i] = -1;
  }
}

__device__ __forceinline__ void place_pair(const RouteParams& p, const int* start, int pair) {
  const int row = start[__ldcg(p.expert + pair)] + __ldcg(p.rank + pair);
  p.dest[pair] = row;
  if (p.src) p.src[row] = pair / p.top;
}

// One warp per token. Ties go to the lower expert number. WHOLE: the last block to finish also lays the pairs out.
template <bool WHOLE>
__global__ void __launch_bounds__(256) moe_route_kernel(const RouteParams p) {
  pdl_wait();
  extern __shared__ int route_start[];
  const int lane = threadIdx.x & 31, t = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (t < p.T) {
    const float* z = p.logits + (size_t)t * p.ld;
    float top = -INFINITY, sum = 0.f;
    for (int e = lane; e < p.E; e += 32) top = fmaxf(top, z[e]);
    top = warp_max(top);
    for (int e = lane; e < p.E; e += 32) sum += expf(z[e] - top);
    sum = warp_sum(sum);
    float last = INFINITY, mine = 0.f;      // lane k mod 32 keeps choice k until 32 of them (or all) are filed together
    int last_e = -1, mine_e = 0;
    float chosen = 0.f;                     // sum of the chosen scores, times `sum`
    for (int k = 0; k < p.top; ++k) {
      float best = -INFINITY;
      int best_e = p.E;
      for (int e = lane; e < p.E; e += 32) {
        const float v = z[e];
        const bool after = v < last || (v == last && e > last_e);     // not taken yet: what follows the last one in order
        if (after && (v > best || best_e == p.E)) best = v, best_e = e;
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float v = __shfl_xor_sync(0xffffffffu, best, o);
        const int e = __shfl_xor_sync(0xffffffffu, best_e, o);
        if (e < p.E && (best_e == p.E || v > best || (v == best && e < best_e))) best = v, best_e = e;
      }
      last = best, last_e = best_e;
      chosen += expf(best - top);
      if (lane == (k & 31)) mine = best, mine_e = min(best_e, p.E - 1);     // logits that are not numbers: any expert
      if ((k & 31) == 31 || k == p.top - 1) {
        const int pair = t * p.top + (k & ~31) + lane;
        if (lane <= (k & 31)) {
          p.expert[pair] = mine_e;
          p.weights[pair] = expf(mine - top) / sum;
          p.rank[pair] = atomicAdd(p.counters + mine_e, 1);
        }
      }
    }
    if (p.renorm) {
      __syncwarp();
      const float share = chosen / sum + 1e-20f;
      for (int k = lane; k < p.top; k += 32) p.weights[t * p.top + k] /= share;      // written by this lane above
    }
  }
  if constexpr (WHOLE) {
    __shared__ int is_last;
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) is_last = atomicAdd(p.counters + p.E, 1) == (int)gridDim.x - 1;
    __syncthreads();
    if (!is_last) return;
    __threadfence();
    segment_starts(p, route_start);
    describe_segments(p, route_start);
    for (int pair = threadIdx.x; pair < p.T * p.top; pair += blockDim.x) place_pair(p, route_start, pair);
    __syncthreads();
    for (int e = threadIdx.x; e < p.E + 1; e += blockDim.x) p.counters[e] = 0;
  }
}

// Lays out the pairs of a large step, a warp per pair, and copies each token's row to its places.
__global__ void __launch_bounds__(256) moe_layout_kernel(const RouteParams p) {
  pdl_wait();
  extern __shared__ int layout_start[];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, pairs = p.T * p.top;
  segment_starts(p, layout_start);
  if (blockIdx.x == 0) describe_segments(p, layout_start);
  for (int pair = blockIdx.x * 8 + warp; pair < pairs; pair += gridDim.x * 8) {
    if (lane == 0) place_pair(p, layout_start, pair);
    if (p.rows_out) {
      const int row = layout_start[p.expert[pair]] + p.rank[pair];
      const uint4* from = p.rows_in + (size_t)(pair / p.top) * p.ld_in;
      uint4* to = p.rows_out + (size_t)row * p.ld_out;
      for (int i = lane; i < p.pieces; i += 32) to[i] = __ldg(from + i);
    }
  }
  __syncthreads();
  __shared__ int is_last;
  if (threadIdx.x == 0) is_last = atomicAdd(p.counters + p.E + 1, 1) == (int)gridDim.x - 1;     // every block has read the counts
  __syncthreads();
  if (!is_last) return;
  for (int e = threadIdx.x; e < p.E + 2; e += blockDim.x) p.counters[e] = 0;
}

constexpr int GR_WARPS = 8;

__device__ __forceinline__ void mma16816(float* c, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint4 ldg_stream(const bf16* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}

struct GroupedRowsParams {
  const bf16* x;
  int ldx;
  const int* src;        // optional: row of x for segment row r (default: r)
  const int* offsets;    // [E + 1]
  const int* active;     // experts with rows; < 0 = none
  const bf16* w;         // [E, N, K]
  bf16* out;
  int ldo, N, K, act;    // act may be a gated pair: rows of w in (gate, up) pairs, out [*, N / 2]
  float act_a;           // its parameter
  int plan_ahead;        // the plan was complete before the kernel in front of this one started
};

// One pass over the CTA's 16 * MT weight rows for up to 8 * NT token rows [r0, r0 + n).
template <int MT, int NT>
__device__ __forceinline__ void grouped_pass(const GroupedRowsParams& p, const bf16* wrow, int f0, int r0, int n, float* red) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  float acc[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int t = 0; t < NT; ++t) acc[m][t][0] = acc[m][t][1] = acc[m][t][2] = acc[m][t][3] = 0.f;
  const bf16* wp[2 * MT];
#pragma unroll
  for (int m = 0; m < 2 * MT; ++m)   // rows past N repeat the last one (their results are not stored)
    wp[m] = wrow + (size_t)min(f0 + m * 8 + g, p.N - 1) * p.K + t4 * 8;
  const bf16* xp[NT];
#pragma unroll
  for (int t = 0; t < NT; ++t) {
    const int r = r0 + min(t * 8 + g, n - 1);
    xp[t] = p.x + (size_t)(p.src ? __ldg(p.src + r) : r) * p.ldx + t4 * 8;
  }
  const int slabs = (p.K + 31) / 32;
#pragma unroll 4
  for (int s = warp; s < slabs; s += GR_WARPS) {
    const int k = s * 32;
    const bool in = k + t4 * 8 < p.K;   // K % 8 == 0: a lane's eight elements are all inside or all outside
    uint4 a[2 * MT], b[NT];
#pragma unroll
    for (int m = 0; m < 2 * MT; ++m) a[m] = in ? ldg_stream(wp[m] + k) : make_uint4(0, 0, 0, 0);
#pragma unroll
    for (int t = 0; t < NT; ++t) b[t] = in ? *reinterpret_cast<const uint4*>(xp[t] + k) : make_uint4(0, 0, 0, 0);
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int t = 0; t < NT; ++t) {
        mma16816(acc[m][t], a[2 * m].x, a[2 * m + 1].x, a[2 * m].y, a[2 * m + 1].y, b[t].x, b[t].y);
        mma16816(acc[m][t], a[2 * m].z, a[2 * m + 1].z, a[2 * m].w, a[2 * m + 1].w, b[t].z, b[t].w);
      }
  }
  // [warp][token][feature], features contiguous for the store; the pad column keeps the banks apart
  constexpr int FW = 16 * MT + 1;
  float* mine = red + warp * (8 * NT * FW);
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) mine[(t * 8 + t4 * 2 + (e & 1)) * FW + m * 16 + g + (e >> 1) * 8] = acc[m][t][e];
  __syncthreads();
  if (gemm_act_pairs(p.act)) {
    for (int i = threadIdx.x; i < n * 8 * MT; i += GR_WARPS * 32) {
      const int tok = i / (8 * MT), f = i % (8 * MT) * 2;
      if (f0 + f < p.N) {
        float a = 0.f, b = 0.f;
#pragma unroll
        for (int w = 0; w < GR_WARPS; ++w) a += red[w * (8 * NT * FW) + tok * FW + f], b += red[w * (8 * NT * FW) + tok * FW + f + 1];
        const float y = p.act == SWB_ACT_CLAMPED_PAIRS ? clamped_gate_f<false>(a, b, p.act_a)
                                                       : (p.act == SWB_ACT_GEGLU_PAIRS ? gelu_tanh_f(a) : silu_f(a)) * b;
        p.out[(size_t)(r0 + tok) * p.ldo + (f0 + f) / 2] = __float2bfloat16(y);
      }
    }
    __syncthreads();
    return;
  }
  for (int i = threadIdx.x; i < n * 16 * MT; i += GR_WARPS * 32) {
    const int tok = i / (16 * MT), f = i % (16 * MT);
    if (f0 + f < p.N) {
      float v = 0.f;
#pragma unroll
      for (int w = 0; w < GR_WARPS; ++w) v += red[w * (8 * NT * FW) + tok * FW + f];
      if (p.act == SWB_ACT_RELU2) v = relu2_f(v);
      else if (p.act == SWB_ACT_SILU) v = silu_f(v);
      else if (p.act == SWB_ACT_GELU_TANH) v = gelu_tanh_f(v);
      p.out[(size_t)(r0 + tok) * p.ldo + f0 + f] = __float2bfloat16(v);
    }
  }
  __syncthreads();
}

template <int MT>
__global__ void __launch_bounds__(GR_WARPS * 32) grouped_rows_kernel(const GroupedRowsParams p) {
  pdl_launch_dependents();
  __shared__ float red[GR_WARPS * 32 * (16 * MT + 1)];
  if (!p.plan_ahead) pdl_wait();
  const int e = p.active[blockIdx.y];
  const int f0 = blockIdx.x * (16 * MT);
  const bf16* wrow = p.w + (size_t)max(e, 0) * p.N * p.K;
  int lo = 0, hi = 0;
  if (e >= 0) lo = p.offsets[e], hi = p.offsets[e + 1];
  if (p.plan_ahead) pdl_wait();
  if (e < 0) return;
  for (int r = lo; r < hi; r += 32) {
    const int n = min(32, hi - r);
    if (n <= 8) grouped_pass<MT, 1>(p, wrow, f0, r, n, red);
    else if (n <= 16) grouped_pass<MT, 2>(p, wrow, f0, r, n, red);
    else grouped_pass<MT, 4>(p, wrow, f0, r, n, red);
  }
}

}  // namespace
}  // namespace swb

extern "C" {

// Routing plan of `layers` table-routed MoE layers for one step of T tokens. tables: int32 [layers, vocab, top].
// dest [layers, T * top]: segment row of each (token, slot) pair. src (nullable) [layers, rows_cap]: token of each segment
// row (rows of the padding are not written). offsets [layers, E + 1]: first row of each expert's segment.
// active (nullable) [layers, min(E, T * top)]: experts that got tokens, then -1. tile_group (nullable)
// [layers, rows_cap / 128]: expert of each 128-row tile, -1 past the end (needs pad 128).
// rows_cap >= T * top + E * (pad - 1), a multiple of 128 with tile_group. Table entries are clamped to [0, E).
int swb_moe_table_plan(const long long* ids, int T, const int* tables, int layers, int vocab, int top, int E, int pad,
                       int* dest, int* src, int* offsets, int* active, int* tile_group, int rows_cap, void* stream) {
  using namespace swb;
  if (T <= 0 || layers <= 0) return 0;
  if (top <= 0 || E <= 0 || E > 4096 || vocab <= 0 || (pad != 1 && pad != 128) || (tile_group && (pad != 128 || rows_cap % 128)) ||
      (long long)T * top + (long long)E * (pad - 1) > (long long)rows_cap)
    return -3;
  return launch_kernel(moe_table_plan_kernel, dim3((unsigned)layers), dim3(1024), (2 * (size_t)E + 1) * sizeof(int),
                       reinterpret_cast<cudaStream_t>(stream), ids, T, tables, vocab, top, E, pad, dest, src, offsets, active,
                       tile_group, rows_cap);
}

// Routing plan of one layer from router logits [T, ld] (fp32): the `top` experts of the largest softmax scores over all E, weights
// [T, top] = their scores, as they are or (renorm) divided by their sum + 1e-20. dest, src, offsets, active, tile_group, pad and rows_cap as in swb_moe_table_plan.
// expert and rank: int32 scratch [T * top]; counters: int32 [E + 2], zero at the first launch, launches that share it ordered on
// one stream. rows_in (nullable): bf16 / fp32 rows of `pieces` 16-byte pieces, ld_in pieces apart, copied to rows dest[t, k] of rows_out.
int swb_moe_route(const float* logits, int ld, int T, int E, int top, int renorm, int pad, int* expert, int* rank, float* weights, int* counters,
                  int* dest, int* src, int* offsets, int* active, int* tile_group, int rows_cap, const void* rows_in, long long ld_in,
                  void* rows_out, long long ld_out, int pieces, void* stream) {
  using namespace swb;
  if (T <= 0) return 0;
  if (top <= 0 || E <= 0 || E > 4096 || top > E || ld < E || (pad != 1 && pad != 128) || (tile_group && (pad != 128 || rows_cap % 128)) ||
      (long long)T * top + (long long)E * (pad - 1) > (long long)rows_cap || !expert || !rank || !weights || !counters || !dest || !offsets ||
      (rows_in && (!rows_out || pieces <= 0)))
    return -3;
  const RouteParams p{logits, ld, T, E, top, pad, expert, rank, weights, renorm, counters, dest, src, offsets, active, tile_group, rows_cap,
                      reinterpret_cast<const uint4*>(rows_in), reinterpret_cast<uint4*>(rows_out), ld_in, ld_out, pieces};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid((unsigned)((T + 7) / 8));
  const size_t smem = (size_t)(E + 1) * sizeof(int);
  if (T <= 128 && !rows_in) return launch_kernel(moe_route_kernel<true>, grid, dim3(256), smem, s, p);
  const int rc = launch_kernel(moe_route_kernel<false>, grid, dim3(256), 0, s, p);
  if (rc) return rc;
  const long long blocks = ((long long)T * top + 7) / 8;
  return launch_kernel(moe_layout_kernel, dim3((unsigned)(blocks < 148 * 8 ? blocks : 148 * 8)), dim3(256), smem, s, p);
}

// out[r, :] = act(x[src ? src[r] : r, :] W[e]^T) for every row r of expert e's segment [offsets[e], offsets[e + 1]).
// W [E, N, K] bf16, K % 8 == 0, ldx % 8 == 0, x and W 16-byte aligned; n_active = length of `active`. plan_ahead: see
// GroupedRowsParams.
int swb_gemm_grouped_rows(const void* x, int ldx, const int* src, const int* offsets, const int* active, int n_active,
                          const void* w, void* out, int ldo, int N, int K, int act, float act_a, int plan_ahead, void* stream) {
  using namespace swb;
  if (n_active <= 0 || N <= 0 || K <= 0) return 0;
  if ((K % 8) || (ldx % 8) || !offsets || !active || (gemm_act_pairs(act) && (N & 1)) ||
      ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w)) & 15))
    return -3;
  GroupedRowsParams p{reinterpret_cast<const bf16*>(x), ldx, src, offsets, active, reinterpret_cast<const bf16*>(w),
                      reinterpret_cast<bf16*>(out), ldo, N, K, act, act_a, plan_ahead};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  // 32 weight rows per CTA halve the token re-reads; 16 when that is needed to give every SM two CTAs
  if ((long long)((N + 31) / 32) * n_active >= 2 * 148)
    return launch_kernel(grouped_rows_kernel<2>, dim3((N + 31) / 32, n_active), dim3(GR_WARPS * 32), 0, s, p);
  return launch_kernel(grouped_rows_kernel<1>, dim3((N + 15) / 16, n_active), dim3(GR_WARPS * 32), 0, s, p);
}

}  // extern "C"
