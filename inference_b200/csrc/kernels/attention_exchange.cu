// Decode attention whose heads exchange their weights, over the paged KV cache (block_size 16): every query head is applied to the values of
// all key/value heads, and head h's result is sum_g talk[h, g] of what head g found in the values of h's group.
//
// exchange_decode_kernel: one CTA per (KV split, sequence) takes all heads, so that every key and value is read once. Warp 8 is the producer:
// per page one TMA copy per 64-column half brings the keys of all heads and one the values (128-byte swizzle, a ring of whole pages). Per page
// the eight compute warps first deal out tiles of eight query rows of one key head, S^T = K Q^T (16 keys by 8 rows) with the online softmax
// along the fragment, and leave the weights and the rows' rescale factors in shared memory (two buffers, so one barrier per page); then each
// warp takes an eighth of the value columns for all rows, O += P V. Per split the un-normalised O and (max, sum) go to the workspace.
// exchange_merge_kernel: merges the splits, joins the sink, mixes the heads and applies the gates, one CTA per token and 128 columns (32 with
// few tokens).
#include "attention_common.cuh"
#include "gemm_tcgen05.cuh"

namespace swb {
using namespace attn;

SWB_REGISTER_STATUS_UNIT(attn_exchange);

namespace {

constexpr int PAGE = 16, WARPS = 8, P_STRIDE = 48;          // bytes between rows of the weights (16 keys and padding)
constexpr int MAX_RING = 8, MAX_SPLITS = 32, MAX_ROWS = 64;
constexpr uint32_t SMEM_LIMIT = 227 * 1024;

struct ExchangeParams {
  const bf16* q;             // [tokens, H, D], q_stride_tok apart
  long long q_stride_tok;
  const int* block_table;
  int max_blocks;
  const int* kv_lens;
  int q_len;                 // query tokens of every sequence
  int H, G, D, NV, Dv;       // Dv: columns of one of the NV cached value heads
  float scale_log2;
  int window, num_splits, stages;
  float* part_o;             // [seq, split, rows, NV * Dv]
  float2* part_ml;           // [seq, split, rows]; row = (key head, query token, head of the group)
};

__host__ __device__ inline int halves(int d) { return (d + 63) / 64; }
__host__ __device__ inline uint32_t k_page_bytes(int G, int D) { return (uint32_t)halves(D) * G * PAGE * 128; }
__host__ __device__ inline uint32_t v_page_bytes(int NV, int Dv) { return (uint32_t)halves(Dv) * NV * PAGE * 128; }
__host__ __device__ inline int q_row_bytes(int D) { return (D + 15) / 16 * 32 + 16; }
inline uint32_t fixed_bytes(int rows, int D) {                // queries, weights, factors, barriers, alignment slack
  return (uint32_t)(rows * q_row_bytes(D) + 15) / 16 * 16 + 2 * MAX_ROWS * (P_STRIDE + 4) + 256 + 1024;
}
inline int ring_stages(int H, int G, int D, int NV, int Dv, int q_len) {
  const int rows = H * q_len, mt = (rows + 15) / 16, cols = NV * Dv;
  if (H < 1 || G < 1 || H % G || q_len < 1 || rows > MAX_ROWS || D < 8 || Dv < 8 || D > 128 || Dv > 128 || ((D | Dv) % 8) || G > 16 || NV < 1 || NV > 16 ||
      cols > (mt <= 1 ? 1024 : mt == 2 ? 512 : 256))
    return 0;
  const uint32_t page = k_page_bytes(G, D) + v_page_bytes(NV, Dv);
  const int n = (int)((SMEM_LIMIT - fixed_bytes(rows, D)) / page);
  return n < 2 ? 0 : n > MAX_RING ? MAX_RING : n;
}

// MT tiles of 16 rows, NT pairs of 8-column tiles per warp; TILES: query-row tiles that a warp may own.
template <int MT, int NT, int TILES>
__global__ void __launch_bounds__((WARPS + 1) * 32, 1)
exchange_decode_kernel(const __grid_constant__ CUtensorMap tmap_k, const __grid_constant__ CUtensorMap tmap_v, const ExchangeParams p) {
  pdl_launch_dependents();
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
  const uint32_t kb = k_page_bytes(p.G, p.D), vb = v_page_bytes(p.NV, p.Dv), stage_bytes = kb + vb;
  const int rows = p.H * p.q_len, per = p.H / p.G, group_rows = per * p.q_len, qb = q_row_bytes(p.D);
  uint8_t* ring = smem;
  uint8_t* sQ = ring + (size_t)p.stages * stage_bytes;
  uint8_t* sP = sQ + (rows * qb + 15) / 16 * 16;                           // [2][MAX_ROWS][P_STRIDE]
  float* sF = reinterpret_cast<float*>(sP + 2 * MAX_ROWS * P_STRIDE);      // [2][MAX_ROWS]
  uint64_t* bar_full = reinterpret_cast<uint64_t*>(sF + 2 * MAX_ROWS);
  uint64_t* bar_empty = bar_full + MAX_RING;
  volatile int* s_abort = reinterpret_cast<volatile int*>(bar_empty + MAX_RING);
  const int split = blockIdx.x, seq = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  if (threadIdx.x == 0) {
    for (int s = 0; s < p.stages; ++s) mbar_init(&bar_full[s], 1), mbar_init(&bar_empty[s], WARPS);
    *s_abort = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tmap_k);
    tma_prefetch_desc(&tmap_v);
  }
  for (int i = threadIdx.x; i < 2 * MAX_ROWS * P_STRIDE / 4; i += blockDim.x) reinterpret_cast<uint32_t*>(sP)[i] = 0u;    // rows past the last one
  for (int i = threadIdx.x; i < 2 * MAX_ROWS; i += blockDim.x) sF[i] = 1.f;
  pdl_wait(TL_ATTN_DECODE);

  const int kv_len = p.kv_lens[seq], shift = kv_len - p.q_len;             // position of the first query
  const int page_lo = p.window > 0 ? max(shift - p.window + 1, 0) / PAGE : 0, pages = (kv_len + PAGE - 1) / PAGE;
  const int each = (pages - page_lo + p.num_splits - 1) / p.num_splits, p0 = page_lo + split * each;
  const int n_pages = max(0, min(pages, p0 + each) - p0);
  const int k_steps = (p.D + 15) / 16;
  // queries, row (key head, query token, head of the group); columns past D are zero
  for (int i = threadIdx.x; i < rows * k_steps * 2; i += blockDim.x) {
    const int row = i / (k_steps * 2), c = i % (k_steps * 2), g = row / group_rows, r = row % group_rows;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (c * 8 < p.D)
      v = *reinterpret_cast<const uint4*>(p.q + (size_t)(seq * p.q_len + r / per) * p.q_stride_tok + (size_t)(g * per + r % per) * p.D + c * 8);
    *reinterpret_cast<uint4*>(sQ + row * qb + c * 16) = v;
  }
  __syncthreads();

  if (warp == WARPS) {
    // ------------------------------ producer ------------------------------
    if (lane == 0) {
      const int* table = p.block_table + (size_t)seq * p.max_blocks;
      const int kh = halves(p.D), vh = halves(p.Dv);
      int stage = 0, issued = 0;
      uint32_t phase = 0;
      for (int j = 0; j < n_pages; ++j) {
        if (!mbar_wait(&bar_empty[stage], phase ^ 1, s_abort, 700 + stage)) break;
        uint8_t* at = ring + (size_t)stage * stage_bytes;
        const int page = __ldg(&table[p0 + j]);
        mbar_arrive_expect_tx(&bar_full[stage], stage_bytes);
        for (int h = 0; h < kh; ++h) tma_load_2d(at + (size_t)h * p.G * PAGE * 128, &tmap_k, &bar_full[stage], h * 64, page * p.G * PAGE);
        for (int h = 0; h < vh; ++h) tma_load_2d(at + kb + (size_t)h * p.NV * PAGE * 128, &tmap_v, &bar_full[stage], h * 64, page * p.NV * PAGE);
        issued = j + 1;
        if (++stage == p.stages) stage = 0, phase ^= 1;
      }
      if (*s_abort) {              // every copy in flight lands before the CTA's shared memory is released
        for (int j = max(0, issued - p.stages); j < issued; ++j)
          for (int it = 0; it < (1 << 20); ++it)
            if (mbar_try_wait(&bar_full[j % p.stages], (uint32_t)(j / p.stages) & 1u)) break;
      }
    }
  } else {
    // ------------------------------ compute ------------------------------
    const int g4 = lane >> 2, t4 = lane & 3, mi = lane >> 3, l8 = lane & 7;
    const int tiles_per_group = (group_rows + 7) / 8, tiles = p.G * tiles_per_group, cols = p.NV * p.Dv;
    // columns of this warp, in pairs of 8-column tiles (the last one may reach past the end: it repeats the last tile and is not stored)
    const int pairs = (cols + 15) / 16, pairs_per_warp = (pairs + WARPS - 1) / WARPS, pair0 = warp * pairs_per_warp;
    const int my_pairs = max(0, min(pairs, pair0 + pairs_per_warp) - pair0);
    float o[MT][2 * NT][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < 2 * NT; ++n) o[m][n][0] = o[m][n][1] = o[m][n][2] = o[m][n][3] = 0.f;
    float m_run[TILES][2], l_run[TILES][2];
#pragma unroll
    for (int i = 0; i < TILES; ++i) m_run[i][0] = m_run[i][1] = -INFINITY, l_run[i][0] = l_run[i][1] = 0.f;
    const uint32_t q_addr = smem_u32(sQ), p_addr = smem_u32(sP), ring_addr = smem_u32(ring);
    uint32_t v_off[NT];            // of this lane's row in the V page, by pair
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      const int col = min((pair0 + n) * 16 + (mi >> 1) * 8, cols - 8), v = col / p.Dv, cc = col % p.Dv, row = v * PAGE + (mi & 1) * 8 + l8;
      v_off[n] = kb + (uint32_t)((cc >> 6) * p.NV * PAGE * 128 + row * 128 + ((((cc >> 3) & 7) ^ (row & 7)) << 4));
    }
    int stage = 0;
    uint32_t phase = 0;
    for (int j = 0; j < n_pages; ++j) {
      // after a wait that ran out the loop goes on without waiting, so that every warp takes part in every barrier
      mbar_wait(&bar_full[stage], phase, s_abort, 720 + stage);
      const uint32_t sK = ring_addr + (uint32_t)stage * stage_bytes;
      const int buf = j & 1, tok0 = (p0 + j) * PAGE;
#pragma unroll
      for (int i = 0; i < TILES; ++i) {
        const int tile = warp + i * WARPS;
        if (tile >= tiles) break;
        const int kvh = tile / tiles_per_group, r0 = tile % tiles_per_group * 8;       // first row within the group
        const uint32_t q_row = q_addr + (uint32_t)(kvh * group_rows + min(r0 + l8, group_rows - 1)) * qb;
        float s[4] = {0.f, 0.f, 0.f, 0.f};
        const int row = kvh * PAGE + (mi & 1) * 8 + l8;
#pragma unroll
        for (int kk = 0; kk < 8; kk += 2) {
          if (kk >= k_steps) break;
          uint32_t b[4];
          // two steps of the queries at once (the second may lie past the row: not used then)
          ldsm_x4(q_row + (uint32_t)min(kk * 2 + mi, k_steps * 2 - 1) * 16, b[0], b[1], b[2], b[3]);
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            if (kk + u >= k_steps) break;
            const int c = (kk + u) * 2 + (mi >> 1);
            uint32_t a[4];
            ldsm_x4(sK + (uint32_t)((c >> 3) * p.G * PAGE * 128 + row * 128 + (((c & 7) ^ (row & 7)) << 4)), a[0], a[1], a[2], a[3]);
            mma_16816(s, a, b[2 * u], b[2 * u + 1]);
          }
        }
        // s[0], s[1]: key g4, rows r0 + 2 t4 and the next; s[2], s[3]: key g4 + 8
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int r = r0 + t4 * 2 + e, pos = shift + r / per;
          auto score = [&](float x, int key) {
            return key < kv_len && key <= pos && (p.window <= 0 || key > pos - p.window) ? x * p.scale_log2 : -INFINITY;
          };
          const float s0 = score(s[e], tok0 + g4), s1 = score(s[2 + e], tok0 + g4 + 8);
          float mx = fmaxf(s0, s1);
          mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 4));
          mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 8));
          mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 16));
          const float m_new = fmaxf(m_run[i][e], mx), safe = m_new == -INFINITY ? 0.f : m_new;
          const float f = exp2f(m_run[i][e] - safe), w0 = exp2f(s0 - safe), w1 = exp2f(s1 - safe);
          m_run[i][e] = m_new;
          l_run[i][e] = l_run[i][e] * f + w0 + w1;
          if (r < group_rows) {
            const int at = kvh * group_rows + r;
            bf16* w = reinterpret_cast<bf16*>(sP + (buf * MAX_ROWS + at) * P_STRIDE);
            w[g4] = __float2bfloat16(w0);
            w[g4 + 8] = __float2bfloat16(w1);
            if (g4 == 0) sF[buf * MAX_ROWS + at] = f;
          }
        }
      }
      asm volatile("bar.sync 1, 256;" ::: "memory");
      float f[MT][2];
      bool grow = false;
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        f[m][0] = sF[buf * MAX_ROWS + m * 16 + g4], f[m][1] = sF[buf * MAX_ROWS + m * 16 + g4 + 8];
        grow |= f[m][0] != 1.f || f[m][1] != 1.f;
      }
      if (__any_sync(0xffffffffu, grow)) {
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int n = 0; n < 2 * NT; ++n) o[m][n][0] *= f[m][0], o[m][n][1] *= f[m][0], o[m][n][2] *= f[m][1], o[m][n][3] *= f[m][1];
      }
      uint32_t a[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
        ldsm_x4(p_addr + (uint32_t)((buf * MAX_ROWS + m * 16 + (mi & 1) * 8 + l8) * P_STRIDE + (mi >> 1) * 16), a[m][0], a[m][1], a[m][2], a[m][3]);
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        if (n >= my_pairs) break;
        uint32_t b0, b1, b2, b3;
        ldsm_x4_trans(sK + v_off[n], b0, b1, b2, b3);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mma_16816(o[m][2 * n], a[m], b0, b1);
          mma_16816(o[m][2 * n + 1], a[m], b2, b3);
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&bar_empty[stage]);
      if (++stage == p.stages) stage = 0, phase ^= 1;
    }
    const size_t base = ((size_t)seq * p.num_splits + split) * rows;
#pragma unroll
    for (int i = 0; i < TILES; ++i) {
      const int tile = warp + i * WARPS;
      if (tile >= tiles) break;
      const int kvh = tile / tiles_per_group, r0 = tile % tiles_per_group * 8;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float l = l_run[i][e];
        l += __shfl_xor_sync(0xffffffffu, l, 4);
        l += __shfl_xor_sync(0xffffffffu, l, 8);
        l += __shfl_xor_sync(0xffffffffu, l, 16);
        const int r = r0 + t4 * 2 + e;
        if (g4 == 0 && r < group_rows) p.part_ml[base + kvh * group_rows + r] = make_float2(m_run[i][e], l);
      }
    }
#pragma unroll
    for (int n = 0; n < 2 * NT; ++n) {
      const int col = (pair0 + n / 2) * 16 + (n & 1) * 8 + t4 * 2;
      if (n >= 2 * my_pairs || col >= cols) continue;
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int hr = 0; hr < 2; ++hr) {
          const int row = m * 16 + g4 + hr * 8;
          if (row < rows) *reinterpret_cast<float2*>(p.part_o + (base + row) * cols + col) = make_float2(o[m][n][2 * hr], o[m][n][2 * hr + 1]);
        }
    }
  }
  __syncthreads();
}

struct MergeParams {
  const float* part_o;
  const float2* part_ml;
  const float* sink;         // optional [H]
  const float* talk;         // as in head_mix_kernel (llm_ops.cu)
  const bf16* gate;          // optional logits [tokens, >= H]
  long long gate_stride;
  bf16* out;                 // [tokens, H * vp]
  long long out_stride;
  int q_len, H, G, vp, num_splits;
};

constexpr int MERGE_HEADS = 8, MERGE_THREADS = 256;

// PAIRS column pairs by MERGE_THREADS / PAIRS slices of the query heads; blockIdx.z: which MERGE_HEADS of each group.
template <int PAIRS>
__global__ void __launch_bounds__(MERGE_THREADS) exchange_merge_kernel(const MergeParams p) {
  constexpr int SLICES = MERGE_THREADS / PAIRS;
  pdl_launch_dependents();
  pdl_wait(TL_ATTN_MERGE);
  __shared__ float weight[MAX_SPLITS * MAX_ROWS];             // [split][head]
  __shared__ float sums[SLICES][2 * MERGE_HEADS][PAIRS + 1];
  const int t = blockIdx.y, seq = t / p.q_len, qtok = t % p.q_len, per = p.H / p.G, rows = p.H * p.q_len, cols = p.G * p.vp;
  const int S = p.num_splits, h0 = blockIdx.z * MERGE_HEADS, hp = (per + MERGE_HEADS - 1) / MERGE_HEADS * MERGE_HEADS;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  auto row_of = [&](int h) { return h / per * per * p.q_len + qtok * per + h % per; };
  const size_t base = (size_t)seq * S * rows;
  for (int h = warp; h < p.H; h += MERGE_THREADS / 32) {      // a lane per split
    const float sink = p.sink ? p.sink[h] * 1.4426950408889634f : -INFINITY;
    const float2 ml = lane < S ? __ldcg(p.part_ml + base + (size_t)lane * rows + row_of(h)) : make_float2(-INFINITY, 0.f);
    const float top = fmaxf(warp_max(ml.x), sink), e = ml.x == -INFINITY ? 0.f : exp2f(ml.x - top);
    const float den = warp_sum(e * ml.y) + (p.sink ? exp2f(sink - top) : 0.f);
    if (lane < S) weight[lane * p.H + h] = den > 0.f ? e / den : 0.f;
  }
  __syncthreads();
  const int pair = threadIdx.x % PAIRS, slice = threadIdx.x / PAIRS, col = (blockIdx.x * PAIRS + pair) * 2;
  float acc[MERGE_HEADS][2] = {};
  if (col < cols) {
    const int c = col / p.vp;
    const float* talk = p.talk + (size_t)c * hp + h0;
#pragma unroll 4
    for (int h = slice; h < p.H; h += SLICES) {
      const float* o = p.part_o + (base + row_of(h)) * cols + col;
      float x = 0.f, y = 0.f;
#pragma unroll 8
      for (int s = 0; s < S; ++s) {
        const float2 v = __ldcg(reinterpret_cast<const float2*>(o + (size_t)s * rows * cols));
        const float w = weight[s * p.H + h];
        x = fmaf(w, v.x, x), y = fmaf(w, v.y, y);
      }
      const float4 w0 = __ldg(reinterpret_cast<const float4*>(talk + (size_t)h * p.G * hp)), w1 = __ldg(reinterpret_cast<const float4*>(talk + (size_t)h * p.G * hp) + 1);
      const float w[MERGE_HEADS] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
      for (int i = 0; i < MERGE_HEADS; ++i) acc[i][0] = fmaf(w[i], x, acc[i][0]), acc[i][1] = fmaf(w[i], y, acc[i][1]);
    }
  }
#pragma unroll
  for (int i = 0; i < MERGE_HEADS; ++i) sums[slice][2 * i][pair] = acc[i][0], sums[slice][2 * i + 1][pair] = acc[i][1];
  __syncthreads();
  for (int i = threadIdx.x; i < MERGE_HEADS * PAIRS * 2; i += MERGE_THREADS) {
    const int head = i / (PAIRS * 2), cc = i % (PAIRS * 2), at = blockIdx.x * PAIRS * 2 + cc;
    if (h0 + head >= per || at >= cols) continue;
    float x = 0.f;
#pragma unroll
    for (int s = 0; s < SLICES; ++s) x += sums[s][2 * head + (cc & 1)][cc >> 1];
    const int h = at / p.vp * per + h0 + head;
    if (p.gate) x /= 1.f + __expf(-__bfloat162float(p.gate[t * p.gate_stride + h]));
    p.out[t * p.out_stride + (size_t)h * p.vp + at % p.vp] = __float2bfloat16(x);
  }
}

template <int MT, int NT, int TILES>
int launch_exchange(const ExchangeParams& p, int num_seqs, int num_blocks, const bf16* k, const bf16* v, uint32_t smem, cudaStream_t st) {
  auto kernel = exchange_decode_kernel<MT, NT, TILES>;
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64 || !configured[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM_LIMIT);
    if (e != cudaSuccess) return -(int)e;
    if (dev >= 0 && dev < 64) configured[dev] = true;
  }
  CUtensorMap tk, tv;
  int rc = make_tmap_bf16_2d(&tk, k, num_blocks * p.G * PAGE, p.D, p.D, p.G * PAGE);
  if (!rc) rc = make_tmap_bf16_2d(&tv, v, num_blocks * p.NV * PAGE, p.Dv, p.Dv, p.NV * PAGE);
  if (rc) return rc;
  return launch_kernel(kernel, dim3(p.num_splits, num_seqs), dim3((WARPS + 1) * 32), smem, st, tk, tv, p);
}

}  // namespace
}  // namespace swb

extern "C" {

size_t swb_exchange_workspace_bytes(int num_seqs, int H, int q_len, int cols, int num_splits) {
  return (size_t)num_seqs * num_splits * H * q_len * ((size_t)cols * sizeof(float) + sizeof(float2));
}

// Stages of the page ring, 0 when the shape is outside the kernel's reach (see ring_stages).
int swb_exchange_decode_stages(int H, int G, int D, int NV, int Dv, int q_len) { return swb::ring_stages(H, G, D, NV, Dv, q_len); }

// Decode attention with exchanged weights: q [num_seqs * q_len, H, D] (rows q_stride_tok apart), kcache [num_blocks, G, 16, D], vcache
// [num_blocks, NV, 16, Dv] with NV * Dv = G * vp columns, head h's values being the vp columns from h / (H / G) * vp on; talk as swb_head_mix;
// sink (nullable) fp32 [H]; gate (nullable): logits per head, rows gate_stride apart -> out [num_seqs * q_len, H * vp]. window > 0: only the
// last `window` keys, the query's own included. Returns -3 when the shape is outside the kernel's reach.
int swb_exchange_decode(const void* q, long long q_stride_tok, const void* kcache, const void* vcache, void* out, long long out_stride,
                        const int* block_table, int max_blocks, int num_blocks, const int* kv_lens, int num_seqs, int q_len, int H, int G, int D,
                        int NV, int Dv, int vp, float scale, int window, const float* sink, const float* talk, const void* gate,
                        long long gate_stride, int num_splits, void* workspace, size_t workspace_bytes, void* stream) {
  using namespace swb;
  if (num_seqs <= 0) return 0;
  const int stages = ring_stages(H, G, D, NV, Dv, q_len), rows = H * q_len, cols = NV * Dv;
  if (!stages || cols != G * vp || (vp % 2) || !(scale > 0.f) || window < 0 || num_splits < 1 || num_splits > MAX_SPLITS || (q_stride_tok % 8) ||
      num_blocks < 1 || !talk || !block_table || !kv_lens)
    return -3;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(kcache) | reinterpret_cast<uintptr_t>(vcache)) & 15) return -3;
  if (!workspace || workspace_bytes < swb_exchange_workspace_bytes(num_seqs, H, q_len, cols, num_splits)) return -5;
  const int tiles = G * ((H / G * q_len + 7) / 8), mt = (rows + 15) / 16;
  if (tiles > 8 * WARPS) return -3;
  float* part_o = reinterpret_cast<float*>(workspace);
  float2* part_ml = reinterpret_cast<float2*>(part_o + (size_t)num_seqs * num_splits * rows * cols);
  const ExchangeParams p{reinterpret_cast<const bf16*>(q), q_stride_tok, block_table, max_blocks, kv_lens, q_len, H, G, D, NV, Dv,
                         scale * 1.4426950408889634f, window, num_splits, stages, part_o, part_ml};
  const uint32_t smem = (uint32_t)stages * (k_page_bytes(G, D) + v_page_bytes(NV, Dv)) + fixed_bytes(rows, D);
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  auto go = [&](auto one, auto two, auto eight) {
    auto* f = tiles <= WARPS ? one : tiles <= 2 * WARPS ? two : eight;
    return f(p, num_seqs, num_blocks, reinterpret_cast<const bf16*>(kcache), reinterpret_cast<const bf16*>(vcache), smem, st);
  };
  const int rc = mt <= 1 ? go(&launch_exchange<1, 8, 1>, &launch_exchange<1, 8, 2>, &launch_exchange<1, 8, 8>)
                 : mt == 2 ? go(&launch_exchange<2, 4, 1>, &launch_exchange<2, 4, 2>, &launch_exchange<2, 4, 8>)
                           : go(&launch_exchange<4, 2, 1>, &launch_exchange<4, 2, 2>, &launch_exchange<4, 2, 8>);
  if (rc) return rc;
  const MergeParams m{part_o, part_ml, sink, talk, reinterpret_cast<const bf16*>(gate), gate_stride, reinterpret_cast<bf16*>(out), out_stride, q_len,
                      H, G, vp, num_splits};
  const int tokens = num_seqs * q_len, z = (H / G + MERGE_HEADS - 1) / MERGE_HEADS;
  if ((cols + 127) / 128 * tokens >= 148)
    return launch_kernel(exchange_merge_kernel<64>, dim3((cols + 127) / 128, tokens, z), dim3(MERGE_THREADS), 0, st, m);
  return launch_kernel(exchange_merge_kernel<16>, dim3((cols + 31) / 32, tokens, z), dim3(MERGE_THREADS), 0, st, m);
}

}  // extern "C"
