// Decode attention over the paged KV cache with TMA-fed, warp-specialised CTAs (block_size 16, head widths up to 128:
// columns past the width of q / k or v are zero fill of the tensor maps, whole 64-column halves past it are not fetched).
//
// One CTA per (KV split, kv head, sequence). Warp 4 is the producer: for every 64-token tile it looks up
// the four 16-token blocks in the block table and issues one tiled TMA copy per (block, K|V, 64-column
// half) with the 128-byte swizzle into a 3-stage ring, completing on an mbarrier. Warps 0..3 each take a
// 16-token slice of every tile: S = Q K^T and O += P V on mma.sync with ldmatrix from the swizzled ring,
// online softmax in registers, then a cross-warp merge in shared memory. The <=16 MMA rows are the GQA
// group's query heads times the (1..4) query tokens of the step. With num_splits > 1 the CTA writes an
// un-normalised partial (O, max, sum); the last split CTA of a (sequence, kv head) to finish merges them (ticket
// counter in the workspace, reset by the merger), so split-KV decode is still one launch.
// The decode step is bandwidth bound (KV bytes >> FLOPs), so the design goal is bytes in flight:
// 2 CTAs/SM x 3 stages x 32 KB with no per-thread address arithmetic on the load path.
#include "attention_common.cuh"
#include "gemm_tcgen05.cuh"

namespace swb {
using namespace attn;

SWB_REGISTER_STATUS_UNIT(attn_decode_tma);

namespace {

#ifndef SWB_DEC_STAGES
#define SWB_DEC_STAGES 3
#endif
constexpr int STAGES = SWB_DEC_STAGES;
constexpr int STAGE_BYTES = 2 * TILE_BYTES;  // K tile + V tile = 32 KB
constexpr int Q_BYTES = 16 * 256;            // 4 KB
constexpr int SMEM_BYTES = 1024 + Q_BYTES + STAGES * STAGE_BYTES + 256;

// Offset of 16-byte chunk c (0..15) of token row `tok` (0..63) inside a tile written by TMA as
// 8 boxes of [16 rows][64 bf16] with SWIZZLE_128B: box = (tok / 16) * 2 + (c / 8), 2 KB each.
__device__ __forceinline__ uint32_t tma_tile_off(int tok, int c) {
  const int r = tok & 15;
  return (uint32_t)((((tok >> 4) * 2 + (c >> 3)) << 11) + r * 128 + (((c & 7) ^ (r & 7)) << 4));
}
// Q rows are written by ordinary stores with the simple XOR swizzle of the other kernels.
__device__ __forceinline__ uint32_t q_off(int r, int c) { return (uint32_t)(r * 256 + ((c ^ (r & 7)) << 4)); }

// 1 / softmax denominator of a row with running max M (log2 units) and sum L relative to it; the numerators are relative
// to M as well. A sink adds exp(sink) to the denominator; one far above every score makes the weights vanish.
template <bool EXT>
__device__ __forceinline__ float softmax_inv(const AttnParams& p, int head, float M, float L) {
  if (EXT && p.sink) {
    const float sk = p.sink[head] * 1.4426950408889634f;
    const float top = fmaxf(sk, M), e = exp2f(M - top);
    return e / (L * e + exp2f(sk - top));
  }
  return L > 0.f ? 1.f / L : 0.f;
}

// cap tanh(s scale / cap) in log2 units, tanh y = 1 - 2 / (e^(2 y) + 1); the absolute error is that of fp32 numbers of the size of cap
__device__ __forceinline__ float capped_score(float s, float scale, float to_cap, float cap) {
  if (cap <= 0.f) return s * (scale * 1.4426950408889634f);
  const float k = 1.4426950408889634f * cap;
  return fmaf(-2.f * k, __fdividef(1.f, exp2f(s * to_cap) + 1.f), k);
}

// Sums of up to eight values per thread over the 128 merging threads (warps 0-3); `red` holds 32 floats.
__device__ __forceinline__ void sum_over_128(float* v, float* red, int n) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    if (i >= n) break;
    v[i] = warp_sum(v[i]);
    if (lane == 0) red[i * 4 + warp] = v[i];
  }
  asm volatile("bar.sync 1, 128;" ::: "memory");
#pragma unroll
  for (int i = 0; i < 8; ++i)
    if (i < n) v[i] = (red[i * 4] + red[i * 4 + 1]) + (red[i * 4 + 2] + red[i * 4 + 3]);
}

// EXT: chunked and windowed masking, sinks, output gates, values of every head (blockIdx.y then runs over key head, value head). FULL: q / k
// and v are HD wide (their loop bounds are then constants). DIFF: the two maps of a head are neighbouring query rows, each zero outside its
// own columns of the key row, so that both maps' scores come from one product; the merge subtracts the second map and norms the difference.
// Two CTAs per SM put three warps on a scheduler's quarter of the registers, which leaves 168 for a thread: a bound of 192 threads asks the
// compiler for that (160 are launched).
template <bool EXT, bool FULL, bool DIFF>
__global__ void __launch_bounds__(192, 2) attn_decode_tma_kernel(const __grid_constant__ CUtensorMap tmap_k,
                                                              const __grid_constant__ CUtensorMap tmap_v,
                                                              const AttnParams p) {
  pdl_launch_dependents();
  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw = smem_u32(smem_raw);
  uint8_t* smem = smem_raw + ((1024u - (raw & 1023u)) & 1023u);
  uint8_t* ring = smem;                                  // STAGES x 32 KB, 1024-aligned
  uint8_t* sQp = smem + STAGES * STAGE_BYTES;            // 4 KB
  uint64_t* bar_full = reinterpret_cast<uint64_t*>(sQp + Q_BYTES);
  uint64_t* bar_empty = bar_full + STAGES;
  volatile int* s_abort = reinterpret_cast<volatile int*>(bar_empty + STAGES);
  float* sMerge = reinterpret_cast<float*>(ring);        // reused after the loop (33 KB)
  float* sRed = sMerge + STAGES * STAGE_BYTES / 4 - 32;  // DIFF: 32 floats behind it

  const int split = blockIdx.x;
  const int v_heads = EXT && p.v_heads > 0 ? p.v_heads : 1;
  const int kvh = EXT ? blockIdx.y / v_heads : blockIdx.y;
  const int vh = EXT && p.v_heads > 0 ? blockIdx.y % v_heads : kvh, v_rows = EXT && p.v_heads > 0 ? v_heads : p.Hkv;
  const int seq = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const size_t part0 = ((size_t)seq * gridDim.y + blockIdx.y) * p.num_splits * 16;     // first row of this problem's partials

  if (threadIdx.x == 0) {
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(&bar_full[s], 1);
      mbar_init(&bar_empty[s], 4);
    }
    *s_abort = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tmap_k);
    tma_prefetch_desc(&tmap_v);
  }
  pdl_wait(TL_ATTN_DECODE);  // everything below reads what the preceding kernels wrote (q, the newest K/V, kv_lens)

  const int q_start = p.cu_q ? p.cu_q[seq] : seq * p.uniform_q_len;
  const int q_len = p.cu_q ? p.cu_q[seq + 1] - q_start : p.uniform_q_len;
  const int kv_len = p.kv_lens[seq];
  const int nrows = min(16, q_len * p.G);
  const int causal_shift = kv_len - q_len;
  // chunked attention starts at the tile that holds the first key of the first query's chunk
  int tile_lo = (EXT && p.chunk > 0) ? max(causal_shift, 0) / p.chunk * p.chunk / KV_TILE : 0;
  if (EXT && p.window > 0) tile_lo = max(tile_lo, max(causal_shift - p.window + 1, 0) / KV_TILE);
  const int total_tiles = (kv_len + KV_TILE - 1) / KV_TILE;
  const int per = (total_tiles - tile_lo + p.num_splits - 1) / p.num_splits;
  const int t0 = tile_lo + split * per;
  const int n_tiles = max(0, min(total_tiles, t0 + per) - t0);
  const int k_dim = FULL ? HD : p.k_dim, v_dim = FULL ? HD : p.v_dim;
  const int k_steps = (k_dim + 15) >> 4, v_steps = (v_dim + 15) >> 4;   // 16-column MMA steps that hold data
  const int k_halves = (k_dim + 63) >> 6, v_halves = (v_dim + 63) >> 6;

  // Q rows -> shared (row r = query token r / G, head kvh * G + r % G), zero rows past nrows
  for (int idx = threadIdx.x; idx < 256; idx += blockDim.x) {
    const int row = idx >> 4, c = idx & 15;
    uint4 val = make_uint4(0, 0, 0, 0);
    const int qtok = row / p.G, hg = row % p.G;
    const int c0 = DIFF ? c * 8 - (hg & 1) * p.diff.dim : c * 8;          // column within the head's q row
    if (row < nrows && c0 >= 0 && c0 < (DIFF ? p.diff.dim : k_dim)) {
      val = *reinterpret_cast<const uint4*>(p.q + (size_t)(q_start + qtok) * p.q_stride_tok +
                                            (size_t)(kvh * p.G + hg) * p.q_stride_head + c0);
    }
    *reinterpret_cast<uint4*>(sQp + q_off(row, c)) = val;
  }
  if (EXT && !DIFF && p.gate) {          // the gates are read by the merge: have them near by then
    for (int i = threadIdx.x; i < nrows * 2; i += blockDim.x) {
      const int row = i >> 1, half = i & 1;
      if (half * 64 < v_dim) {
        const bf16* g = p.gate + (size_t)(q_start + row / p.G) * p.gate_stride + (size_t)(kvh * p.G + row % p.G) * v_dim + half * 64;
        asm volatile("prefetch.global.L2 [%0];" ::"l"(g));
      }
    }
  }
  __syncthreads();

  float o[16][4];
#pragma unroll
  for (int i = 0; i < 16; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY};
  float l_run[2] = {0.f, 0.f};

  if (warp == 4) {
    // ------------------------------ producer ------------------------------
    if (lane == 0) {
      const int* table = p.block_table + (size_t)seq * p.max_blocks;
      const int first_block = __ldg(&table[0]);
      int stage = 0;
      uint32_t phase = 0;
      uint32_t outstanding = 0, issue_phase = 0;
      for (int j = 0; j < n_tiles; ++j) {
        if (!mbar_wait(&bar_empty[stage], phase ^ 1, s_abort, 500 + stage)) break;
        outstanding &= ~(1u << stage);
        uint8_t* sK = ring + stage * STAGE_BYTES;
        uint8_t* sV = sK + TILE_BYTES;
        mbar_arrive_expect_tx(&bar_full[stage], (uint32_t)(k_halves + v_halves) * 4 * 2048);
        const int tok0 = (t0 + j) * KV_TILE;
#pragma unroll
        for (int b = 0; b < 4; ++b) {
          const int tstart = tok0 + b * 16;
          // blocks wholly past the context reuse the first block: finite data, masked in the softmax
          const int blk = tstart < kv_len ? __ldg(&table[tstart >> 4]) : first_block;
          const int row0 = (blk * p.Hkv + kvh) * 16, vrow0 = (blk * v_rows + vh) * 16;
          tma_load_2d(sK + (b * 2 + 0) * 2048, &tmap_k, &bar_full[stage], 0, row0);
          if (k_halves > 1) tma_load_2d(sK + (b * 2 + 1) * 2048, &tmap_k, &bar_full[stage], 64, row0);
          tma_load_2d(sV + (b * 2 + 0) * 2048, &tmap_v, &bar_full[stage], 0, vrow0);
          if (v_halves > 1) tma_load_2d(sV + (b * 2 + 1) * 2048, &tmap_v, &bar_full[stage], 64, vrow0);
        }
        outstanding |= 1u << stage;
        issue_phase = (issue_phase & ~(1u << stage)) | (phase << stage);
        if (++stage == STAGES) {
          stage = 0;
          phase ^= 1;
        }
      }
      if (*s_abort) {
        for (int s = 0; s < STAGES; ++s)
          if (outstanding & (1u << s))
            for (int it = 0; it < (1 << 20); ++it)
              if (mbar_try_wait(&bar_full[s], (issue_phase >> s) & 1u)) break;
      }
    }
  } else {
    // ------------------------------ consumers (4 warps, 16 tokens of each tile per warp) --------------
    const int g = lane >> 2, t4 = lane & 3;
    const uint32_t sQ = smem_u32(sQp);
    uint32_t qf[8][4];
#pragma unroll
    for (int kk = 0; kk < 8; ++kk) {
      const int mi = lane >> 3;
      const int row = (mi & 1) * 8 + (lane & 7);
      ldsm_x4(sQ + q_off(row, kk * 2 + (mi >> 1)), qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3]);
    }
    int stage = 0;
    uint32_t phase = 0;
    float row_scale[2] = {p.scale, p.scale};
    if (DIFF && p.diff.q_temp) {
#pragma unroll
      for (int hr = 0; hr < 2; ++hr) row_scale[hr] *= p.diff.q_temp[min((g + hr * 8) / p.G, q_len - 1) + max(causal_shift, 0)];
    }
    int first_key[2], last_key[2];         // visible keys of this lane's two rows
#pragma unroll
    for (int hr = 0; hr < 2; ++hr) {
      const int qpos = (g + hr * 8) / p.G + causal_shift;
      first_key[hr] = EXT && p.chunk > 0 ? qpos / p.chunk * p.chunk : 0;
      if (EXT && p.window > 0) first_key[hr] = max(first_key[hr], qpos - p.window + 1);
      last_key[hr] = p.causal ? min(kv_len - 1, qpos) : kv_len - 1;
    }
    float row_cap[2] = {0.f, 0.f};         // 2 log2(e) scale / cap
    if (DIFF && p.diff.cap > 0.f) row_cap[0] = 2.8853900818f * row_scale[0] / p.diff.cap, row_cap[1] = 2.8853900818f * row_scale[1] / p.diff.cap;
    for (int j = 0; j < n_tiles; ++j) {
      if (!mbar_wait(&bar_full[stage], phase, s_abort, 600 + stage)) break;
      const uint32_t sK = smem_u32(ring + stage * STAGE_BYTES);
      const uint32_t sV = sK + TILE_BYTES;
      float s[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
#pragma unroll
      for (int kk = 0; kk < 8; ++kk) {
        if (kk >= k_steps) break;
        const int mi = lane >> 3;
        const int tok = warp * 16 + (mi >> 1) * 8 + (lane & 7);
        uint32_t b0, b1, b2, b3;
        ldsm_x4(sK + tma_tile_off(tok, kk * 2 + (mi & 1)), b0, b1, b2, b3);
        mma_16816(s[0], qf[kk], b0, b1);
        mma_16816(s[1], qf[kk], b2, b3);
      }
      const int tok_base = (t0 + j) * KV_TILE + warp * 16;
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float val = DIFF ? capped_score(s[nt][e], row_scale[e >> 1], row_cap[e >> 1], p.diff.cap) : score_transform(s[nt][e], p.scale, p.softcap);
          const int col = tok_base + nt * 8 + t4 * 2 + (e & 1);
          const bool ok = col <= last_key[e >> 1] && (!EXT || col >= first_key[e >> 1]);
          s[nt][e] = ok ? val : -INFINITY;
        }
      }
#pragma unroll
      for (int hr = 0; hr < 2; ++hr) {
        float mx = fmaxf(fmaxf(s[0][2 * hr], s[0][2 * hr + 1]), fmaxf(s[1][2 * hr], s[1][2 * hr + 1]));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float m_new = fmaxf(m_run[hr], mx);
        const float m_safe = (m_new == -INFINITY) ? 0.f : m_new;
        const float alpha = exp2f(m_run[hr] - m_safe);
        float rs = 0.f;
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          const float p0 = exp2f(s[nt][2 * hr] - m_safe);
          const float p1 = exp2f(s[nt][2 * hr + 1] - m_safe);
          s[nt][2 * hr] = p0;
          s[nt][2 * hr + 1] = p1;
          rs += p0 + p1;
        }
        l_run[hr] = l_run[hr] * alpha + rs;
        m_run[hr] = m_new;
#pragma unroll
        for (int dn = 0; dn < 16; ++dn) {
          o[dn][2 * hr] *= alpha;
          o[dn][2 * hr + 1] *= alpha;
        }
      }
      {
        uint32_t a[4];
        a[0] = pack_bf16(s[0][0], s[0][1]);
        a[1] = pack_bf16(s[0][2], s[0][3]);
        a[2] = pack_bf16(s[1][0], s[1][1]);
        a[3] = pack_bf16(s[1][2], s[1][3]);
#pragma unroll
        for (int dp = 0; dp < 8; ++dp) {
          if (dp >= v_steps) break;
          const int mi = lane >> 3;
          const int tok = warp * 16 + (mi & 1) * 8 + (lane & 7);
          uint32_t b0, b1, b2, b3;
          ldsm_x4_trans(sV + tma_tile_off(tok, dp * 2 + (mi >> 1)), b0, b1, b2, b3);
          mma_16816(o[2 * dp], a, b0, b1);
          mma_16816(o[2 * dp + 1], a, b2, b3);
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&bar_empty[stage]);
      if (++stage == STAGES) {
        stage = 0;
        phase ^= 1;
      }
    }
  }
  __syncthreads();  // every issued tile has been consumed (or the CTA aborted and drained): the ring is free

  if (warp < 4) {
    const int g = lane >> 2, t4 = lane & 3;
    float* wO = sMerge + warp * (16 * HD);
    float* wM = sMerge + 4 * 16 * HD + warp * 16;
    float* wL = wM + 4 * 16;
#pragma unroll
    for (int hr = 0; hr < 2; ++hr) {
      float l = l_run[hr];
      l += __shfl_xor_sync(0xffffffffu, l, 1);
      l += __shfl_xor_sync(0xffffffffu, l, 2);
      const int row = g + hr * 8;
      if (t4 == 0) {
        wM[row] = m_run[hr];
        wL[row] = l;
      }
#pragma unroll
      for (int dn = 0; dn < 16; ++dn) {
        *reinterpret_cast<float2*>(&wO[row * HD + dn * 8 + t4 * 2]) = make_float2(o[dn][2 * hr], o[dn][2 * hr + 1]);
      }
    }
  }
  __syncthreads();
  float keep[8];                           // DIFF: differences of the row pairs
  auto put = [&](int row, int d, float x) {      // output column d of query row `row`
    const int head = kvh * p.G + row % p.G;
    const size_t tok = q_start + row / p.G, col = (size_t)(EXT && p.v_heads > 0 ? head * v_heads + vh : head) * v_dim + d;
    if (EXT && !DIFF && p.gate) {
      const float z = __bfloat162float(p.gate[tok * p.gate_stride + col]);
      x *= __fdividef(1.f, 1.f + __expf(-z));
    }
    p.out[tok * p.out_stride_tok + col] = __float2bfloat16(x);
  };
  if (threadIdx.x < 128) {
    const int d = threadIdx.x;
    for (int row = 0; row < nrows; ++row) {
      float M = -INFINITY;
#pragma unroll
      for (int w = 0; w < 4; ++w) M = fmaxf(M, sMerge[4 * 16 * HD + w * 16 + row]);
      const float Ms = (M == -INFINITY) ? 0.f : M;
      float L = 0.f, acc = 0.f;
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        const float sc = exp2f(sMerge[4 * 16 * HD + w * 16 + row] - Ms);
        L += sc * sMerge[4 * 16 * HD + 4 * 16 + w * 16 + row];
        acc += sc * sMerge[w * 16 * HD + row * HD + d];
      }
      if (p.num_splits == 1) {
        const float inv = softmax_inv<EXT>(p, kvh * p.G + row % p.G, M, L);
        if (DIFF) {
          sMerge[row * HD + d] = acc * inv;      // warp 0's partial of this row and column, read by this thread alone
        } else if (d < v_dim) put(row, d, acc * inv);
      } else {
        const size_t base = part0 + (size_t)split * 16 + row;
        p.part_o[base * HD + d] = acc;
        if (d == 0) {
          p.part_ml[base * 2] = M;
          p.part_ml[base * 2 + 1] = L;
        }
      }
    }
  }
  auto store_pairs = [&](const float* at) {      // at [nrows, HD]: normalised outputs of the two maps of every pair of rows
    const int d = threadIdx.x, pairs = nrows / 2;
    float ss[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      keep[i] = i < pairs && d < v_dim ? at[2 * i * HD + d] - p.diff.share * at[(2 * i + 1) * HD + d] : 0.f;
      ss[i] = keep[i] * keep[i];
    }
    sum_over_128(ss, sRed, pairs);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      if (i >= pairs || d >= v_dim) continue;
      const int qtok = 2 * i / p.G, hg = 2 * i % p.G;
      p.out[(size_t)(q_start + qtok) * p.out_stride_tok + (size_t)((kvh * p.G + hg) / 2) * v_dim + d] =
          __float2bfloat16(keep[i] * rsqrtf(ss[i] / (float)p.diff.n + p.diff.eps) * p.diff.post);
    }
  };
  if (DIFF && p.num_splits == 1) {
    if (threadIdx.x < 128) store_pairs(sMerge);
    return;
  }
  if (p.num_splits > 1 && p.split_counters) {
    // Merge of the splits inside this launch. Cluster launch (the splits of a (sequence, kv head) form one
    // thread-block cluster): a cluster barrier orders the partials, the first CTA merges. Otherwise the last split
    // to arrive (ticket counter in the workspace, reset by the merger) merges.
    int* ctr = p.split_counters + (size_t)seq * gridDim.y + blockIdx.y;
    if (p.cluster_merge) {
      asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
      asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
      if (split != 0) return;
    } else {
      __shared__ int s_last;
      __threadfence();                       // this CTA's partials are visible device-wide before its ticket
      __syncthreads();
      if (threadIdx.x == 0) s_last = (atomicAdd(ctr, 1) == p.num_splits - 1) ? 1 : 0;
      __syncthreads();
      if (!s_last) return;
      __threadfence();
    }
    const int S = p.num_splits;            // <= 32
    float* sSc = sMerge;                   // [16][32] weights of the splits, then normalised
    float* sL = sMerge + 16 * 32;          // [16][32]
    const size_t base0 = part0;
    __syncthreads();                       // (cluster path: the cross-warp merge area is free)
    for (int i = threadIdx.x; i < nrows * S; i += blockDim.x) {
      const int row = i / S, sp = i % S;
      const float2 ml = __ldcg(reinterpret_cast<const float2*>(p.part_ml + (base0 + (size_t)sp * 16 + row) * 2));
      sSc[row * 32 + sp] = ml.x;
      sL[row * 32 + sp] = ml.y;
    }
    // the partial outputs do not depend on the weights: request them now (up to 4 rows x 8 splits stay in registers)
    float po[4][8];
    const bool small = !DIFF && nrows <= 4 && S <= 8 && threadIdx.x < 128;
    if (small) {
#pragma unroll
      for (int row = 0; row < 4; ++row)
#pragma unroll
        for (int sp = 0; sp < 8; ++sp)
          po[row][sp] = (row < nrows && sp < S)
                            ? __ldcg(p.part_o + (base0 + (size_t)sp * 16 + row) * HD + threadIdx.x) : 0.f;
    }
    __syncthreads();
    if ((int)threadIdx.x < nrows) {
      const int row = threadIdx.x;
      float M = -INFINITY;
      for (int sp = 0; sp < S; ++sp) M = fmaxf(M, sSc[row * 32 + sp]);
      const float Ms = (M == -INFINITY) ? 0.f : M;
      float L = 0.f;
      for (int sp = 0; sp < S; ++sp) {
        const float sc = exp2f(sSc[row * 32 + sp] - Ms);
        sSc[row * 32 + sp] = sc;
        L += sc * sL[row * 32 + sp];
      }
      const float inv = softmax_inv<EXT>(p, kvh * p.G + row % p.G, M, L);
      for (int sp = 0; sp < S; ++sp) sSc[row * 32 + sp] *= inv;
    }
    __syncthreads();
    if constexpr (DIFF) {
      if (threadIdx.x < 128) {
        float* at = sMerge + 2 * 16 * 32;
        const int d = threadIdx.x;
        for (int row = 0; row < nrows; ++row) {
          float acc = 0.f;
#pragma unroll 8
          for (int sp = 0; sp < S; ++sp) acc += sSc[row * 32 + sp] * __ldcg(p.part_o + (base0 + (size_t)sp * 16 + row) * HD + d);
          at[row * HD + d] = acc;
        }
        store_pairs(at);
      }
    } else if ((int)threadIdx.x < v_dim) {
      const int d = threadIdx.x;
      if (small) {
#pragma unroll
        for (int row = 0; row < 4; ++row) {
          if (row < nrows) {
            float acc = 0.f;
#pragma unroll
            for (int sp = 0; sp < 8; ++sp)
              if (sp < S) acc += sSc[row * 32 + sp] * po[row][sp];
            put(row, d, acc);
          }
        }
      } else {
        for (int row = 0; row < nrows; ++row) {
          float acc = 0.f;
#pragma unroll 8
          for (int sp = 0; sp < S; ++sp)
            acc += sSc[row * 32 + sp] * __ldcg(p.part_o + (base0 + (size_t)sp * 16 + row) * HD + d);
          put(row, d, acc);
        }
      }
    }
    if (!p.cluster_merge && threadIdx.x == 0) *ctr = 0;        // ready for the next launch
  }
}

}  // namespace

// Launches the TMA decode kernel; kcache / vcache are one layer's [blocks, Hkv, 16, 128] tensors.
int attn_decode_tma_launch(const AttnParams& p, int num_blocks, cudaStream_t stream) {
  const bool ext = p.chunk > 0 || p.sink != nullptr || p.window > 0 || p.v_heads > 0 || p.gate, full = p.k_dim == HD && p.v_dim == HD;
  const int which = p.diff.maps ? (full ? 3 : 4) : full ? (ext ? 1 : 0) : 2;
  auto kernel = which == 0   ? attn_decode_tma_kernel<false, true, false>
                : which == 1 ? attn_decode_tma_kernel<true, true, false>
                : which == 2 ? attn_decode_tma_kernel<true, false, false>
                : which == 3 ? attn_decode_tma_kernel<true, true, true>
                             : attn_decode_tma_kernel<true, false, true>;
  static bool configured[5][64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !configured[which][dev]) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_BYTES);
    if (e != cudaSuccess) return -(int)e;
    configured[which][dev] = true;
  }
  CUtensorMap tk, tv;
  const int rows = num_blocks * p.Hkv * 16;
  int rc = make_tmap_bf16_2d(&tk, p.k, rows, p.k_dim, p.k_dim, 16);
  if (rc) return rc;
  rc = make_tmap_bf16_2d(&tv, p.v, p.v_heads > 0 ? num_blocks * p.v_heads * 16 : rows, p.v_dim, p.v_dim, 16);
  if (rc) return rc;
  dim3 grid(p.num_splits, p.Hkv * (p.v_heads > 0 ? p.v_heads : 1), p.num_seqs);
  if (p.num_splits > 1 && p.num_splits <= 8 && p.split_counters) {
    // the splits of one (sequence, kv head) as a thread-block cluster: merged after a cluster barrier
    AttnParams pc = p;
    pc.cluster_merge = 1;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = dim3(160);
    cfg.dynamicSmemBytes = SMEM_BYTES;
    cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = p.num_splits;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = 1;
    int na = 1;
    if (pdl_enabled()) {
      attr[na].id = cudaLaunchAttributeProgrammaticStreamSerialization;
      attr[na].val.programmaticStreamSerializationAllowed = 1;
      ++na;
    }
    cfg.attrs = attr;
    cfg.numAttrs = na;
    cudaError_t e = cudaLaunchKernelEx(&cfg, kernel, tk, tv, pc);
    return e == cudaSuccess ? 0 : -(int)e;
  }
  return launch_kernel(kernel, grid, dim3(160), SMEM_BYTES, stream, tk, tv, p);
}

}  // namespace swb
