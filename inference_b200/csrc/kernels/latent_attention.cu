// Latent attention: a token's keys and values of all heads are projections of one cached row [c | k_rot], c the normed latent
// (rank numbers) and k_rot the rotated key part shared by the heads.
//   latent_prep     norm of c (and of a low-rank query latent beside it), rotation of k_rot and of every head's rotated query part,
//                   cache write. Queries that come out of a low-rank latent only exist later: a second launch rotates them.
//   latent_decode   attention in the latent space for steps with few tokens per sequence. The queries were taken through the
//                   key projection, so all heads read the same cached rows, which serve as keys (all columns) and as values
//                   (the latent columns). Everything is computed transposed on the tensor cores: S^T = K Q^T puts 64 keys on
//                   the rows of the MMA and the (few) query rows on its columns, O^T = C^T P^T 128 latent columns on the rows;
//                   C^T is the very tile that served as K, read as an MN-major operand. A page row is fetched once per 16 or
//                   32 query rows. Scores and weights are double-buffered, so the softmax of one tile overlaps the MMAs of
//                   its neighbours and the copies of the next. Partial results of KV splits stay un-normalised in fp32.
//   head_mma        per-head products with the key and value projections around it; the value side merges the splits, adds
//                   the sink to the denominator and applies the output gate.
#include "attention_common.cuh"
#include "common.cuh"
#include "gemm_tcgen05.cuh"

namespace swb {

SWB_REGISTER_STATUS_UNIT(latent_attention);

namespace {

struct LatentPrepParams {
  void* q;                   // queries [T, ldq]: H heads of dn + rp (H 0: none in this launch)
  int ldq;
  void* buf;                 // optional projections [T, ld]: c (rk) at col_c, k_rot (rp) behind it, a query latent (qk) at 0
  int ld, col_c;
  const float* w;            // [rk]
  const float* wq;           // optional [qk]: norm of the query latent, q_rank real columns
  int q_rank, qk;
  float eps;
  const float *cos, *sin;    // [positions, rot / 2]
  const int* positions;
  const long long* slots;    // row of the cache, < 0: none
  void* cache;               // [rows, rk + rc]
  void* q_abs;               // optional [rows, H, rk + rc]: receives the rotated query part at column rk
  const int* q_row;          // optional [T]: row of q_abs of each token, < 0: none
  int T, H, dn, rot, rp, rc, rank, rk;   // rc: columns of the rotated part in `cache` and `q_abs`, zero beyond rp
};

// v <- v / sqrt(mean(v^2) + eps) * w over a row of `n` padded columns (`real` of them in the mean), by one warp; also to dst.
template <typename E>
__device__ __forceinline__ void norm_latent(E* v, const float* w, int n, int real, float eps, E* dst, int lane) {
  float ss = 0.f;
  for (int i = lane * 8; i < n; i += 256) {            // padding columns are zero
    float x[8];
    load_row8(v + i, x);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss = fmaf(x[j], x[j], ss);
  }
  const float r = rsqrtf(warp_sum(ss) / (float)real + eps);
  for (int i = lane * 8; i < n; i += 256) {
    float x[8], y[8];
    load_row8(v + i, x);
    load_row8(w + i, y);
#pragma unroll
    for (int j = 0; j < 8; ++j) x[j] *= r * y[j];
    store_row8(v + i, x);
    if (dst) store_row8(dst + i, x);
  }
}

// One CTA per token: warp 0 norms the latent and warp 1 the query latent, the others rotate in groups of eight dimensions (four pairs).
template <typename E>
__global__ void __launch_bounds__(128) latent_prep_kernel(const LatentPrepParams p) {
  pdl_launch_dependents();
  pdl_wait(TL_ROPE_KV);
  const int t = blockIdx.x, pos = p.positions[t], width = p.rk + p.rc, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  E* row = reinterpret_cast<E*>(p.buf) + (size_t)t * p.ld;
  E* c = row + p.col_c;
  const long long slot = p.buf ? p.slots[t] : -1;
  E* dst = slot >= 0 ? reinterpret_cast<E*>(p.cache) + (size_t)slot * width : nullptr;
  int busy = 0;                                        // warps that norm
  if (p.buf) {
    if (warp == 0) norm_latent(c, p.w, p.rk, p.rank, p.eps, dst, lane);
    busy = 1;
    if (p.wq) {
      if (warp == 1) norm_latent(row, p.wq, p.qk, p.q_rank, p.eps, (E*)nullptr, lane);
      busy = 2;
    }
  }
  if (warp < busy) return;
  const int q_row = !p.q_abs ? -1 : p.q_row ? p.q_row[t] : t, per = p.rc / 8;
  const float* cs = p.cos + (size_t)pos * (p.rot / 2);
  const float* sn = p.sin + (size_t)pos * (p.rot / 2);
  E* q = reinterpret_cast<E*>(p.q) + (size_t)t * p.ldq;
  const int heads = p.H + (p.buf ? 1 : 0);
  for (int i = threadIdx.x - busy * 32; i < heads * per; i += 128 - busy * 32) {    // the heads' queries, then the shared key part
    const int h = i / per, k = i % per * 8;
    E* x = (h < p.H ? q + h * (p.dn + p.rp) + p.dn : c + p.rk) + k;
    float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (k < p.rp) load_row8(x, v);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (k + 2 * j >= p.rot) continue;
      const float a = cs[k / 2 + j], b = sn[k / 2 + j], u = v[2 * j], w = v[2 * j + 1];
      v[2 * j] = u * a - w * b;
      v[2 * j + 1] = w * a + u * b;
    }
    if (k < p.rp) store_row8(x, v);
    E* to = h < p.H ? (q_row >= 0 ? reinterpret_cast<E*>(p.q_abs) + ((size_t)q_row * p.H + h) * width : nullptr) : dst;
    if (to) store_row8(to + p.rk + k, v);
  }
}

// Cached rows of several sequences side by side: out row cu_k[s] + i is row first[s] + i of sequence s (16-byte pieces).
__global__ void __launch_bounds__(256) latent_gather_kernel(const uint4* __restrict__ cache, const int* __restrict__ block_table,
                                                            int max_blocks, int block_size, const int* __restrict__ seqs,
                                                            const int* __restrict__ first, const int* __restrict__ cu_k, int num_seqs, int rows, int pieces, uint4* out) {
  pdl_launch_dependents();
  pdl_wait();
  for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < (long long)rows * pieces; i += (long long)gridDim.x * 256) {
    const int r = (int)(i / pieces), c = (int)(i % pieces);
    const int z = seq_of_token(cu_k, num_seqs, 1, r), k = r - cu_k[z] + (first ? first[z] : 0), s = seqs ? seqs[z] : z;
    const int page = block_table[(size_t)s * max_blocks + k / block_size];
    out[i] = cache[((size_t)page * block_size + k % block_size) * pieces + c];
  }
}

// ---- attention in the latent space ---------------------------------------------------------------------------------
constexpr int DEC_KEYS = 64;                       // keys per tile: the rows of the S^T MMA
constexpr int DEC_STEPS = DEC_KEYS / 16;           // 16-key steps of a tile: the K of an MMA, and what is freed at a time
constexpr int DEC_MAX_TILES = 8;                   // tiles in flight
constexpr int DEC_THREADS = 320;                   // warps 0-3 / 4-7 softmax of half the query rows each, warp 8 TMA, warp 9 MMA

struct LatentDecodeParams {
  const int* block_table;
  int max_blocks, block_size;
  const int* cu_q;           // [num_seqs + 1] or null (uniform_q tokens each)
  const int* kv_lens;
  int uniform_q, H, num_splits, rows_total;
  int window;                // > 0: a query sees only the last `window` keys, its own included
  float scale_log2;
  float* part_o;             // [splits, rows_total, rk]
  float* part_ml;            // [splits, rows_total, 2]: running max (log2 units), sum relative to it
  int rk, latent_atoms, pairs, atoms, rot_steps, ring;   // atoms: 64-column blocks of a cached row, rotated part last
};

struct DecBarriers {
  uint64_t q_full, pv_done, o_final;
  uint64_t s_full[2], p_full[2];                   // tile j uses buffer j & 1
  uint64_t full[DEC_MAX_TILES], empty[DEC_MAX_TILES * DEC_STEPS];
  uint32_t tmem_base;
  int abort;
};

// A tile in shared memory is 8 groups of 8 keys; a group is `atoms` blocks of 8 rows x 64 columns (1 KB, swizzled). As the A
// operand of S^T (K-major) 8-row groups are atoms KB apart; as that of O^T (MN-major: keys are the MMA's K dimension) the next 64
// columns are 1 KB further and the next 8 keys atoms KB.
__device__ __forceinline__ uint64_t dec_desc(uint32_t smem_addr, uint32_t leading, uint32_t stride) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr & 0x3FFFF) >> 4);
  d |= (uint64_t)(leading >> 4) << 16;
  d |= (uint64_t)(stride >> 4) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}
__device__ __forceinline__ void tmem_ld_cols16(uint32_t taddr, float* v) {
  uint32_t r[16];
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]),
        "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
      : "r"(taddr)
      : "memory");
#pragma unroll
  for (int i = 0; i < 16; ++i) v[i] = __uint_as_float(r[i]);
}
__device__ __forceinline__ void tmem_st_cols16(uint32_t taddr, const float* v) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};" ::"r"(taddr),
      "f"(v[0]), "f"(v[1]), "f"(v[2]), "f"(v[3]), "f"(v[4]), "f"(v[5]), "f"(v[6]), "f"(v[7]), "f"(v[8]), "f"(v[9]), "f"(v[10]),
      "f"(v[11]), "f"(v[12]), "f"(v[13]), "f"(v[14]), "f"(v[15])
      : "memory");
}
__device__ __forceinline__ void tmem_ld_cols8(uint32_t taddr, float* v) {
  uint32_t r[8];
  asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7])
               : "r"(taddr)
               : "memory");
#pragma unroll
  for (int i = 0; i < 8; ++i) v[i] = __uint_as_float(r[i]);
}
__device__ __forceinline__ void tmem_st_cols8(uint32_t taddr, const float* v) {
  asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8};" ::"r"(taddr), "f"(v[0]), "f"(v[1]), "f"(v[2]),
               "f"(v[3]), "f"(v[4]), "f"(v[5]), "f"(v[6]), "f"(v[7])
               : "memory");
}
template <int NB>
__device__ __forceinline__ void tmem_st_cols(uint32_t taddr, const float* v) {
  if constexpr (NB == 8) tmem_st_cols8(taddr, v);
  else tmem_st_cols16(taddr, v);
}
template <int NB>
__device__ __forceinline__ void tmem_ld_cols(uint32_t taddr, float* v) {
  if constexpr (NB == 8) tmem_ld_cols8(taddr, v);
  else tmem_ld_cols16(taddr, v);
  tmem_ld_wait();
#pragma unroll
  for (int c = 0; c < NB; ++c) asm volatile("" : "+f"(v[c]));      // uses stay behind the wait
}

// Barrier of the four warps of softmax group `id` (1 or 2) that also agrees on whether everyone is still fine.
__device__ __forceinline__ bool softmax_sync(bool ok, int id) {
  uint32_t all;
  asm volatile(
      "{\n.reg .pred p, q;\nsetp.ne.b32 p, %1, 0;\nbarrier.cta.red.and.pred q, %2, 128, p;\nselp.u32 %0, 1, 0, q;\n}\n"
      : "=r"(all)
      : "r"((uint32_t)ok), "r"(id)
      : "memory");
  return all != 0;
}

// Reduces v[c] over the lanes of the warp for NB columns at once; lane c (mod NB) returns column c. Destroys v.
template <int NB, bool MAX>
__device__ __forceinline__ float reduce_columns(float* v, int lane) {
#pragma unroll
  for (int o = NB / 2; o > 0; o >>= 1) {
    const bool hi = lane & o;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float keep = hi ? v[i + o] : v[i], send = hi ? v[i] : v[i + o];
      const float got = __shfl_xor_sync(0xffffffffu, send, o);
      v[i] = MAX ? fmaxf(keep, got) : keep + got;
    }
  }
#pragma unroll
  for (int o = NB; o < 32; o <<= 1) {
    const float got = __shfl_xor_sync(0xffffffffu, v[0], o);
    v[0] = MAX ? fmaxf(v[0], got) : v[0] + got;
  }
  return v[0];
}

template <int NB>
__global__ void __launch_bounds__(DEC_THREADS, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_kv,
                     const LatentDecodeParams p) {
  constexpr uint32_t Q_ATOM = NB * 128, TMEM_COLS = NB == 16 ? 128 : 256, COL_O = 2 * NB;   // S at [0, NB) and [NB, 2 NB)
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t group_bytes = p.atoms * 1024, tile_bytes = 8 * group_bytes;
  uint8_t* s_q = smem + p.ring * tile_bytes;
  uint8_t* s_p = s_q + p.atoms * Q_ATOM;
  float* red = reinterpret_cast<float*>(s_p + 2 * Q_ATOM);      // [2][4][NB]
  DecBarriers* bars = reinterpret_cast<DecBarriers*>(red + 8 * NB);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  volatile int* abort_flag = &bars->abort;

  pdl_launch_dependents();
  pdl_wait(TL_ATTN_DECODE);
  const int seq = blockIdx.z, split = blockIdx.x, row0 = blockIdx.y * NB;
  const int q_start = p.cu_q ? p.cu_q[seq] : seq * p.uniform_q;
  const int q_len = p.cu_q ? p.cu_q[seq + 1] - q_start : p.uniform_q;
  const int nrows = min(NB, q_len * p.H - row0);
  if (nrows <= 0) return;
  const int kv_len = p.kv_lens[seq], base_row = q_start * p.H + row0;
  // keys that the last row of this block sees
  const int kv_end = min(kv_len, kv_len - q_len + (row0 + nrows - 1) / p.H + 1);
  // first tile that the first row sees
  const int tile_lo = p.window > 0 ? max(kv_len - q_len + row0 / p.H - p.window + 1, 0) / DEC_KEYS : 0;
  const int tiles = (kv_end + DEC_KEYS - 1) / DEC_KEYS, per = (tiles - tile_lo + p.num_splits - 1) / p.num_splits;
  const int t0 = tile_lo + split * per, n_tiles = min(tiles, t0 + per) - t0;
  if (n_tiles <= 0) {
    for (int i = threadIdx.x; i < nrows; i += DEC_THREADS) {
      float* ml = p.part_ml + ((size_t)split * p.rows_total + base_row + i) * 2;
      ml[0] = -INFINITY, ml[1] = 0.f;
    }
    return;
  }
  if (threadIdx.x == 0) {
    mbar_init(&bars->q_full, 1);
    mbar_init(&bars->pv_done, 1);
    mbar_init(&bars->o_final, 1);
    for (int i = 0; i < 2; ++i) mbar_init(&bars->s_full[i], 1), mbar_init(&bars->p_full[i], 256);
    for (int i = 0; i < p.ring; ++i) mbar_init(&bars->full[i], 1);
    for (int i = 0; i < p.ring * DEC_STEPS; ++i) mbar_init(&bars->empty[i], 1);
    bars->abort = 0;
    mbar_fence_init();
  }
  if (warp == 8 && lane == 0) {
    tma_prefetch_desc(&tmap_q);
    tma_prefetch_desc(&tmap_kv);
  }
  if (warp == 9) {
    tmem_alloc(&bars->tmem_base, TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = bars->tmem_base;

  if (warp == 8) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0) {
      mbar_arrive_expect_tx(&bars->q_full, p.atoms * Q_ATOM);
      tma_load_3d(s_q, &tmap_q, &bars->q_full, 0, base_row, 0);
      const int* pages = p.block_table + (size_t)seq * p.max_blocks;
      const int last_group = (kv_len - 1) / 8;
      bool ok = true;
      int started = 0;                               // tiles with copies under way or landed
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int slot = j % p.ring;
        int rows[8];                                 // first cache row of each group; groups past the last repeat it (masked)
#pragma unroll
        for (int g = 0; g < 8; ++g) {
          const int key = min((t0 + j) * 8 + g, last_group) * 8;
          rows[g] = pages[key / p.block_size] * p.block_size + key % p.block_size;
        }
#pragma unroll
        for (int k = 0; k < DEC_STEPS; ++k) {
          ok = ok && mbar_wait(&bars->empty[slot * DEC_STEPS + k], ((j / p.ring) & 1) ^ 1, abort_flag, 711);
          if (!ok) break;
          if (k == 0) {
            mbar_arrive_expect_tx(&bars->full[slot], tile_bytes);
            started = j + 1;
          }
          uint8_t* dst = smem + slot * tile_bytes + 2 * k * group_bytes;
          tma_load_3d(dst, &tmap_kv, &bars->full[slot], 0, rows[2 * k], 0);
          tma_load_3d(dst + group_bytes, &tmap_kv, &bars->full[slot], 0, rows[2 * k + 1], 0);
        }
      }
      if (!ok) {
        // drain: every copy this thread started must land before the CTA's shared memory is released. The last tile may have
        // been started in part; its barrier then expects more than will come, and this (bounded) wait runs out
        volatile int never = 0;
        mbar_wait(&bars->q_full, 0, &never, 712);
        for (int i = max(0, started - p.ring); i < started; ++i) mbar_wait(&bars->full[i % p.ring], (i / p.ring) & 1, &never, 714);
      }
    }
  } else if (warp == 9) {
    // ------------------------------------------------------------------ MMA issuer
    // Two streams: S^T of a tile once its copies have landed (at most one tile ahead of the other stream, because S and P have two
    // buffers), O^T of a tile once its weights are written. Whichever is ready goes first. The warp runs in step, one lane issues.
    constexpr uint32_t IDESC_S = umma_idesc_bf16_f32(DEC_KEYS, NB);
    constexpr uint32_t IDESC_O = umma_idesc_bf16_f32(128, NB) | (1u << 15);     // A is MN-major
    constexpr uint32_t Q16 = Q_ATOM / 16;                                       // descriptors count 16-byte units
    const uint32_t tile16 = tile_bytes / 16, step16 = group_bytes / 8;          // one tile; two groups
    const uint64_t ring_k = dec_desc(smem_u32(smem), 16, group_bytes), ring_mn = dec_desc(smem_u32(smem), 1024, group_bytes),
                   q = umma_desc_kmajor_sw128(smem_u32(s_q)), pp = umma_desc_kmajor_sw128(smem_u32(s_p));
    auto ready = [&](uint64_t* bar, uint32_t phase) { return __all_sync(0xffffffffu, mbar_test_wait(bar, phase)) != 0; };
    bool ok = __all_sync(0xffffffffu, mbar_wait(&bars->q_full, 0, abort_flag, 720));
    int qk = 0, pv = 0, qk_slot = 0, pv_slot = 0;
    uint32_t qk_phase = 0, spins = 0;
    uint64_t idle_since = 0;
    while (ok && pv < n_tiles) {
      if (pv < qk && ready(&bars->p_full[pv & 1], (pv >> 1) & 1)) {
        tc_fence_after_sync();
        if (elect_one()) {
          const uint64_t a = ring_mn + pv_slot * tile16, b = pp + (pv & 1) * Q16;
#pragma unroll
          for (int k = 0; k < DEC_STEPS; ++k) {
            for (int i = 0; i < p.pairs; ++i)
              umma_f16_ss(tmem + COL_O + i * NB, a + k * step16 + i * 128, b + k * 2, IDESC_O, (pv > 0) || (k > 0));
            umma_commit(&bars->empty[pv_slot * DEC_STEPS + k]);
          }
          umma_commit(&bars->pv_done);
        }
        __syncwarp();
        if (++pv_slot == p.ring) pv_slot = 0;
        ++pv, spins = 0;
      } else if (qk < n_tiles && qk <= pv + 1 && ready(&bars->full[qk_slot], qk_phase)) {
        tc_fence_after_sync();
        if (elect_one()) {
          const uint64_t a = ring_k + qk_slot * tile16;
          const uint32_t d = tmem + (qk & 1) * NB;
          for (int i = 0; i < p.latent_atoms; ++i) {
#pragma unroll
            for (int k = 0; k < 4; ++k) umma_f16_ss(d, a + i * 64 + k * 2, q + i * Q16 + k * 2, IDESC_S, (i > 0) || (k > 0));
          }
          for (int k = 0; k < p.rot_steps; ++k)
            umma_f16_ss(d, a + (p.latent_atoms + (k >> 2)) * 64 + (k & 3) * 2, q + (p.latent_atoms + (k >> 2)) * Q16 + (k & 3) * 2, IDESC_S, 1);
          umma_commit(&bars->s_full[qk & 1]);
        }
        __syncwarp();
        if (++qk_slot == p.ring) qk_slot = 0, qk_phase ^= 1;
        ++qk, spins = 0;
      } else if ((++spins & 0xFF) == 0) {              // nothing ready: bounded like every wait
        const uint64_t now = global_timer_ns();
        if (spins == 0x100) idle_since = now;
        if (__any_sync(0xffffffffu, *abort_flag != 0)) ok = false;
        else if (__any_sync(0xffffffffu, now - idle_since > g_wait_limit_ns)) {
          if (lane == 0) {
            *abort_flag = 1;
            report_error(SWB_ERR_WAIT_TIMEOUT, 721, (int)blockIdx.x, pv);
          }
          ok = false;
        }
      }
    }
    __syncwarp();
    if (elect_one()) umma_commit(&bars->o_final);      // also on the abort path: it only tracks MMAs already issued
    __syncwarp();
    if (!ok) {                                         // TMEM must not be freed under MMAs that are still running
      volatile int never = 0;
      mbar_wait(&bars->o_final, 0, &never, 724);
    }
  } else {
    // ------------------------------------------------------------------ softmax: NC query rows per thread. The 64 rows of S^T lie in lanes
    // 0-15 of every 32: those threads hold a key each, the others only take part in the reductions.
    constexpr int NC = NB / 2;
    const int grp = warp >> 2, w4 = warp & 3, r0 = grp * NC;      // this group's first query row of the block
    const uint32_t t_s = tmem + ((uint32_t)(w4 * 32) << 16) + r0, t_o = t_s + COL_O;
    const bool has_key = lane < 16;
    const int key = w4 * 16 + (lane & 15);
    float* red_g = red + grp * 8 * NC;                            // [2][4][NC]
    float m[NC], l[NC];
#pragma unroll
    for (int n = 0; n < NC; ++n) m[n] = -INFINITY, l[n] = 0.f;
    bool ok = true;
    for (int j = 0; j < n_tiles; ++j) {
      float s[NC];
      float* red_j = red_g + (j & 1) * 4 * NC;
      ok = __all_sync(0xffffffffu, mbar_wait(&bars->s_full[j & 1], (j >> 1) & 1, abort_flag, 730));
      if (ok) {
        tc_fence_after_sync();
        tmem_ld_cols<NC>(t_s + (j & 1) * NB, s);
        const int k0 = (t0 + j) * DEC_KEYS;
        if (k0 + DEC_KEYS > kv_len - q_len + row0 / p.H + 1) {      // some key of the tile lies behind the first row
#pragma unroll
          for (int n = 0; n < NC; ++n)
            if (k0 + key > kv_len - q_len + (row0 + r0 + n) / p.H || k0 + key >= kv_len) s[n] = -INFINITY;
        }
        if (p.window > 0 && k0 <= kv_len - q_len + (row0 + nrows - 1) / p.H - p.window) {      // some key is out of the last row's window
#pragma unroll
          for (int n = 0; n < NC; ++n)
            if (k0 + key <= kv_len - q_len + (row0 + r0 + n) / p.H - p.window) s[n] = -INFINITY;
        }
        float v[NC];
#pragma unroll
        for (int n = 0; n < NC; ++n) v[n] = s[n] = has_key ? s[n] : -INFINITY;
        const float top = reduce_columns<NC, true>(v, lane);
        if (lane < NC) red_j[w4 * NC + lane] = top;
      }
      ok = softmax_sync(ok, 1 + grp);
      if (!ok) break;
      float mn[NC];
      bool grow = false;
#pragma unroll
      for (int n = 0; n < NC; n += 4) {
        float4 a = *reinterpret_cast<const float4*>(&red_j[n]);
#pragma unroll
        for (int w = 1; w < 4; ++w) {
          const float4 b = *reinterpret_cast<const float4*>(&red_j[w * NC + n]);
          a.x = fmaxf(a.x, b.x), a.y = fmaxf(a.y, b.y), a.z = fmaxf(a.z, b.z), a.w = fmaxf(a.w, b.w);
        }
        mn[n] = fmaxf(m[n], a.x), mn[n + 1] = fmaxf(m[n + 1], a.y), mn[n + 2] = fmaxf(m[n + 2], a.z), mn[n + 3] = fmaxf(m[n + 3], a.w);
      }
#pragma unroll
      for (int n = 0; n < NC; ++n) grow |= (mn[n] - m[n]) * p.scale_log2 > 8.f;
      if (grow) {                    // the same in every thread of the group: move its rows to their current maximum
        float f[NC];
#pragma unroll
        for (int n = 0; n < NC; ++n) {
          f[n] = mn[n] == -INFINITY ? 1.f : exp2f((m[n] - mn[n]) * p.scale_log2);
          m[n] = mn[n];
          l[n] *= f[n];
        }
        // O may be touched once the PV of the tile before has completed
        if (j > 0) ok = __all_sync(0xffffffffu, mbar_wait(&bars->pv_done, (j - 1) & 1, abort_flag, 732));
        if (j > 0 && ok) {
          tc_fence_after_sync();
          for (int i = 0; i < p.pairs; ++i) {
            float o[NC];
            tmem_ld_cols<NC>(t_o + i * NB, o);
#pragma unroll
            for (int n = 0; n < NC; ++n) o[n] *= f[n];
            tmem_st_cols<NC>(t_o + i * NB, o);
          }
          asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
        }
      }
      uint8_t* dst = s_p + (j & 1) * Q_ATOM + r0 * 128 + (key & 7) * 2;
#pragma unroll
      for (int n = 0; n < NC; ++n) {
        const float e = exp2f(fmaf(s[n], p.scale_log2, m[n] == -INFINITY ? 0.f : -m[n] * p.scale_log2));
        l[n] += e;
        if (has_key) *reinterpret_cast<bf16*>(dst + n * 128 + (((key >> 3) ^ (n & 7)) << 4)) = __float2bfloat16(e);
      }
      fence_proxy_async_smem();
      tc_fence_before_sync();
      mbar_arrive(&bars->p_full[j & 1]);
    }
    if (ok) ok = __all_sync(0xffffffffu, mbar_wait(&bars->o_final, 0, abort_flag, 731));
    float* lred = red_g + (n_tiles & 1) * 4 * NC;    // the half that the last tile did not use
    {
      float v[NC];
#pragma unroll
      for (int n = 0; n < NC; ++n) v[n] = l[n];
      const float sum = reduce_columns<NC, false>(v, lane);
      if (lane < NC) lred[w4 * NC + lane] = sum;
    }
    if (softmax_sync(ok, 1 + grp)) {
      tc_fence_after_sync();
      const size_t base = (size_t)split * p.rows_total + base_row + r0;
#pragma unroll
      for (int n = 0; n < NC; ++n)
        if (w4 * 32 + lane == n && r0 + n < nrows) {
          float* ml = p.part_ml + (base + n) * 2;
          ml[0] = m[n] * p.scale_log2;
          ml[1] = lred[n] + lred[NC + n] + lred[2 * NC + n] + lred[3 * NC + n];
        }
      for (int i = 0; i < p.pairs; ++i) {
        float o[NC];
        tmem_ld_cols<NC>(t_o + i * NB, o);
        const int col = i * 128 + w4 * 32 + lane;
#pragma unroll
        for (int n = 0; n < NC; ++n)
          if (r0 + n < nrows && col < p.rk) p.part_o[(base + n) * p.rk + col] = o[n];
      }
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 9) {
    tc_fence_after_sync();
    tmem_dealloc(tmem, TMEM_COLS);
  }
}

// ---- per-head products ----------------------------------------------------------------------------------------------
struct HeadMmaParams {
  const bf16* a;             // [tokens, heads, K] strided (MERGE: unused)
  long long a_tok;
  int a_head;
  const bf16* w;             // [H, N, K]
  bf16* out;                 // [tokens, heads, N] strided
  long long out_tok;
  int out_head;
  const bf16* gate;          // optional [tokens, >= H] logits
  long long gate_tok;
  const int *rows_in, *rows_out;   // optional: token of row i in `a`, and in `out` and `gate`
  int n, H, N, K;
  // MERGE: a is the merged split partials
  const float *part_o, *part_ml, *sink;
  int num_splits, rows_total;
  // optional (not MERGE): columns [rot_in, rot_in + rot_pad) of a's head rows are rotated (the first `rot`, neighbouring pairs) and
  // stored at column rot_out of out's head rows, zero up to rot_cols
  const float *cos, *sin;
  const int* positions;
  int rot_in, rot_out, rot, rot_pad, rot_cols;
};

constexpr int HM_TOK = 16;   // tokens per CTA: the rows of the MMA

constexpr int HM_WARPS = 8;

constexpr int HM_SLABS = 16; // 32-wide K slabs whose weights are fetched ahead (K <= 512)

// out[t, h, n] = gate * sum_k a[t, h, k] w[h, n, k], eight columns per warp. A lane's eight consecutive k are spread over two
// MMAs the same way for both operands, so every load is 16 bytes. The weights depend on no earlier kernel: they are fetched in
// front of the dependency wait.
template <bool MERGE>
__global__ void __launch_bounds__(HM_WARPS * 32) head_mma_kernel(const HeadMmaParams p) {
  extern __shared__ __align__(16) uint8_t hm_smem[];
  const int ld = p.K + 8;
  bf16* sa = reinterpret_cast<bf16*>(hm_smem);                             // [16][K + 8]
  float* wt = reinterpret_cast<float*>(hm_smem + (size_t)HM_TOK * ld * 2); // [16][32]: weight of each split
  const int h = blockIdx.y, t0 = blockIdx.z * HM_TOK, m = min(HM_TOK, p.n - t0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  const int n0 = (blockIdx.x * HM_WARPS + warp) * 8;
  const bf16* wr = p.w + ((size_t)h * p.N + min(n0 + g, p.N - 1)) * p.K + t4 * 8;
  uint4 b[HM_SLABS];
#pragma unroll
  for (int s = 0; s < HM_SLABS; ++s)
    b[s] = s * 32 + t4 * 8 < p.K ? __ldg(reinterpret_cast<const uint4*>(wr + s * 32)) : make_uint4(0, 0, 0, 0);
  pdl_launch_dependents();
  pdl_wait();
  auto token_in = [&](int i) { return p.rows_in ? p.rows_in[t0 + i] : t0 + i; };
  auto token_out = [&](int i) { return p.rows_out ? p.rows_out[t0 + i] : t0 + i; };
  if constexpr (MERGE) {
    for (int i = warp; i < m; i += HM_WARPS) {         // a warp per token: lane = split
      const size_t row = (size_t)token_in(i) * p.H + h;
      const float sk = p.sink ? p.sink[h] * 1.4426950408889634f : -INFINITY;
      float2 ml = make_float2(-INFINITY, 0.f);
      if (lane < p.num_splits) ml = *reinterpret_cast<const float2*>(p.part_ml + ((size_t)lane * p.rows_total + row) * 2);
      const float top = fmaxf(warp_max(ml.x), sk), w = ml.y > 0.f ? exp2f(ml.x - top) : 0.f;
      const float den = warp_sum(w * ml.y) + (p.sink ? exp2f(sk - top) : 0.f);
      wt[i * 32 + lane] = w / den;
    }
    __syncthreads();
    const int nv = p.K / 4;
    for (int idx = threadIdx.x; idx < HM_TOK * nv; idx += HM_WARPS * 32) {
      const int i = idx / nv, c = (idx % nv) * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i < m) {
        const float* o = p.part_o + ((size_t)token_in(i) * p.H + h) * p.K + c;
        const size_t step = (size_t)p.rows_total * p.K;
        for (int s0 = 0; s0 < p.num_splits; s0 += 8) {
          float4 x[8];
          float w[8];
#pragma unroll
          for (int s = 0; s < 8; ++s) {                // an empty split wrote nothing and is not read
            w[s] = s0 + s < p.num_splits ? wt[i * 32 + s0 + s] : 0.f;
            x[s] = w[s] != 0.f ? *reinterpret_cast<const float4*>(o + (s0 + s) * step) : make_float4(0.f, 0.f, 0.f, 0.f);
          }
#pragma unroll
          for (int s = 0; s < 8; ++s)
            v.x = fmaf(w[s], x[s].x, v.x), v.y = fmaf(w[s], x[s].y, v.y), v.z = fmaf(w[s], x[s].z, v.z), v.w = fmaf(w[s], x[s].w, v.w);
        }
      }
      *reinterpret_cast<uint2*>(sa + i * ld + c) = make_uint2(attn::pack_bf16(v.x, v.y), attn::pack_bf16(v.z, v.w));
    }
  } else {
    const int nv = p.K / 8;
    for (int idx = threadIdx.x; idx < HM_TOK * nv; idx += HM_WARPS * 32) {
      const int i = idx / nv, c = (idx % nv) * 8;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (i < m) v = *reinterpret_cast<const uint4*>(p.a + token_in(i) * p.a_tok + (long long)h * p.a_head + c);
      *reinterpret_cast<uint4*>(sa + i * ld + c) = v;
    }
  }
  if (!MERGE && p.cos && blockIdx.x == 0) {
    const int per = p.rot_cols / 8;
    for (int idx = threadIdx.x; idx < m * per; idx += HM_WARPS * 32) {
      const int i = idx / per, k = idx % per * 8, ti = token_in(i);
      const bf16* x = p.a + ti * p.a_tok + (long long)h * p.a_head + p.rot_in + k;
      const float* cs = p.cos + (size_t)p.positions[ti] * (p.rot / 2);
      const float* sn = p.sin + (size_t)p.positions[ti] * (p.rot / 2);
      float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      if (k < p.rot_pad) load_row8(x, v);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        if (k + 2 * j >= p.rot) continue;
        const float c = cs[k / 2 + j], s = sn[k / 2 + j], u = v[2 * j], w = v[2 * j + 1];
        v[2 * j] = u * c - w * s;
        v[2 * j + 1] = w * c + u * s;
      }
      store_row8(p.out + token_out(i) * p.out_tok + (long long)h * p.out_head + p.rot_out + k, v);
    }
  }
  __syncthreads();
  if (n0 >= p.N) return;
  float acc[4] = {0.f, 0.f, 0.f, 0.f};
  auto slab = [&](int k, uint4 w) {
    uint4 lo = make_uint4(0, 0, 0, 0), hi = lo;
    if (k + t4 * 8 < p.K) {
      lo = *reinterpret_cast<const uint4*>(sa + g * ld + k + t4 * 8);
      hi = *reinterpret_cast<const uint4*>(sa + (g + 8) * ld + k + t4 * 8);
    }
    const uint32_t a0[4] = {lo.x, hi.x, lo.y, hi.y}, a1[4] = {lo.z, hi.z, lo.w, hi.w};
    attn::mma_16816(acc, a0, w.x, w.y);
    attn::mma_16816(acc, a1, w.z, w.w);
  };
#pragma unroll
  for (int s = 0; s < HM_SLABS; ++s)
    if (s * 32 < p.K) slab(s * 32, b[s]);
  for (int k = HM_SLABS * 32; k < p.K; k += 32)
    slab(k, k + t4 * 8 < p.K ? __ldg(reinterpret_cast<const uint4*>(wr + k)) : make_uint4(0, 0, 0, 0));
  const int n = n0 + t4 * 2;
  if (n >= p.N) return;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int i = g + r * 8;
    if (i >= m) continue;
    const int tok = token_out(i);
    float s = 1.f;
    if (p.gate) s = 1.f / (1.f + expf(-__bfloat162float(p.gate[tok * p.gate_tok + h])));
    *reinterpret_cast<uint32_t*>(p.out + tok * p.out_tok + (long long)h * p.out_head + n) = attn::pack_bf16(acc[2 * r] * s, acc[2 * r + 1] * s);
  }
}

template <bool MERGE>
int launch_head_mma(const HeadMmaParams& p, cudaStream_t s) {
  const size_t smem = (size_t)HM_TOK * (p.K + 8) * 2 + (MERGE ? HM_TOK * 32 * 4 : 0);
  constexpr int COLS = HM_WARPS * 8;
  return launch_kernel(head_mma_kernel<MERGE>, dim3((p.N + COLS - 1) / COLS, p.H, (p.n + HM_TOK - 1) / HM_TOK), dim3(HM_WARPS * 32), smem,
                       s, p);
}

template <int NB>
int launch_latent_decode(const CUtensorMap& tq, const CUtensorMap& tk, LatentDecodeParams p, int seqs, int max_rows, cudaStream_t s) {
  constexpr size_t LIMIT = 227 * 1024;
  const size_t fixed = 1024 + (size_t)(p.atoms + 2) * NB * 128 + 8 * NB * 4 + sizeof(DecBarriers), tile = (size_t)p.atoms * 8192;
  if (fixed + 2 * tile > LIMIT) return -3;                                  // two tiles are held at a time
  p.ring = (int)((LIMIT - fixed) / tile);
  if (p.ring > DEC_MAX_TILES) p.ring = DEC_MAX_TILES;
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64 || !configured[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<NB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)LIMIT);
    if (e != cudaSuccess) return -(int)e;
    if (dev >= 0 && dev < 64) configured[dev] = true;
  }
  const size_t smem = fixed + p.ring * tile;
  return launch_kernel(latent_decode_kernel<NB>, dim3(p.num_splits, (max_rows + NB - 1) / NB, seqs), dim3(DEC_THREADS), smem, s, tq, tk, p);
}

}  // namespace
}  // namespace swb

extern "C" {

// See LatentPrepParams. buf null: only the queries of q are rotated; H 0: only the latents.
int swb_latent_prep(void* q, int ldq, void* buf, int ld, int col_c, const float* w, const float* wq, int q_rank, int qk, float eps,
                    const float* cos, const float* sin, const int* positions, const long long* slots, void* cache, void* q_abs,
                    const int* q_row, int T, int H, int dn, int rot, int rp, int rc, int rank, int rk, int fp32, void* stream) {
  using namespace swb;
  if (T <= 0) return 0;
  if (H < 0 || (H > 0 && !q) || (!buf && H == 0) || dn <= 0 || rot <= 0 || (rot % 2) || rot > rp || ((dn | rp | rc | rk | ldq) % 8) || rc < rp)
    return -3;
  if (buf && (((ld | col_c) % 8) || !w || rank <= 0 || rank > rk || !cache || !slots)) return -3;
  if (wq && (!buf || (qk % 8) || q_rank <= 0 || q_rank > qk || qk > col_c)) return -3;
  const LatentPrepParams p{q, ldq, buf, ld, col_c, w, wq, q_rank, qk, eps, cos, sin, positions, slots, cache, q_abs, q_row, T, H, dn, rot,
                           rp, rc, rank, rk};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return fp32 ? launch_kernel(latent_prep_kernel<float>, dim3((unsigned)T), dim3(128), 0, s, p)
              : launch_kernel(latent_prep_kernel<bf16>, dim3((unsigned)T), dim3(128), 0, s, p);
}

// out [rows, width] bf16 <- the cached rows of num_seqs sequences (seqs: their indices in block_table, null: 0, 1, ...), those of
// sequence s from its row first[s] (null: 0) on at [cu_k[s], cu_k[s + 1]). width % 8 == 0.
int swb_latent_gather(const void* cache, const int* block_table, int max_blocks, int block_size, const int* seqs, const int* first,
                      const int* cu_k, int num_seqs, int rows, int width, void* out, void* stream) {
  using namespace swb;
  if (rows <= 0) return 0;
  if (width % 8 || num_seqs <= 0 || block_size <= 0 || ((reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(out)) & 15)) return -3;
  const long long n = (long long)rows * (width / 8);
  const unsigned grid = (unsigned)((n + 255) / 256 < 148 * 8 ? (n + 255) / 256 : 148 * 8);
  return launch_kernel(latent_gather_kernel, dim3(grid), dim3(256), 0, reinterpret_cast<cudaStream_t>(stream),
                       reinterpret_cast<const uint4*>(cache), block_table, max_blocks, block_size, seqs, first, cu_k, num_seqs, rows, width / 8,
                       reinterpret_cast<uint4*>(out));
}

// Prefill attention on expanded keys and values; see attn_latent_tcgen05_launch.
int swb_latent_prefill(const void* q, long long q_stride_tok, const void* k, const void* v, long long kv_stride_tok, const void* k2,
                       long long k2_stride_tok, int key_rows, void* out, long long out_stride_tok, int num_seqs, int max_q_len,
                       int total_tokens, int H, int d1, int d2, int Dv, float scale, const float* sink, const void* gate,
                       long long gate_stride, const int* cu_q, const int* seqs, const int* cu_k, int window, void* stream) {
  using namespace swb;
  if (num_seqs <= 0 || total_tokens <= 0) return 0;
  if (max_q_len <= 0 || key_rows <= 0) return -3;
  return attn_latent_tcgen05_launch(q, q_stride_tok, k, v, kv_stride_tok, k2, k2_stride_tok, key_rows, out, out_stride_tok, num_seqs,
                                    max_q_len, total_tokens, H, d1, d2, Dv, scale, sink, gate, gate_stride, cu_q, seqs, cu_k,
                                    reinterpret_cast<cudaStream_t>(stream), window);
}

// Attention of q_abs [T * H, rk + rp] over the cached rows [num_blocks * block_size, rk + rc] (q rows likewise) into
// split partials (see LatentDecodeParams). rc: the rotated part with its padding (zero in q), a multiple of 64; rot of it is used. max_q: most tokens of a sequence.
int swb_latent_decode(const void* q_abs, const void* cache, int num_blocks, int block_size, const int* block_table, int max_blocks,
                      const int* cu_q, const int* kv_lens, int n_seqs, int uniform_q, int max_q, int T, int H, int rk,
                      int rc, int rot, float scale, int num_splits, int window, float* part_o, float* part_ml, void* stream) {
  using namespace swb;
  if (T <= 0 || n_seqs <= 0) return 0;
  if (rk % 64 || rk < 64 || rk > 512 || rc % 64 || rot < 1 || rot > rc || rc > 128 || block_size < 8 || block_size % 8 ||
      !(scale > 0.f) || num_splits < 1 || num_splits > 32 || H < 1 || max_q < 1 || window < 0 || (!cu_q && uniform_q < 1))
    return -3;
  if ((reinterpret_cast<uintptr_t>(q_abs) | reinterpret_cast<uintptr_t>(cache)) & 15) return -3;
  LatentDecodeParams p{};
  p.block_table = block_table, p.max_blocks = max_blocks, p.block_size = block_size;
  p.cu_q = cu_q, p.kv_lens = kv_lens;
  p.uniform_q = uniform_q, p.H = H, p.num_splits = num_splits, p.rows_total = T * H, p.window = window;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.part_o = part_o, p.part_ml = part_ml;
  p.rk = rk, p.latent_atoms = rk / 64, p.pairs = (p.latent_atoms + 1) / 2, p.atoms = (rk + rc) / 64, p.rot_steps = (rot + 15) / 16;
  const int rows = max_q * H, nb = rows <= 16 ? 16 : 32;
  CUtensorMap tq, tk;
  int err = make_tmap_bf16_blocks(&tq, q_abs, T * H, rk + rc, rk + rc, nb);
  if (err) return err;
  err = make_tmap_bf16_blocks(&tk, cache, num_blocks * block_size, rk + rc, rk + rc, 8);
  if (err) return err;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return nb == 16 ? launch_latent_decode<16>(tq, tk, p, n_seqs, rows, s) : launch_latent_decode<32>(tq, tk, p, n_seqs, rows, s);
}

// out[t, h, n] = sigmoid(gate[t, h]) sum_k a[t, h, k] w[h, n, k] in bf16 for n tokens: row i is token rows_in[i] of a and
// rows_out[i] of out and gate (null: i). With cos, the rotated query parts travel along (see HeadMmaParams). With
// part_o, a[t, h] are the merged split partials of swb_latent_decode (K = rk), with optional sinks, and `a` is unused. K, N and all strides
// are multiples of 8.
int swb_head_mma(const void* a, long long a_tok, int a_head, const void* w, void* out, long long out_tok, int out_head, const void* gate,
                 long long gate_tok, const int* rows_in, const int* rows_out, int n, int H, int N, int K, const float* part_o, const float* part_ml,
                 const float* sink, int num_splits, int rows_total, const float* cos, const float* sin, const int* positions, int rot_in,
                 int rot_out, int rot, int rot_pad, int rot_cols, void* stream) {
  using namespace swb;
  if (n <= 0 || H <= 0) return 0;
  if (cos && (part_o || !sin || !positions || rot < 2 || (rot % 2) || rot > rot_pad || rot_pad > rot_cols || ((rot_in | rot_out | rot_pad | rot_cols) % 8) ||
              (reinterpret_cast<uintptr_t>(out) & 15)))
    return -3;
  if (N < 8 || N % 8 || K < 8 || K % 8 || K > 1024 || (out_tok % 8) || (out_head % 8) || (part_o && (!part_ml || num_splits > 32)) ||
      (!part_o && (!a || (a_tok % 8) || (a_head % 8) || (reinterpret_cast<uintptr_t>(a) & 15))) ||
      (reinterpret_cast<uintptr_t>(w) & 15) || (reinterpret_cast<uintptr_t>(out) & 3))
    return -3;
  const HeadMmaParams p{reinterpret_cast<const bf16*>(a), a_tok, a_head, reinterpret_cast<const bf16*>(w), reinterpret_cast<bf16*>(out),
                        out_tok, out_head, reinterpret_cast<const bf16*>(gate), gate_tok, rows_in, rows_out, n, H, N, K, part_o, part_ml, sink,
                        num_splits, rows_total, cos, sin, positions, rot_in, rot_out, rot, rot_pad, rot_cols};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return part_o ? launch_head_mma<true>(p, s) : launch_head_mma<false>(p, s);
}

}  // extern "C"
