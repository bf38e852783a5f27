// Dense (non-causal) flash attention on the 5th-generation tensor cores, head dim 128, bf16 in / bf16 out.
//
// One CTA owns 256 query rows of one head (two 128-row tiles, "q0" and "q1") and walks the keys in tiles of 128.
//   warp 8 (one lane)   TMA producer: Q once, then K and V tiles through two 2-stage rings (4-D tensor maps over
//                       [d, head, token, batch], 64-column boxes, 128-byte swizzle).
//   warp 9 (one lane)   tcgen05.mma issuer. S_q = Q_q K^T accumulates into TMEM; O_q += P_q V reads P from TMEM
//                       (P overwrites the first half of S in place as packed bf16) and V from shared memory as an
//                       MN-major operand, so V needs no transpose. Issue order
//                           S0(0) S1(0) | PV0(j) S0(j+1) PV1(j) S1(j+1) ...
//                       keeps the tensor pipe busy with one tile's MMAs while the other tile is in softmax.
//   warps 0-3 / 4-7     softmax warpgroups for q0 / q1: thread = row. tcgen05.ld the S row, running max with lazy
//                       rescale (O is only rescaled when the max grew by more than 2^8), exp2, tcgen05.st of P.
// TMEM map (512 columns): [0,128) S0/P0, [128,256) O0, [256,384) S1/P1, [384,512) O1.
// It replaces the mma.sync kernel for the FLUX joint attention (reference: candle-gen-flux/src/ip_dit.rs:64-85 runs
// SDPA through cuBLAS matmuls + softmax, or FlashAttention-2 sm80 kernels).
// Every wait is bounded; on expiry the CTA raises its abort flag, drains its own copies, frees TMEM and returns.
#include "attention_common.cuh"
#include "common.cuh"

#include <cuda.h>
#include <cudaTypedefs.h>

#include <mutex>
#include <unordered_map>

namespace swb {

SWB_REGISTER_STATUS_UNIT(attention_tcgen05);

namespace {

constexpr int BM = 128;          // query rows per tile (two tiles per CTA)
constexpr int BN = 128;          // keys per tile
constexpr int MAX_STAGES = 2;
constexpr int THREADS = 320;
constexpr uint32_t ATOM_BYTES = BM * 64 * 2;       // 16 KB: 128 rows of one 64-column swizzle atom
// Tile widths of q / k (QK) and of v (VD). 128 is two swizzle atoms per tile, 64 one atom (half the shared memory and half the
// MMA work of the padded path); q and k of latent attention take up to three, which leaves room for one V stage.
template <int QK, int VD>
struct FaCfg {
  static_assert((QK == 64 || QK == 128 || QK == 192) && (VD == 64 || VD == 128), "tile widths");
  static constexpr int ATOMS = QK / 64, V_ATOMS = VD / 64;
  static constexpr int K_STAGES = 2, V_STAGES = QK == 192 ? 1 : 2;
  static constexpr uint32_t TILE_BYTES = BM * QK * 2, V_TILE_BYTES = BM * VD * 2;
  static constexpr uint32_t SMEM_Q = 0;                                   // 2 tiles
  static constexpr uint32_t SMEM_K = 2 * TILE_BYTES;
  static constexpr uint32_t SMEM_V = SMEM_K + K_STAGES * TILE_BYTES;
  static constexpr uint32_t SMEM_BAR = SMEM_V + V_STAGES * V_TILE_BYTES;
  static constexpr size_t SMEM_BYTES = SMEM_BAR + 256 + 1024 /*alignment slack*/;
  static constexpr int ROW_BYTES = VD * 2;                                // one output row of one head
  static constexpr int CHUNKS = ROW_BYTES / 16;                           // 16-byte chunks per row
};
constexpr uint32_t TMEM_COLS = 512;
constexpr uint32_t COL_S0 = 0, COL_O0 = 128, COL_S1 = 256, COL_O1 = 384;
constexpr float RESCALE_THRESHOLD = 8.f;           // in log2 units

// Sequence-parallel return path: query row g (global token index, batch 1) belongs to rank
// (g < split ? g / n0 : (g - split) / n1) at local row (g < split ? g % n0 : n0 + (g - split) % n1); the output row is
// stored straight into that rank's buffer at column col_offset + head * 128.
struct OutScatter {
  bf16* peer[8];
  int enabled, split, n0, n1, col_offset;
};

struct FaParams {
  OutScatter scatter;
  bf16* out;
  long long out_stride_tok;   // elements; token index = b * q_len + s
  int q_len, kv_len, Hq, Hkv;
  float scale_log2;
  int tiles;   // query tiles per CTA: 2 (MMAs of one tile overlap the softmax of the other) or 1 (twice the CTAs)
  int causal;  // key j attends to query i only if j <= i (sequences start at position 0: fresh prefill)
  const int* cu_q;   // optional [num_seqs + 1] token offsets: blockIdx.z is then a sequence of a packed batch
  // Paged keys / values (prefill on top of earlier context): tmap_k / tmap_v then describe the page pool
  // [page, kv head, row in page, d]; sequence z owns pages block_table[z * max_blocks + i] and kv_lens[z] keys, and
  // its queries are the last q_len of those positions (bottom-right aligned causal mask). Needs cu_q.
  const int* kv_lens;
  const int* block_table;
  int max_blocks, block_size;
  // Extended problems (the EXT instantiations only):
  int chunk;           // > 0: query i sees key j <= i only if floor(i / chunk) == floor(j / chunk), positions of the sequence
  const float* sink;   // optional [Hq]: exp(sink[h]) joins the softmax denominator (no key, no value, not scaled)
  int window;          // > 0: query i sees only keys j > i - window
  int v_dim;           // width of the v heads and of the output heads (<= VD; the tile is zero filled beyond it)
  attn::DiffAttn diff; // DIFF only
  int v_heads;         // > 0: blockIdx.y runs over (query head, value head); every query head is applied to all value heads
  const bf16* out_gate;         // optional logits in the layout of a token's output: out is scaled by their sigmoid
  long long out_gate_stride;
  // Latent attention (LAT): q and k in two parts, k's second part shared by the heads; keys and values are rows
  // [cu_k[z], cu_k[z + 1]) of one flat axis (null: those of the queries), the queries the last positions of them.
  const int* seqs;     // optional: sequence of blockIdx.z (cu_q is indexed by it, cu_k by blockIdx.z)
  const int* cu_k;
  const bf16* gate;    // optional [tokens, >= Hq] logits: head outputs are scaled by their sigmoid
  long long gate_stride;
  int first_atoms;     // 64-column atoms of the first part; the second takes the rest of the tile
};

__device__ __forceinline__ void tma_load_4d(void* smem_dst, const void* tmap, uint64_t* bar, int c0, int c1, int c2,
                                            int c3) {
  asm volatile(
      "cp.async.bulk.tensor.4d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4, %5}], [%6];"
      ::"r"(smem_u32(smem_dst)),
      "l"(reinterpret_cast<uint64_t>(tmap)), "r"(c0), "r"(c1), "r"(c2), "r"(c3), "r"(smem_u32(bar))
      : "memory");
}

// D[tmem] (+)= A[tmem, packed bf16] * B[smem desc]
__device__ __forceinline__ void umma_f16_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t bdesc, uint32_t idesc,
                                            uint32_t accumulate) {
  asm volatile(
      "{\n"
      ".reg .pred p;\n"
      "setp.ne.b32 p, %4, 0;\n"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n"
      "}\n" ::"r"(tmem_d),
      "r"(tmem_a), "l"(bdesc), "r"(idesc), "r"(accumulate)
      : "memory");
}

// V tile as the B operand of O += P V: rows are keys (the MMA K dimension), 64 head-dim columns per 128-byte row
// (MN-major), 8-key groups 1024 bytes apart, the second 64-column block one atom (16 KB) further.
__device__ __forceinline__ uint64_t umma_desc_mnmajor_sw128(uint32_t smem_addr) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr & 0x3FFFF) >> 4);
  d |= (uint64_t)(ATOM_BYTES >> 4) << 16;   // leading byte offset: next 64-element block along N
  d |= (uint64_t)(1024 >> 4) << 32;         // stride byte offset: next 8-row group along K
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}

// 32 consecutive 32-bit columns of this thread's TMEM lane (no wait inside).
__device__ __forceinline__ void tmem_ld_x32(uint32_t taddr, uint32_t* r) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
      "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,"
      "%30,%31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
        "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]),
        "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]),
        "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
      : "r"(taddr)
      : "memory");
}
__device__ __forceinline__ void tmem_st_x32(uint32_t taddr, const uint32_t* r) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,"
      "%31,%32};" ::"r"(taddr),
      "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]),
      "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]), "r"(r[18]),
      "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]),
      "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
      : "memory");
}
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp_approx(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t pack_bf16x2(float lo, float hi) {
  __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&h);
}

// tanh(x) / x on |x| <= 1 as a polynomial in x^2: a least-squares fit reweighted towards equal ripples; |error of tanh| < 2.4e-7.
constexpr float TANH_0 = 0.99999685f, TANH_1 = -0.33324004f, TANH_2 = 0.13253525f, TANH_3 = -0.05097286f, TANH_4 = 0.01611418f,
                TANH_5 = -0.00283947f;
constexpr float MAX_FIXED_CAP = 64.f;      // sums of exp(cap) over 2^20 keys stay finite in fp32

struct Barriers {
  uint64_t q_full;
  uint64_t k_full[MAX_STAGES], k_empty[MAX_STAGES];
  uint64_t v_full[MAX_STAGES], v_empty[MAX_STAGES];
  uint64_t s_full[2];   // MMA -> softmax q: S_q of the current key tile is complete
  uint64_t p_full[2];   // softmax q -> MMA: P_q is in TMEM (128 arrivals)
  uint64_t o_final;     // every MMA of the CTA has completed
  uint32_t tmem_base;
  int abort;
};

// 168 registers per thread is the cap for ten warps: two of the four scheduler partitions hold three warps, and a
// partition's file is 16 K registers (a build with 200 registers per thread does not launch).
// EXT adds chunked and windowed masking, attention sinks, output gates, values of every head for every query head, and head widths below the tile widths (q . k and P V then run over zero
// columns that the tensor maps fill in). LAT adds what latent attention needs: two-part q / k, key ranges, output gates.
// DIFF is differential attention: the two tiles of a CTA are the two softmax maps of the same 128 query rows. Each map's keys are
// one 64-column atom of the K tile (columns of the other map that fall into it meet zero columns of q), the V tile serves both, and
// the second map's result is handed to the first one's threads through shared memory for the difference and its norm. DIFF 2 is for
// caps up to MAX_FIXED_CAP: the scores are bounded, so the exponentials are taken as they are, without a running maximum.
template <int QK, int VD, bool EXT, bool LAT, int DIFF>
__global__ void __launch_bounds__(THREADS, 1)
attn_dense_tcgen05_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                          const __grid_constant__ CUtensorMap tmap_v, const __grid_constant__ CUtensorMap tmap_q2,
                          const __grid_constant__ CUtensorMap tmap_k2, const FaParams p) {
  using C = FaCfg<QK, VD>;
  constexpr int K_STAGES = C::K_STAGES, V_STAGES = C::V_STAGES, V_ATOMS = C::V_ATOMS;
  constexpr uint32_t TILE_BYTES = C::TILE_BYTES, V_TILE_BYTES = C::V_TILE_BYTES, SMEM_Q = C::SMEM_Q, SMEM_K = C::SMEM_K, SMEM_V = C::SMEM_V, SMEM_BAR = C::SMEM_BAR;
  constexpr int ATOMS = C::ATOMS, ROW_BYTES = C::ROW_BYTES, CHUNKS = C::CHUNKS;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  Barriers* bars = reinterpret_cast<Barriers*>(smem + SMEM_BAR);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  constexpr int TILE_STEP = DIFF ? 0 : BM;                  // query rows between the two tiles of a CTA
  const int cta_rows = DIFF ? BM : p.tiles * BM;
  const int q_base = blockIdx.x * cta_rows;
  constexpr bool WIDE = EXT && !LAT && DIFF == 0;             // v_heads and out_gate are looked at
  const int head = WIDE && p.v_heads > 0 ? blockIdx.y / p.v_heads : blockIdx.y;
  // packed variable-length batch: this CTA's sequence covers tokens [tok0, tok0 + q_len) of one flat token axis
  const int seq = (LAT && p.seqs) ? p.seqs[blockIdx.z] : blockIdx.z;
  const int tok0 = p.cu_q ? p.cu_q[seq] : 0;
  const int q_len = p.cu_q ? p.cu_q[seq + 1] - tok0 : p.q_len;
  const bool paged = !LAT && p.block_table != nullptr, ranged = LAT && p.cu_k;
  const int key0_row = ranged ? p.cu_k[blockIdx.z] : tok0;
  const int kv_len = paged ? p.kv_lens[blockIdx.z] : ranged ? p.cu_k[blockIdx.z + 1] - key0_row : (p.cu_q ? q_len : p.kv_len);
  const int coff = paged || ranged ? max(kv_len - q_len, 0) : 0;   // position of query 0 among the sequence's keys
  const int batch = p.cu_q ? 0 : blockIdx.z;
  if (q_base >= q_len || kv_len <= 0) return;   // uniform for the whole CTA, before any barrier or TMEM allocation
  const int kv_head = head / (p.Hq / p.Hkv), v_head = WIDE && p.v_heads > 0 ? blockIdx.y % p.v_heads : kv_head;
  const int kv_end = p.causal ? min(kv_len, q_base + cta_rows + coff) : kv_len;
  // first key that a row sees, and first key tile that any row of this CTA sees (rows are ascending, so the first row's is lowest)
  auto first_key_of = [&](int pos) {
    int first = p.chunk > 0 ? pos / p.chunk * p.chunk : 0;
    if (p.window > 0) first = max(first, pos - p.window + 1);
    return first;
  };
  const int j0 = EXT ? first_key_of(q_base + coff) / BN : 0;
  const int n_tiles = (kv_end + BN - 1) / BN - j0;
  volatile int* abort_flag = &bars->abort;

  if (threadIdx.x == 0) {
    mbar_init(&bars->q_full, 1);
    for (int s = 0; s < MAX_STAGES; ++s) {
      mbar_init(&bars->k_full[s], 1);
      mbar_init(&bars->k_empty[s], 1);
      mbar_init(&bars->v_full[s], 1);
      mbar_init(&bars->v_empty[s], 1);
    }
    for (int q = 0; q < 2; ++q) {
      mbar_init(&bars->s_full[q], 1);
      mbar_init(&bars->p_full[q], BM);
    }
    mbar_init(&bars->o_final, 1);
    bars->abort = 0;
    mbar_fence_init();
  }
  if (warp == 8 && lane == 0) {
    tma_prefetch_desc(&tmap_q);
    tma_prefetch_desc(&tmap_k);
    tma_prefetch_desc(&tmap_v);
    if constexpr (LAT) {
      tma_prefetch_desc(&tmap_q2);
      tma_prefetch_desc(&tmap_k2);
    }
  }
  if (warp == 9) {
    tmem_alloc(&bars->tmem_base, TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = bars->tmem_base;
  pdl_launch_dependents();
  pdl_wait();

  if (warp == 8) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0) {
      mbar_arrive_expect_tx(&bars->q_full, DIFF ? 2 * ATOM_BYTES : p.tiles * TILE_BYTES);
      for (int q = 0; q < p.tiles; ++q)
        for (int a = 0; a < (DIFF ? 1 : ATOMS); ++a) {
          if constexpr (DIFF != 0) {
            tma_load_4d(smem + SMEM_Q + q * TILE_BYTES, &tmap_q, &bars->q_full, 0, 2 * head + q, tok0 + q_base, batch);
            continue;
          }
          const bool second = LAT && a >= p.first_atoms;
          tma_load_4d(smem + SMEM_Q + q * TILE_BYTES + a * ATOM_BYTES, second ? &tmap_q2 : &tmap_q, &bars->q_full,
                      (second ? a - p.first_atoms : a) * 64, head, tok0 + q_base + q * BM, batch);
        }
      bool ok = true;
      int issued_k = 0, issued_v = 0;
      // paged: a tile is BN / block_size pages, each a box of block_size rows that lands at its place in the swizzled
      // tile (a page is a whole number of 8-row swizzle groups); tiles past the last page repeat it, masked below
      const int* pages = paged ? p.block_table + (long long)blockIdx.z * p.max_blocks : nullptr;
      const int per_tile = paged ? BN / p.block_size : 1, last_page = paged ? (kv_len - 1) / p.block_size : 0;
      const uint32_t page_bytes = paged ? (uint32_t)p.block_size * 128u : 0u;
      auto load_tile = [&](uint32_t dst_off, const CUtensorMap* map, uint64_t* bar, int jrel, int atoms, bool is_k) {
        const int j = jrel + j0;
        const int atom_cols = DIFF && is_k ? p.diff.dim : 64;        // DIFF: each map's keys start an atom
        if (!paged) {
          for (int a = 0; a < atoms; ++a) {
            if (LAT && is_k && a >= p.first_atoms)
              tma_load_4d(smem + dst_off + a * ATOM_BYTES, &tmap_k2, bar, (a - p.first_atoms) * 64, 0, key0_row + j * BN, batch);
            else
              tma_load_4d(smem + dst_off + a * ATOM_BYTES, map, bar, a * atom_cols, is_k ? kv_head : v_head, key0_row + j * BN, batch);
          }
          return;
        }
        for (int g = 0; g < per_tile; ++g) {
          const int page = pages[min(j * per_tile + g, last_page)];
          for (int a = 0; a < atoms; ++a)
            tma_load_4d(smem + dst_off + a * ATOM_BYTES + g * page_bytes, map, bar, a * atom_cols, 0, is_k ? kv_head : v_head, page);
        }
      };
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int s = j % K_STAGES, sv = j % V_STAGES;
        ok = mbar_wait(&bars->k_empty[s], ((j / K_STAGES) & 1) ^ 1, abort_flag, 10);
        if (!ok) break;
        mbar_arrive_expect_tx(&bars->k_full[s], TILE_BYTES);
        load_tile(SMEM_K + s * TILE_BYTES, &tmap_k, &bars->k_full[s], j, ATOMS, true);
        issued_k = j + 1;
        ok = mbar_wait(&bars->v_empty[sv], ((j / V_STAGES) & 1) ^ 1, abort_flag, 11);
        if (!ok) break;
        mbar_arrive_expect_tx(&bars->v_full[sv], V_TILE_BYTES);
        load_tile(SMEM_V + sv * V_TILE_BYTES, &tmap_v, &bars->v_full[sv], j, V_ATOMS, false);
        issued_v = j + 1;
      }
      if (!ok) {
        // drain: every copy this thread started must land before the CTA's shared memory is released
        volatile int never = 0;
        mbar_wait(&bars->q_full, 0, &never, 12);
        for (int j = max(0, issued_k - K_STAGES); j < issued_k; ++j)
          mbar_wait(&bars->k_full[j % K_STAGES], (j / K_STAGES) & 1, &never, 13);
        for (int j = max(0, issued_v - V_STAGES); j < issued_v; ++j)
          mbar_wait(&bars->v_full[j % V_STAGES], (j / V_STAGES) & 1, &never, 14);
      }
    }
  } else if (warp == 9) {
    // ------------------------------------------------------------------ MMA issuer
    if (lane == 0) {
      constexpr uint32_t IDESC_QK = umma_idesc_bf16_f32(BM, BN);
      constexpr uint32_t IDESC_PV = umma_idesc_bf16_f32(BM, VD) | (1u << 16);   // B is MN-major
      const uint32_t col_s[2] = {COL_S0, COL_S1}, col_o[2] = {COL_O0, COL_O1};
      const uint32_t q_addr = smem_u32(smem + SMEM_Q), k_addr = smem_u32(smem + SMEM_K),
                     v_addr = smem_u32(smem + SMEM_V);
      auto issue_qk = [&](int q, int s) {
        if constexpr (DIFF != 0) {
          for (int k = 0; k < (p.diff.dim + 15) / 16; ++k)
            umma_f16_ss(tmem + col_s[q], umma_desc_kmajor_sw128(q_addr + q * TILE_BYTES + k * 32),
                        umma_desc_kmajor_sw128(k_addr + s * TILE_BYTES + q * ATOM_BYTES + k * 32), IDESC_QK, k > 0);
          umma_commit(&bars->s_full[q]);
          return;
        }
#pragma unroll
        for (int k = 0; k < QK / 16; ++k) {
          const uint32_t off = (k >> 2) * ATOM_BYTES + (k & 3) * 32;
          umma_f16_ss(tmem + col_s[q], umma_desc_kmajor_sw128(q_addr + q * TILE_BYTES + off),
                      umma_desc_kmajor_sw128(k_addr + s * TILE_BYTES + off), IDESC_QK, k > 0);
        }
        umma_commit(&bars->s_full[q]);
      };
      bool ok = mbar_wait(&bars->q_full, 0, abort_flag, 20);
      if (ok) ok = mbar_wait(&bars->k_full[0], 0, abort_flag, 21);
      if (ok) {
        tc_fence_after_sync();
        issue_qk(0, 0);
        if (p.tiles == 2) issue_qk(1, 0);
        umma_commit(&bars->k_empty[0]);
      }
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int s = j % V_STAGES, sn = (j + 1) % K_STAGES;
        const uint32_t ph = (j / V_STAGES) & 1, phn = ((j + 1) / K_STAGES) & 1;
        ok = mbar_wait(&bars->v_full[s], ph, abort_flag, 22);
        if (ok && j + 1 < n_tiles) ok = mbar_wait(&bars->k_full[sn], phn, abort_flag, 23);
        for (int q = 0; q < p.tiles && ok; ++q) {
          ok = mbar_wait(&bars->p_full[q], j & 1, abort_flag, 24 + q);
          if (!ok) break;
          tc_fence_after_sync();
#pragma unroll
          for (int k = 0; k < BN / 16; ++k)
            umma_f16_ts(tmem + col_o[q], tmem + col_s[q] + k * 8,
                        umma_desc_mnmajor_sw128(v_addr + s * V_TILE_BYTES + k * 2048), IDESC_PV, (j > 0) || (k > 0));
          const bool last_q = (q == p.tiles - 1);
          if (last_q) umma_commit(&bars->v_empty[s]);
          if (j + 1 < n_tiles) {
            issue_qk(q, sn);
            if (last_q) umma_commit(&bars->k_empty[sn]);
          }
        }
      }
      umma_commit(&bars->o_final);   // also on the abort path: it only tracks MMAs already issued
      if (!ok) {                     // TMEM must not be freed under MMAs that are still running
        volatile int never = 0;
        mbar_wait(&bars->o_final, 0, &never, 27);
      }
    }
  } else {
    // ------------------------------------------------------------------ softmax warpgroups (thread = query row)
    const int q = warp >> 2;
    const int my_tiles = (q < p.tiles) ? n_tiles : 0;   // the second warpgroup idles in one-tile mode
    const uint32_t lane_base = (uint32_t)((warp & 3) * 32) << 16;
    const uint32_t t_s = tmem + lane_base + (q ? COL_S1 : COL_S0);
    const uint32_t t_o = tmem + lane_base + (q ? COL_O1 : COL_O0);
    const int row = q_base + q * TILE_STEP + (warp & 3) * 32 + lane;
    const float cap = DIFF ? p.diff.cap : 0.f;
    float to_cap = 0.f;             // 2 log2(e) scale / cap: the capped score is cap (1 - 2 / (2^(to_cap s) + 1))
    float scale_log2 = p.scale_log2;
    if constexpr (DIFF != 0) {
      if (p.diff.q_temp && row < q_len) scale_log2 *= p.diff.q_temp[row + coff];
      if (cap > 0.f) to_cap = 2.f * scale_log2 / cap, scale_log2 = 1.4426950408889634f;
    }
    float m_used = -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = 0; j < my_tiles; ++j) {
      ok = mbar_wait(&bars->s_full[q], j & 1, abort_flag, 30 + q);
      if (!ok) break;
      tc_fence_after_sync();
      uint32_t s[BN];
#pragma unroll
      for (int c = 0; c < BN / 32; ++c) tmem_ld_x32(t_s + c * 32, s + c * 32);
      tmem_ld_wait();
      if constexpr (DIFF == 2) {
        const int key0 = (j + j0) * BN, last = q_base + BM - 1 + coff;
        const float to_x = 0.34657359f * to_cap, k = 1.4426950408889634f * cap;       // x = score / cap; exponents in log2 units
        float far0 = 0.f, far1 = 0.f;
#pragma unroll
        for (int i = 0; i < BN; i += 2) {
          const float x0 = __uint_as_float(s[i]) * to_x, x1 = __uint_as_float(s[i + 1]) * to_x;
          far0 = fmaxf(far0, fabsf(x0)), far1 = fmaxf(far1, fabsf(x1));
          s[i] = __float_as_uint(x0), s[i + 1] = __float_as_uint(x1);
        }
        const bool edge = key0 + BN > min(kv_len, q_base + 1 + coff) || key0 < first_key_of(last);     // some pair is masked
        float l0 = 0.f, l1 = 0.f;
        if (!edge && __all_sync(0xffffffffu, fmaxf(far0, far1) <= 1.f)) {
          auto weight = [&](uint32_t u) {
            const float x = __uint_as_float(u), t = x * x;
            float r = fmaf(t, k * TANH_5, k * TANH_4);
            r = fmaf(t, r, k * TANH_3);
            r = fmaf(t, r, k * TANH_2);
            r = fmaf(t, r, k * TANH_1);
            r = fmaf(t, r, k * TANH_0);
            return ex2(x * r);
          };
#pragma unroll
          for (int i = 0; i < BN; i += 2) {
            const float e0 = weight(s[i]), e1 = weight(s[i + 1]);
            l0 += e0;
            l1 += e1;
            s[i >> 1] = pack_bf16x2(e0, e1);
          }
        } else {
          const int last_rel = min(kv_len - 1, row + coff) - key0, first_rel = first_key_of(row + coff) - key0;
          auto weight = [&](uint32_t u, int i) {
            const float y = ex2(__uint_as_float(u) * 2.8853900818f) + 1.f;
            return i > last_rel || i < first_rel ? 0.f : ex2(fmaf(-2.f * k, rcp_approx(y), k));
          };
#pragma unroll
          for (int i = 0; i < BN; i += 2) {
            const float e0 = weight(s[i], i), e1 = weight(s[i + 1], i + 1);
            l0 += e0;
            l1 += e1;
            s[i >> 1] = pack_bf16x2(e0, e1);
          }
        }
        l += l0 + l1;
        tmem_st_x32(t_s, s);
        tmem_st_x32(t_s + 32, s + 32);
        tmem_st_wait();
        tc_fence_before_sync();
        mbar_arrive(&bars->p_full[q]);
        continue;
      }
      if (DIFF && cap > 0.f) {
#pragma unroll
        for (int i = 0; i < BN; ++i)
          s[i] = __float_as_uint(fmaf(-2.f * cap, rcp_approx(ex2(__uint_as_float(s[i]) * to_cap) + 1.f), cap));
      }
      // keys past the sequence (zero fill, or the next sequence of a packed batch) and, when causal, keys after the
      // query position never contribute
      const int key0 = (j + j0) * BN;
      if (key0 + BN > kv_len || (p.causal && key0 + BN > q_base + q * TILE_STEP + coff)) {
        const int last_key = p.causal ? min(kv_len - 1, row + coff) : kv_len - 1;
#pragma unroll
        for (int i = 0; i < BN; ++i)
          if (key0 + i > last_key) s[i] = __float_as_uint(-INFINITY);
      }
      if constexpr (EXT) {   // keys in front of the chunk or window; only tiles below the last row's first key can hold any
        if (key0 < first_key_of(q_base + q * TILE_STEP + BM - 1 + coff)) {
          const int first_key = first_key_of(row + coff);
#pragma unroll
          for (int i = 0; i < BN; ++i)
            if (key0 + i < first_key) s[i] = __float_as_uint(-INFINITY);
        }
      }
      float mx0 = -INFINITY, mx1 = -INFINITY, mx2 = -INFINITY, mx3 = -INFINITY;
#pragma unroll
      for (int i = 0; i < BN; i += 4) {
        mx0 = fmaxf(mx0, __uint_as_float(s[i]));
        mx1 = fmaxf(mx1, __uint_as_float(s[i + 1]));
        mx2 = fmaxf(mx2, __uint_as_float(s[i + 2]));
        mx3 = fmaxf(mx3, __uint_as_float(s[i + 3]));
      }
      const float m_new = fmaxf(fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3)), m_used);
      const bool grow = (m_new - m_used) * scale_log2 > RESCALE_THRESHOLD;   // true on the first tile (m_used = -inf)
      if (__any_sync(0xffffffffu, grow)) {
        const float f = grow ? ex2((m_used - m_new) * scale_log2) : 1.f;      // -inf -> 0 on the first tile
        if (grow) {
          l *= f;
          m_used = m_new;
        }
        if (j > 0) {   // O holds nothing before the first PV
#pragma unroll
          for (int c = 0; c < VD / 32; ++c) {
            uint32_t o[32];
            tmem_ld_x32(t_o + c * 32, o);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * f);
            tmem_st_x32(t_o + c * 32, o);
          }
        }
      }
      // a row whose chunk starts beyond this tile has seen no key yet: its exponentials are all zero
      const float neg_m = (EXT && m_used == -INFINITY) ? 0.f : -m_used * scale_log2;
      float l0 = 0.f, l1 = 0.f;
      // (Measured alternatives for this loop, all slower on B200: every 4th / 2nd exponential as a cubic on the FMA pipe
      // -8 % / -17 %; pairs of exponentials as one bf16x2 special-function operation -6 %; three-input max with
      // two-lane fp32 multiply-add and add -30 %, from register-pair moves and spills. The loop is issue-bound.)
#pragma unroll
      for (int i = 0; i < BN; i += 2) {   // packed P overwrites the row in place (index i/2 <= i)
        const float e0 = ex2(fmaf(__uint_as_float(s[i]), scale_log2, neg_m));
        const float e1 = ex2(fmaf(__uint_as_float(s[i + 1]), scale_log2, neg_m));
        l0 += e0;
        l1 += e1;
        s[i >> 1] = pack_bf16x2(e0, e1);
      }
      l += l0 + l1;
      tmem_st_x32(t_s, s);
      tmem_st_x32(t_s + 32, s + 32);
      tmem_st_wait();
      tc_fence_before_sync();
      mbar_arrive(&bars->p_full[q]);
    }
    if (ok && my_tiles > 0) ok = mbar_wait(&bars->o_final, 0, abort_flag, 32 + q);
    if constexpr (DIFF != 0) ok = __all_sync(0xffffffffu, ok);      // the barrier below is taken warp by warp
    if (ok && my_tiles > 0) {
      tc_fence_after_sync();
      float inv = l > 0.f ? 1.f / l : 0.f;
      if constexpr (EXT) {
        if (p.sink) {   // join the sink in a frame whose largest exponent is zero
          const float sk = p.sink[head] * 1.4426950408889634f, mm = m_used * scale_log2;
          const float top = fmaxf(sk, mm), e = ex2(mm - top);
          inv = e / (l * e + ex2(sk - top));
        }
      }
      if constexpr (LAT) {
        if (p.gate && row < q_len) {
          const float z = __bfloat162float(p.gate[(long long)(tok0 + row) * p.gate_stride + head]);
          inv *= 1.f / (1.f + ex2(-1.4426950408889634f * z));
        }
      }
      // Stage this warp's 32 rows x VD columns in the (now idle) Q region, then write every row's VD * 2 bytes with
      // VD / 8 lanes x 16 bytes: contiguous runs for local stores and for stores that cross NVLink alike.
      // 16-byte chunk c of row r sits at c ^ (r & 7).
      uint8_t* slab = smem + SMEM_Q + warp * (32 * ROW_BYTES);
      if constexpr (DIFF != 0) {
        // fp32 hand-over in the (idle) K region, row r of VD numbers, 16-byte chunk c at c ^ (r & 31 within the row's chunks)
        float4* hand = reinterpret_cast<float4*>(smem + SMEM_K) + (size_t)((warp & 3) * 32 + lane) * (VD / 4);
        const float f = q ? inv * p.diff.share : inv;
        float ss = 0.f;
        if (q == 0) asm volatile("bar.sync 1, 256;" ::: "memory");
#pragma unroll
        for (int c = 0; c < VD / 32; ++c) {
          uint32_t o[32];
          tmem_ld_x32(t_o + c * 32, o);
          tmem_ld_wait();
#pragma unroll
          for (int v = 0; v < 8; ++v) {
            float4* at = hand + ((c * 8 + v) ^ (lane & (VD / 4 - 1)));
            float4 x = make_float4(__uint_as_float(o[v * 4]) * f, __uint_as_float(o[v * 4 + 1]) * f, __uint_as_float(o[v * 4 + 2]) * f,
                                   __uint_as_float(o[v * 4 + 3]) * f);
            if (q == 0) {
              const float4 y = *at;
              x.x -= y.x, x.y -= y.y, x.z -= y.z, x.w -= y.w;
              ss += (x.x * x.x + x.y * x.y) + (x.z * x.z + x.w * x.w);      // columns past v_dim are zero in both maps
            }
            *at = x;
          }
        }
        if (q == 0) {
          const float r = rsqrtf(ss / (float)p.diff.n + p.diff.eps) * p.diff.post;
#pragma unroll
          for (int c = 0; c < VD / 8; ++c) {
            const float4 x = hand[(2 * c) ^ (lane & (VD / 4 - 1))], y = hand[(2 * c + 1) ^ (lane & (VD / 4 - 1))];
            uint4 u;
            u.x = pack_bf16x2(x.x * r, x.y * r), u.y = pack_bf16x2(x.z * r, x.w * r);
            u.z = pack_bf16x2(y.x * r, y.y * r), u.w = pack_bf16x2(y.z * r, y.w * r);
            *reinterpret_cast<uint4*>(slab + lane * ROW_BYTES + ((c ^ (lane & 7)) << 4)) = u;
          }
        }
      }
#pragma unroll
      for (int c = 0; c < (DIFF ? 0 : VD / 32); ++c) {
        uint32_t o[32];
        tmem_ld_x32(t_o + c * 32, o);
        tmem_ld_wait();
#pragma unroll
        for (int v = 0; v < 4; ++v) {
          uint4 u;
          u.x = pack_bf16x2(__uint_as_float(o[v * 8 + 0]) * inv, __uint_as_float(o[v * 8 + 1]) * inv);
          u.y = pack_bf16x2(__uint_as_float(o[v * 8 + 2]) * inv, __uint_as_float(o[v * 8 + 3]) * inv);
          u.z = pack_bf16x2(__uint_as_float(o[v * 8 + 4]) * inv, __uint_as_float(o[v * 8 + 5]) * inv);
          u.w = pack_bf16x2(__uint_as_float(o[v * 8 + 6]) * inv, __uint_as_float(o[v * 8 + 7]) * inv);
          *reinterpret_cast<uint4*>(slab + lane * ROW_BYTES + (((c * 4 + v) ^ (lane & 7)) << 4)) = u;
        }
      }
      __syncwarp();
      const int row0 = q_base + q * TILE_STEP + (warp & 3) * 32;
      constexpr int AHEAD = 8;                                           // gates requested together
      uint4 gates[AHEAD];
#pragma unroll 8
      for (int it = 0; it < (DIFF && q ? 0 : CHUNKS); ++it) {            // CHUNKS lanes write one row: 32 / CHUNKS rows per pass
        const int r = (32 / CHUNKS) * it + lane / CHUNKS, ch = lane % CHUNKS;
        const int grow = row0 + r;
        if constexpr (WIDE) {
          if (p.out_gate && it % AHEAD == 0) {
#pragma unroll
            for (int a = 0; a < AHEAD; ++a) {
              const int g2 = min(grow + (32 / CHUNKS) * a, q_len - 1);
              gates[a] = __ldg(reinterpret_cast<const uint4*>(p.out_gate + (tok0 + g2) * p.out_gate_stride + (long long)blockIdx.y * p.v_dim +
                                                              min(ch * 8, p.v_dim - 8)));
            }
          }
        }
        if (grow < q_len) {
          uint4 val = *reinterpret_cast<const uint4*>(slab + r * ROW_BYTES + ((ch ^ (r & 7)) << 4));
          if (EXT && ch * 8 >= p.v_dim) continue;
          const long long col = (long long)(WIDE ? blockIdx.y : head) * (EXT ? p.v_dim : VD);
          if constexpr (WIDE) {
            if (p.out_gate) {
              float x[8], z[8];
              load_row8(reinterpret_cast<const bf16*>(&val), x);
              load_row8(reinterpret_cast<const bf16*>(&gates[it % AHEAD]), z);
#pragma unroll
              for (int i = 0; i < 8; ++i) x[i] *= rcp_approx(1.f + ex2(-1.4426950408889634f * z[i]));
              store_row8(reinterpret_cast<bf16*>(&val), x);
            }
          }
          bf16* dst = p.out + ((long long)batch * p.q_len + tok0 + grow) * p.out_stride_tok + col;
          if (p.scatter.enabled) {
            const OutScatter& sc = p.scatter;
            const int g2 = grow - sc.split;
            const int rk = grow < sc.split ? grow / sc.n0 : g2 / sc.n1;
            const int local = grow < sc.split ? grow % sc.n0 : sc.n0 + g2 % sc.n1;
            dst = sc.peer[rk] + (long long)local * p.out_stride_tok + sc.col_offset + head * VD;
          }
          *reinterpret_cast<uint4*>(dst + ch * 8) = val;
        }
      }
    }
    if constexpr (DIFF != 0) {          // the hand-over barrier takes all 256 threads, whatever became of the waits
      if (q == 1 || !ok) asm volatile("bar.sync 1, 256;" ::: "memory");
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 9) {
    tc_fence_after_sync();
    tmem_dealloc(tmem, TMEM_COLS);
  }
}

// ---------------------------------------------------------------------------------------------
// host side
// ---------------------------------------------------------------------------------------------
struct Map4Key {
  const void* ptr;
  long long s1, s2, s3;
  int d1, d2, d3;
  bool operator==(const Map4Key& o) const {
    return ptr == o.ptr && s1 == o.s1 && s2 == o.s2 && s3 == o.s3 && d1 == o.d1 && d2 == o.d2 && d3 == o.d3;
  }
};
struct Map4Hash {
  size_t operator()(const Map4Key& k) const {
    size_t h = reinterpret_cast<size_t>(k.ptr);
    for (long long v : {k.s1, k.s2, k.s3, (long long)k.d1, (long long)k.d2, (long long)k.d3}) h = h * 1000003u ^ (size_t)v;
    return h;
  }
};

// bf16 [batch, tokens, heads, 128] with element strides (tok, head, batch): dims (128, heads, tokens, batch),
// box (64, 1, 128, 1), 128-byte swizzle, zero fill outside.
// With page_rows > 0 the tensor is a page pool [batch = pages, heads, page_rows, 128] (contiguous): dims
// (128, page_rows, heads, pages), box (64, page_rows, 1, 1); `tokens` and the strides are then unused.
int make_tmap_heads(CUtensorMap* out, const void* ptr, int hd, int heads, int tokens, int batch, long long stride_head,
                    long long stride_tok, long long stride_batch, int page_rows = 0) {
  static std::mutex mu;
  static std::unordered_map<Map4Key, CUtensorMap, Map4Hash> cache;
  if (page_rows > 0) {
    tokens = -page_rows;
    stride_head = (long long)page_rows * hd;
    stride_tok = hd;
    stride_batch = (long long)heads * page_rows * hd;
  }
  Map4Key key{ptr, stride_head, stride_tok, stride_batch, heads * 1024 + hd, tokens, batch};
  {
    std::lock_guard<std::mutex> g(mu);
    auto it = cache.find(key);
    if (it != cache.end()) {
      *out = it->second;
      return 0;
    }
  }
  static PFN_cuTensorMapEncodeTiled_v12000 encode = nullptr;
  if (!encode) {
    void* fn = nullptr;
    cudaDriverEntryPointQueryResult qres;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &qres) != cudaSuccess ||
        qres != cudaDriverEntryPointSuccess)
      return -1;
    encode = reinterpret_cast<PFN_cuTensorMapEncodeTiled_v12000>(fn);
  }
  cuuint64_t dims[4] = {(cuuint64_t)hd, (cuuint64_t)heads, (cuuint64_t)tokens, (cuuint64_t)batch};
  cuuint64_t strides[3] = {(cuuint64_t)stride_head * 2, (cuuint64_t)stride_tok * 2, (cuuint64_t)stride_batch * 2};
  cuuint32_t box[4] = {64u, 1u, (cuuint32_t)BM, 1u};
  if (page_rows > 0) {
    dims[1] = (cuuint64_t)page_rows;
    dims[2] = (cuuint64_t)heads;
    strides[0] = (cuuint64_t)stride_tok * 2;
    strides[1] = (cuuint64_t)stride_head * 2;
    box[1] = (cuuint32_t)page_rows;
    box[2] = 1u;
  }
  cuuint32_t estr[4] = {1u, 1u, 1u, 1u};
  CUresult r = encode(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, const_cast<void*>(ptr), dims, strides, box, estr,
                      CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                      CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) return -(int)r - 1000;
  std::lock_guard<std::mutex> g(mu);
  if (cache.size() > 4096) cache.clear();
  cache.emplace(key, *out);
  return 0;
}

}  // namespace

int g_force_tiles = 0;   // 0: choose per problem; 1 / 2: fixed query tiles per CTA (comparison runs)
void attn_dense_tcgen05_set_tiles(int tiles) { g_force_tiles = tiles; }

namespace {

struct FaMaps {
  CUtensorMap q, k, v, q2, k2;     // q2 / k2: second parts of latent attention
};

template <int QK, int VD, bool EXT, bool LAT, int DIFF = 0>
int launch_fa(dim3 grid, cudaStream_t stream, const FaMaps& m, const FaParams& p) {
  static bool configured[64] = {false};
  auto kernel = attn_dense_tcgen05_kernel<QK, VD, EXT, LAT, DIFF>;
  constexpr size_t SMEM = FaCfg<QK, VD>::SMEM_BYTES;
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !configured[dev]) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM);
    if (e != cudaSuccess) return -(int)e;
    configured[dev] = true;
  }
  return launch_kernel(kernel, grid, dim3(THREADS), SMEM, stream, m.q, m.k, m.v, m.q2, m.k2, p);
}

enum class FaKind { DENSE, EXT, LATENT, DIFF };

// qk: tile width of q and k
int launch_tiles(int qk, FaKind kind, int q_len, int Hq, int batch, cudaStream_t stream, const FaMaps& m, FaParams& p) {
  // one-tile CTAs when that shortens the schedule: a one-tile CTA takes ~0.85 of a two-tile CTA's time (measured)
  if (kind == FaKind::DIFF) {
    p.tiles = 2;
    const dim3 rows((q_len + BM - 1) / BM, Hq, batch);
    return p.diff.cap > 0.f && p.diff.cap <= MAX_FIXED_CAP ? launch_fa<128, 128, true, false, 2>(rows, stream, m, p)
                                                           : launch_fa<128, 128, true, false, 1>(rows, stream, m, p);
  }
  const int sms = 148;
  const long c2 = (long)((q_len + 2 * BM - 1) / (2 * BM)) * Hq * batch, c1 = (long)((q_len + BM - 1) / BM) * Hq * batch;
  const double t2 = (double)((c2 + sms - 1) / sms), t1 = 0.85 * (double)((c1 + sms - 1) / sms);
  p.tiles = (g_force_tiles == 1 || g_force_tiles == 2) ? g_force_tiles : (t1 < t2 ? 1 : 2);
  const dim3 grid((q_len + p.tiles * BM - 1) / (p.tiles * BM), Hq, batch);
  if (kind == FaKind::LATENT)
    return qk == 192 ? launch_fa<192, 128, true, true>(grid, stream, m, p) : launch_fa<128, 128, true, true>(grid, stream, m, p);
  if (kind == FaKind::EXT) {
    if (qk == 64 && p.v_dim > 64) return launch_fa<64, 128, true, false>(grid, stream, m, p);
    return qk == 64 ? launch_fa<64, 64, true, false>(grid, stream, m, p) : launch_fa<128, 128, true, false>(grid, stream, m, p);
  }
  return qk == 64 ? launch_fa<64, 64, false, false>(grid, stream, m, p) : launch_fa<128, 128, false, false>(grid, stream, m, p);
}

}  // namespace

// Returns 1 when the tcgen05 kernel handles this problem, 0 otherwise.
int attn_dense_tcgen05_supported(const void* q, const void* k, const void* v, long long q_stride_tok, int q_stride_head,
                                 long long kv_stride_tok, int kv_stride_head, long long out_stride_tok, int D,
                                 int causal) {
  if (D != 128 && D != 64) return 0;
  (void)causal;   // causal problems are supported when queries and keys cover the same positions (checked by callers)
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) & 15) return 0;
  if ((q_stride_tok | q_stride_head | kv_stride_tok | kv_stride_head | out_stride_tok) % 8) return 0;
  return 1;
}

int attn_dense_tcgen05_launch(const void* q, long long q_stride_tok, int q_stride_head, const void* k, const void* v,
                              long long kv_stride_tok, int kv_stride_head, void* out, long long out_stride_tok,
                              int batch, int q_len, int kv_len, int Hq, int Hkv, float scale, cudaStream_t stream,
                              void* const* peers, int world, int split, int n0, int n1, int col_offset, int causal,
                              const int* cu_q, int total_tokens, int head_dim, const int* kv_lens,
                              const int* block_table, int max_blocks, int block_size, int num_blocks) {
  if (head_dim != 64 && head_dim != 128) return -3;
  const bool paged = block_table != nullptr;
  if (paged && (head_dim != 128 || !cu_q || !kv_lens || block_size < 8 || block_size % 8 || BN % block_size ||
                num_blocks <= 0 || max_blocks <= 0 || peers))
    return -3;
  FaMaps m{};
  // packed batches address one flat token axis (batch = the number of sequences only sizes the grid)
  const int map_q_tokens = cu_q ? total_tokens : q_len, map_kv_tokens = cu_q ? total_tokens : kv_len;
  const int map_batch = cu_q ? 1 : batch;
  int rc = make_tmap_heads(&m.q, q, head_dim, Hq, map_q_tokens, map_batch, q_stride_head, q_stride_tok, q_stride_tok * map_q_tokens);
  if (rc) return rc;
  rc = make_tmap_heads(&m.k, k, head_dim, Hkv, map_kv_tokens, paged ? num_blocks : map_batch, kv_stride_head,
                       kv_stride_tok, kv_stride_tok * map_kv_tokens, paged ? block_size : 0);
  if (rc) return rc;
  rc = make_tmap_heads(&m.v, v, head_dim, Hkv, map_kv_tokens, paged ? num_blocks : map_batch, kv_stride_head,
                       kv_stride_tok, kv_stride_tok * map_kv_tokens, paged ? block_size : 0);
  if (rc) return rc;
  FaParams p{};
  p.out = reinterpret_cast<bf16*>(out);
  p.out_stride_tok = out_stride_tok;
  p.q_len = q_len;
  p.kv_len = kv_len;
  p.Hq = Hq;
  p.Hkv = Hkv;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.causal = causal;
  p.cu_q = cu_q;
  p.kv_lens = kv_lens;
  p.block_table = block_table;
  p.max_blocks = max_blocks;
  p.block_size = block_size;
  if (cu_q) p.q_len = 0;   // rows are addressed by their flat token index
  if (peers) {
    if (world < 1 || world > 8 || batch != 1 || n1 <= 0 || (split > 0 && n0 <= 0) || (col_offset % 8) != 0) return -3;
    for (int r = 0; r < world; ++r) p.scatter.peer[r] = reinterpret_cast<bf16*>(peers[r]);
    p.scatter.enabled = 1;
    p.scatter.split = split;
    p.scatter.n0 = n0 > 0 ? n0 : 1;
    p.scatter.n1 = n1;
    p.scatter.col_offset = col_offset;
  }
  return launch_tiles(head_dim, FaKind::DENSE, q_len, Hq, batch, stream, m, p);
}

// Attention over queries and keys of any head widths up to 128 (multiples of 8), with chunked masking and sinks: the
// packed fresh-prefill form (k / v strided rows of one flat token axis) or, with block_table, the paged form (caches
// [num_blocks, Hkv, block_size, D] and [num_blocks, Hkv, block_size, Dv]). Causal; sequences from cu_q.
int attn_ext_tcgen05_launch(const void* q, long long q_stride_tok, const void* k, long long k_stride_tok, const void* v,
                            long long v_stride_tok, void* out, long long out_stride_tok, int num_seqs, int max_q_len,
                            int total_tokens, int Hq, int Hkv, int D, int Dv, float scale, int chunk, const float* sink,
                            const int* cu_q, const int* kv_lens, const int* block_table, int max_blocks, int block_size,
                            int num_blocks, cudaStream_t stream, int window, const attn::DiffAttn* diff, int v_heads, const void* gate,
                            long long gate_stride) {
  const bool paged = block_table != nullptr;
  if (window < 0 || (diff && (sink || chunk || D % 16))) return -3;
  if (D < 8 || Dv < 8 || D > 128 || Dv > 128 || (D % 8) || (Dv % 8) || !cu_q || Hq % Hkv || !(scale > 0.f) || chunk < 0) return -3;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v) |
       reinterpret_cast<uintptr_t>(out)) & 15)
    return -3;
  if ((q_stride_tok | out_stride_tok) % 8) return -3;
  if (paged ? (!kv_lens || block_size < 8 || block_size % 8 || BN % block_size || num_blocks <= 0 || max_blocks <= 0)
            : ((k_stride_tok | v_stride_tok) % 8 != 0))
    return -3;
  FaMaps m{};
  int rc = diff ? make_tmap_heads(&m.q, q, D / 2, 2 * Hq, total_tokens, 1, D / 2, q_stride_tok, q_stride_tok * total_tokens)
                : make_tmap_heads(&m.q, q, D, Hq, total_tokens, 1, D, q_stride_tok, q_stride_tok * total_tokens);
  if (rc) return rc;
  rc = make_tmap_heads(&m.k, k, D, Hkv, total_tokens, paged ? num_blocks : 1, D, k_stride_tok, k_stride_tok * total_tokens,
                       paged ? block_size : 0);
  if (rc) return rc;
  rc = make_tmap_heads(&m.v, v, Dv, v_heads > 0 ? v_heads : Hkv, total_tokens, paged ? num_blocks : 1, Dv, v_stride_tok, v_stride_tok * total_tokens,
                       paged ? block_size : 0);
  if (rc) return rc;
  FaParams p{};
  p.out = reinterpret_cast<bf16*>(out);
  p.out_stride_tok = out_stride_tok;
  p.Hq = Hq;
  p.Hkv = Hkv;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.causal = 1;
  p.cu_q = cu_q;
  p.kv_lens = kv_lens;
  p.block_table = block_table;
  p.max_blocks = max_blocks;
  p.block_size = block_size;
  p.chunk = chunk;
  p.sink = sink;
  p.window = window;
  p.v_dim = Dv;
  p.v_heads = v_heads;
  p.out_gate = reinterpret_cast<const bf16*>(gate);
  p.out_gate_stride = gate_stride;
  if (diff) {
    p.diff = *diff;
    return launch_tiles(128, FaKind::DIFF, max_q_len, Hq, num_seqs, stream, m, p);
  }
  return launch_tiles(D > 64 ? 128 : 64, FaKind::EXT, max_q_len, Hq * (v_heads > 0 ? v_heads : 1), num_seqs, stream, m, p);
}

// Latent attention on expanded keys and values, causal: q [total_tokens] rows of H heads of [d1 | d2] (stride q_stride_tok), k
// and v rows of one flat axis of key_rows rows (heads of d1 and Dv columns), k2 [key_rows] rows of d2 columns shared by the
// heads. cu_k [num_seqs + 1]: each sequence's key rows, ending with those of its queries (null: the queries' own rows). seqs:
// the sequences of this launch (null: all). gate: logits [total_tokens, >= H] or null.
int attn_latent_tcgen05_launch(const void* q, long long q_stride_tok, const void* k, const void* v, long long kv_stride_tok,
                               const void* k2, long long k2_stride_tok, int key_rows, void* out, long long out_stride_tok,
                               int num_seqs, int max_q_len, int total_tokens, int H, int d1, int d2, int Dv, float scale,
                               const float* sink, const void* gate, long long gate_stride, const int* cu_q, const int* seqs,
                               const int* cu_k, cudaStream_t stream, int window) {
  if (window < 0) return -3;
  if (d1 < 8 || d2 < 8 || Dv < 8 || d1 > 128 || d2 > 64 || Dv > 128 || ((d1 | d2 | Dv) % 8) || !cu_q || !(scale > 0.f)) return -3;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v) |
       reinterpret_cast<uintptr_t>(k2) | reinterpret_cast<uintptr_t>(out)) & 15)
    return -3;
  if ((q_stride_tok | kv_stride_tok | k2_stride_tok | out_stride_tok) % 8) return -3;
  FaMaps m{};
  const bf16* qb = reinterpret_cast<const bf16*>(q);
  int rc = make_tmap_heads(&m.q, qb, d1, H, total_tokens, 1, d1 + d2, q_stride_tok, q_stride_tok * total_tokens);
  if (!rc) rc = make_tmap_heads(&m.q2, qb + d1, d2, H, total_tokens, 1, d1 + d2, q_stride_tok, q_stride_tok * total_tokens);
  if (!rc) rc = make_tmap_heads(&m.k, k, d1, H, key_rows, 1, d1, kv_stride_tok, kv_stride_tok * key_rows);
  if (!rc) rc = make_tmap_heads(&m.k2, k2, d2, 1, key_rows, 1, d2, k2_stride_tok, k2_stride_tok * key_rows);
  if (!rc) rc = make_tmap_heads(&m.v, v, Dv, H, key_rows, 1, Dv, kv_stride_tok, kv_stride_tok * key_rows);
  if (rc) return rc;
  FaParams p{};
  p.out = reinterpret_cast<bf16*>(out);
  p.out_stride_tok = out_stride_tok;
  p.Hq = p.Hkv = H;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.causal = 1;
  p.cu_q = cu_q;
  p.sink = sink;
  p.window = window;
  p.v_dim = Dv;
  p.seqs = seqs;
  p.cu_k = cu_k;
  p.gate = reinterpret_cast<const bf16*>(gate);
  p.gate_stride = gate_stride;
  p.first_atoms = (d1 + 63) / 64;
  return launch_tiles(p.first_atoms == 1 ? 128 : 192, FaKind::LATENT, max_q_len, H, num_seqs, stream, m, p);
}

}  // namespace swb
