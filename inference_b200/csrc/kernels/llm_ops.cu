// Bandwidth-bound LLM glue kernels for sm_100a: fused residual-add + RMSNorm, fused QK-norm + RoPE +
// paged-KV write, gated-activation multiply, embedding gather, LayerNorm/adaLN modulation.
//
// They replace chains of small kernels in the reference: rms_norm (candle-llm/src/primitives/nn.rs:22-31,
// six launches), apply_rope + transpose + contiguous (models/llama.rs:1084-1090), KV concat-grow /
// scatter_set (primitives/kv_cache.rs:107-117, paged_kv_cache.rs:269-283), SwiGLU (models/llama.rs:1386-1391).
#include "common.cuh"

namespace swb {

SWB_REGISTER_STATUS_UNIT(llm_ops);
namespace {

__device__ __forceinline__ void unpack8(const uint4& u, float* f) {
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    float2 t = __bfloat1622float2(h[i]);
    f[2 * i] = t.x;
    f[2 * i + 1] = t.y;
  }
}
__device__ __forceinline__ uint4 pack8(const float* f) {
  uint4 u;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
  for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
  return u;
}

template <int THREADS>
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = (lane < THREADS / 32) ? red[lane] : 0.f;
  t = warp_sum(t);
  __syncthreads();
  return t;
}

// out = rmsnorm(x (+ residual)) * w ; when residual != nullptr it is updated in place to x + residual.
// One CTA per row; H % 8 == 0; the row is kept in registers between the two passes (H <= 8 * 8 * THREADS).
template <int THREADS, int VPT>
__global__ void __launch_bounds__(THREADS) rmsnorm_kernel(const bf16* __restrict__ x, int ldx, bf16* residual,
                                                         int ldr, const bf16* __restrict__ w, bf16* out, int ldo,
                                                         int H, float eps, float w_offset, const uint8_t* pf_ptr,
                                                         long long pf_bytes) {
  pdl_launch_dependents();
  pdl_wait(TL_RMSNORM);
  // The weights of the GEMM that consumes this norm do not depend on anything in flight: ask L2 for them now, so the
  // memory system works through the norm and the GEMM's prologue instead of idling (decode steps are bandwidth bound).
  if (pf_ptr) {
    constexpr long long CHUNK = 4096;
    const long long n_chunks = (pf_bytes + CHUNK - 1) / CHUNK;
    for (long long c = (long long)blockIdx.x * THREADS + threadIdx.x; c < n_chunks; c += (long long)gridDim.x * THREADS) {
      const long long off = c * CHUNK;
      const unsigned bytes = (unsigned)min(CHUNK, pf_bytes - off) & ~15u;
      if (bytes) asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(pf_ptr + off), "r"(bytes) : "memory");
    }
  }
  __shared__ float red[32];
  const int row = blockIdx.x;
  const int nvec = H / 8;
  float vals[VPT][8];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * THREADS;
    if (v < nvec) {
      uint4 u = *reinterpret_cast<const uint4*>(x + (size_t)row * ldx + v * 8);
      unpack8(u, vals[i]);
      if (residual) {
        uint4 r = *reinterpret_cast<const uint4*>(residual + (size_t)row * ldr + v * 8);
        float rf[8];
        unpack8(r, rf);
#pragma unroll
        for (int j = 0; j < 8; ++j) vals[i][j] += rf[j];
        uint4 s = pack8(vals[i]);
        *reinterpret_cast<uint4*>(residual + (size_t)row * ldr + v * 8) = s;
        unpack8(s, vals[i]);  // normalise exactly what was stored (bf16-rounded residual stream)
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += vals[i][j] * vals[i][j];
    }
  }
  ss = block_sum<THREADS>(ss, red);
  const float inv = rsqrtf(ss / (float)H + eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * THREADS;
    if (v < nvec) {
      uint4 wu = __ldg(reinterpret_cast<const uint4*>(w + v * 8));
      float wf[8], o[8];
      unpack8(wu, wf);
#pragma unroll
      for (int j = 0; j < 8; ++j) o[j] = vals[i][j] * inv * (wf[j] + w_offset);
      *reinterpret_cast<uint4*>(out + (size_t)row * ldo + v * 8) = pack8(o);
    }
  }
}

// LayerNorm without affine followed by adaLN modulation: out = LN(x) * (1 + scale) + shift, where
// scale/shift are per-batch vectors (row / rows_per_batch selects the batch).
template <int THREADS, int VPT>
__global__ void __launch_bounds__(THREADS) layernorm_mod_kernel(const bf16* __restrict__ x, int ldx,
                                                               const bf16* __restrict__ scale,
                                                               const bf16* __restrict__ shift, int ld_mod,
                                                               int rows_per_batch, const bf16* __restrict__ gamma,
                                                               const bf16* __restrict__ beta, bf16* out, int ldo, int H,
                                                               float eps) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[32];
  const int row = blockIdx.x;
  const int nvec = H / 8;
  float vals[VPT][8];
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * THREADS;
    if (v < nvec) {
      unpack8(*reinterpret_cast<const uint4*>(x + (size_t)row * ldx + v * 8), vals[i]);
#pragma unroll
      for (int j = 0; j < 8; ++j) s += vals[i][j];
    }
  }
  const float mean = block_sum<THREADS>(s, red) / (float)H;
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * THREADS;
    if (v < nvec) {
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float d = vals[i][j] - mean;
        ss += d * d;
      }
    }
  }
  const float inv = rsqrtf(block_sum<THREADS>(ss, red) / (float)H + eps);
  const int b = rows_per_batch > 0 ? row / rows_per_batch : 0;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * THREADS;
    if (v < nvec) {
      float o[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) o[j] = (vals[i][j] - mean) * inv;
      if (gamma) {
        float g[8];
        unpack8(__ldg(reinterpret_cast<const uint4*>(gamma + v * 8)), g);
#pragma unroll
        for (int j = 0; j < 8; ++j) o[j] *= g[j];
      }
      if (beta) {
        float g[8];
        unpack8(__ldg(reinterpret_cast<const uint4*>(beta + v * 8)), g);
#pragma unroll
        for (int j = 0; j < 8; ++j) o[j] += g[j];
      }
      if (scale) {
        float sc[8];
        unpack8(*reinterpret_cast<const uint4*>(scale + (size_t)b * ld_mod + v * 8), sc);
#pragma unroll
        for (int j = 0; j < 8; ++j) o[j] *= (1.f + sc[j]);
      }
      if (shift) {
        float sh[8];
        unpack8(*reinterpret_cast<const uint4*>(shift + (size_t)b * ld_mod + v * 8), sh);
#pragma unroll
        for (int j = 0; j < 8; ++j) o[j] += sh[j];
      }
      *reinterpret_cast<uint4*>(out + (size_t)row * ldo + v * 8) = pack8(o);
    }
  }
}

__device__ __forceinline__ float elem_to_f(bf16 x) { return __bfloat162float(x); }
__device__ __forceinline__ float elem_to_f(float x) { return x; }
__device__ __forceinline__ void elem_from_f(bf16& d, float x) { d = __float2bfloat16(x); }
__device__ __forceinline__ void elem_from_f(float& d, float x) { d = x; }

// Per (token, head) warp: optional per-head RMSNorm (q_norm / k_norm), rotary embedding from a
// precomputed fp32 cos/sin table [max_pos, rot_dim/2], then: q heads are written back in place, k and v
// heads are written into the paged cache (layout [block, kv_head, block_size, head_dim]) at slot_mapping[t].
// interleaved = 0: NeoX half-split pairs (i, i + rot_dim/2); 1: GPT-J pairs (2i, 2i+1).
// E is the element type of the projection buffer and the cache (bf16, or float for the 32-bit mode); EPL elements per
// lane bound the head width to 32 * EPL; v heads may have a width Dv of their own.
template <typename E, int EPL>
__global__ void __launch_bounds__(256) rope_kv_write_kernel(
    E* qkv, int ld_qkv, const int* __restrict__ positions, const long long* __restrict__ slot_mapping,
    const float* __restrict__ cos_tab, const float* __restrict__ sin_tab, int rot_dim, int interleaved,
    const bf16* __restrict__ q_norm_w, const bf16* __restrict__ k_norm_w, float norm_eps, float norm_w_offset,
    E* kcache, E* vcache, int block_size, int T, int Hq, int Hkv, int Dqk, int Dv) {
  pdl_launch_dependents();
  pdl_wait(TL_ROPE_KV);
  __shared__ float rope_smem[8 * 32 * EPL];
  const int warps_per_block = blockDim.x >> 5;
  const int lane = threadIdx.x & 31;
  const long long gw = (long long)blockIdx.x * warps_per_block + (threadIdx.x >> 5);
  const int heads = Hq + 2 * Hkv;
  if (gw >= (long long)T * heads) return;
  const int t = (int)(gw / heads);
  const int h = (int)(gw % heads);
  const bool is_q = h < Hq;
  const bool is_k = !is_q && h < Hq + Hkv;
  const int D = (is_q || is_k) ? Dqk : Dv;
  E* src = qkv + (size_t)t * ld_qkv +
           ((is_q || is_k) ? (size_t)h * Dqk : (size_t)(Hq + Hkv) * Dqk + (size_t)(h - Hq - Hkv) * Dv);
  const int pos = positions[t];
  const int epl = (D + 31) / 32;  // elements per lane, <= EPL
  float v[EPL];
#pragma unroll
  for (int i = 0; i < EPL; ++i) {
    const int d = lane + i * 32;
    v[i] = (i < epl && d < D) ? elem_to_f(src[d]) : 0.f;
  }
  E* dst = src;
  if (!is_q && (is_k ? kcache : vcache) != nullptr) {
    // with a cache the k / v heads go to their slot (in-place otherwise: dense attention reads qkv directly)
    const long long slot = slot_mapping ? slot_mapping[t] : -1;
    if (slot < 0) {
      dst = nullptr;  // padding token: nothing to cache
    } else {
      const long long blk = slot / block_size;
      const int off = (int)(slot % block_size);
      const int kvh = is_k ? (h - Hq) : (h - Hq - Hkv);
      E* base = is_k ? kcache : vcache;
      dst = base + (((size_t)blk * Hkv + kvh) * block_size + off) * (size_t)D;
    }
  }
  if (is_q || is_k) {
    const bf16* nw = is_q ? q_norm_w : k_norm_w;
    if (nw) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < EPL; ++i) ss += v[i] * v[i];
      ss = warp_sum(ss);
      const float inv = rsqrtf(ss / (float)D + norm_eps);
#pragma unroll
      for (int i = 0; i < EPL; ++i) {
        const int d = lane + i * 32;
        if (i < epl && d < D) {
          // round through bf16 like an unfused norm would before the rotation
          v[i] = __bfloat162float(__float2bfloat16(v[i] * inv * (__bfloat162float(nw[d]) + norm_w_offset)));
        }
      }
    }
    const int half = rot_dim / 2;
    const float* cs = cos_tab + (size_t)pos * half;
    const float* sn = sin_tab + (size_t)pos * half;
    if (!interleaved) {
      // partner of element d (< rot_dim) is d +/- half; exchange through this warp's shared-memory row
      float* row = rope_smem + (threadIdx.x >> 5) * (32 * EPL);
#pragma unroll
      for (int i = 0; i < EPL; ++i) {
        const int d = lane + i * 32;
        if (i < epl && d < D) row[d] = v[i];
      }
      __syncwarp();
#pragma unroll
      for (int i = 0; i < EPL; ++i) {
        const int d = lane + i * 32;
        if (i < epl && d < rot_dim) {
          const bool lo = d < half;
          const float partner = row[lo ? d + half : d - half];
          const int fi = lo ? d : d - half;
          const float c = cs[fi], sgn = sn[fi];
          v[i] = lo ? (v[i] * c - partner * sgn) : (v[i] * c + partner * sgn);
        }
      }
    } else {
#pragma unroll
      for (int i = 0; i < EPL; ++i) {
        const int d = lane + i * 32;
        const float partner = __shfl_xor_sync(0xffffffffu, v[i], 1);
        if (i < epl && d < rot_dim) {
          const int fi = d >> 1;
          const float c = cs[fi], sgn = sn[fi];
          v[i] = (d & 1) ? (v[i] * c + partner * sgn) : (v[i] * c - partner * sgn);
        }
      }
    }
  }
  if (dst) {
#pragma unroll
    for (int i = 0; i < EPL; ++i) {
      const int d = lane + i * 32;
      if (i < epl && d < D) elem_from_f(dst[d], v[i]);
    }
  }
  if (is_k && dst != src) {   // the rotated key also stays in the projection buffer
#pragma unroll
    for (int i = 0; i < EPL; ++i) {
      const int d = lane + i * 32;
      if (i < epl && d < D) elem_from_f(src[d], v[i]);
    }
  }
}

// Head dim 128 with full rotary width: every lane owns four elements so that both members of each rotation pair are
// lane-local (interleaved: elements 4l..4l+3; half-split: 2l, 2l+1, 64+2l, 65+2l) and all accesses are 4- or 8-byte
// vectors. V heads are only touched when they have to be copied into a cache.
template <bool INTERLEAVED>
__global__ void __launch_bounds__(256) rope_kv_write_d128_kernel(
    bf16* qkv, int ld_qkv, const int* __restrict__ positions, const long long* __restrict__ slot_mapping,
    const float* __restrict__ cos_tab, const float* __restrict__ sin_tab, const bf16* __restrict__ q_norm_w,
    const bf16* __restrict__ k_norm_w, float norm_eps, float norm_w_offset, bf16* kcache, bf16* vcache, int block_size,
    int T, int Hq, int Hkv, int heads_active) {
  pdl_launch_dependents();
  pdl_wait(TL_ROPE_KV);
  constexpr int D = 128;
  const int lane = threadIdx.x & 31;
  const long long gw = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (gw >= (long long)T * heads_active) return;
  const int t = (int)(gw / heads_active);
  const int h = (int)(gw % heads_active);
  bf16* src = qkv + (size_t)t * ld_qkv + (size_t)h * D;
  const bool is_q = h < Hq;
  const bool is_k = !is_q && h < Hq + Hkv;
  const int e0 = INTERLEAVED ? 4 * lane : 2 * lane;         // first element of the low pair block
  const int e1 = INTERLEAVED ? 4 * lane + 2 : 64 + 2 * lane;  // first element of the second block
  float v[4];
  {
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(src + e0));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(src + e1));
    v[0] = a.x, v[1] = a.y, v[2] = b.x, v[3] = b.y;
  }
  bf16* dst = src;
  if (!is_q && (is_k ? kcache : vcache) != nullptr) {
    const long long slot = slot_mapping ? slot_mapping[t] : -1;
    if (slot < 0) {
      dst = nullptr;
    } else {
      const long long blk = slot / block_size;
      const int off = (int)(slot % block_size);
      const int kvh = is_k ? (h - Hq) : (h - Hq - Hkv);
      dst = (is_k ? kcache : vcache) + (((size_t)blk * Hkv + kvh) * block_size + off) * (size_t)D;
    }
  }
  if (is_q || is_k) {
    const bf16* nw = is_q ? q_norm_w : k_norm_w;
    if (nw) {
      float ss = v[0] * v[0] + v[1] * v[1] + v[2] * v[2] + v[3] * v[3];
      ss = warp_sum(ss);
      const float inv = rsqrtf(ss / (float)D + norm_eps);
      const float2 wa = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(nw + e0));
      const float2 wb = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(nw + e1));
      // round through bf16 like an unfused norm would before the rotation
      v[0] = __bfloat162float(__float2bfloat16(v[0] * inv * (wa.x + norm_w_offset)));
      v[1] = __bfloat162float(__float2bfloat16(v[1] * inv * (wa.y + norm_w_offset)));
      v[2] = __bfloat162float(__float2bfloat16(v[2] * inv * (wb.x + norm_w_offset)));
      v[3] = __bfloat162float(__float2bfloat16(v[3] * inv * (wb.y + norm_w_offset)));
    }
    const int pos = positions[t];
    const float2 c = *reinterpret_cast<const float2*>(cos_tab + (size_t)pos * 64 + 2 * lane);
    const float2 sn = *reinterpret_cast<const float2*>(sin_tab + (size_t)pos * 64 + 2 * lane);
    float o[4];
    if (INTERLEAVED) {   // pairs (v0, v1) with angle 2l and (v2, v3) with angle 2l + 1
      o[0] = v[0] * c.x - v[1] * sn.x;
      o[1] = v[1] * c.x + v[0] * sn.x;
      o[2] = v[2] * c.y - v[3] * sn.y;
      o[3] = v[3] * c.y + v[2] * sn.y;
    } else {             // pairs (v0, v2) with angle 2l and (v1, v3) with angle 2l + 1
      o[0] = v[0] * c.x - v[2] * sn.x;
      o[2] = v[2] * c.x + v[0] * sn.x;
      o[1] = v[1] * c.y - v[3] * sn.y;
      o[3] = v[3] * c.y + v[1] * sn.y;
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) v[i] = o[i];
  }
  if (dst) {
    *reinterpret_cast<__nv_bfloat162*>(dst + e0) = __floats2bfloat162_rn(v[0], v[1]);
    *reinterpret_cast<__nv_bfloat162*>(dst + e1) = __floats2bfloat162_rn(v[2], v[3]);
  }
  if (is_k && dst != src) {   // the rotated key also stays in the projection buffer (prefill attention reads it there)
    *reinterpret_cast<__nv_bfloat162*>(src + e0) = __floats2bfloat162_rn(v[0], v[1]);
    *reinterpret_cast<__nv_bfloat162*>(src + e1) = __floats2bfloat162_rn(v[2], v[3]);
  }
}

// Norms over whole query / key projections (all heads of a token at once) or over every head by itself, rotation, cache write: one CTA
// per token.
struct RowRopeParams {
  void* buf;                  // [T, ld]: q (H heads of D) at 0, k (G heads of D) behind it, v (G heads of Dv) at v_col
  int ld, v_col, H, G, D, Dv, rot;
  const float *wq, *wk;       // norm weights [H * D], [G * D]; null: no norm
  int nq, nk;                 // numbers that enter the mean of q and k (padding columns are zero)
  float eps;
  const float *cos, *sin;     // [positions, rot / 2]; pairs are neighbouring dimensions
  const int* positions;
  const long long* slots;     // row of the caches, < 0: none
  void *kcache, *vcache;      // [block, G, block_size, D | Dv]
  int block_size;
  int v_from_k;               // values are the keys as projected (Dv == D)
  int store_v;                // v_from_k: also store them at v_col
  int GV;                     // value heads
  int unit;                   // > 0: q and k heads are divided by their own root mean square over `unit` columns, no weight
};

template <typename E>
__global__ void __launch_bounds__(256) row_rope_kv_kernel(const RowRopeParams p) {
  pdl_launch_dependents();
  pdl_wait(TL_ROPE_KV);
  __shared__ float red[2][8];
  extern __shared__ float part[];            // unit: sums of squares of the pieces of eight columns
  const int t = blockIdx.x, nq8 = p.H * p.D / 8, nk8 = p.G * p.D / 8, nv8 = p.GV * p.Dv / 8;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  E* q = reinterpret_cast<E*>(p.buf) + (size_t)t * p.ld;
  E* k = q + nq8 * 8;
  E* v = q + p.v_col;
  float rq = 1.f, rk = 1.f;
  if (p.wk) {
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x; i < nq8 + nk8; i += blockDim.x) {
      float x[8], ss = 0.f;
      load_row8(q + i * 8, x);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss = fmaf(x[j], x[j], ss);
      if (i < nq8) sq += ss;
      else sk += ss;
    }
    sq = warp_sum(sq), sk = warp_sum(sk);
    if (lane == 0) red[0][warp] = sq, red[1][warp] = sk;
    __syncthreads();
    sq = sk = 0.f;
    for (int w = 0; w < warps; ++w) sq += red[0][w], sk += red[1][w];
    rq = rsqrtf(sq / (float)p.nq + p.eps), rk = rsqrtf(sk / (float)p.nk + p.eps);
  }
  if (p.unit > 0) {           // a rotation leaves the sum of squares as it is
    for (int i = threadIdx.x; i < nq8 + nk8; i += blockDim.x) {
      float x[8], ss = 0.f;
      load_row8(q + i * 8, x);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss = fmaf(x[j], x[j], ss);
      part[i] = ss;
    }
    __syncthreads();
  }
  const long long slot = p.slots[t];
  E *kc = nullptr, *vc = nullptr;
  const size_t page = slot >= 0 ? (size_t)(slot / p.block_size) * p.G * p.block_size + slot % p.block_size : 0;
  const size_t vpage = slot >= 0 ? (size_t)(slot / p.block_size) * p.GV * p.block_size + slot % p.block_size : 0;
  if (slot >= 0) kc = reinterpret_cast<E*>(p.kcache), vc = reinterpret_cast<E*>(p.vcache);
  const int half = p.rot / 2;
  const float* cs = p.cos + (size_t)p.positions[t] * half;
  const float* sn = p.sin + (size_t)p.positions[t] * half;
  const int first = p.wk || p.unit > 0 || p.rot > 0 ? 0 : nq8;            // nothing to do for the queries
  for (int i = first + threadIdx.x; i < nq8 + nk8; i += blockDim.x) {
    const bool is_q = i < nq8;
    const int j8 = is_q ? i : i - nq8, h = j8 * 8 / p.D, d = j8 * 8 - h * p.D;
    E* at = is_q ? q + j8 * 8 : k + j8 * 8;
    float x[8];
    load_row8(at, x);
    if (!is_q && p.v_from_k) {
      if (vc) store_row8(vc + (page + (size_t)h * p.block_size) * p.Dv + d, x);
      if (p.store_v) store_row8(v + j8 * 8, x);
    }
    if (p.wk) {
      float w[8];
      load_row8((is_q ? p.wq : p.wk) + j8 * 8, w);
      const float r = is_q ? rq : rk;
#pragma unroll
      for (int j = 0; j < 8; ++j) x[j] *= r * w[j];
    }
    if (p.unit > 0) {
      const float* ps = part + i - d / 8;                   // the pieces of this head
      float ss = 0.f;
      for (int m = 0; m < p.D / 8; ++m) ss += ps[m];
      const float r = rsqrtf(ss / (float)p.unit + p.eps);
#pragma unroll
      for (int j = 0; j < 8; ++j) x[j] *= r;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (d + 2 * j >= p.rot) continue;
      const float c = cs[d / 2 + j], s = sn[d / 2 + j], a = x[2 * j], b = x[2 * j + 1];
      x[2 * j] = a * c - b * s;
      x[2 * j + 1] = b * c + a * s;
    }
    if (p.wk || p.unit > 0 || p.rot > 0) store_row8(at, x);
    if (!is_q && kc) store_row8(kc + (page + (size_t)h * p.block_size) * p.D + d, x);
  }
  if (!p.v_from_k && vc) {
    for (int i = threadIdx.x; i < nv8; i += blockDim.x) {
      const int h = i * 8 / p.Dv, d = i * 8 - h * p.Dv;
      float x[8];
      load_row8(v + i * 8, x);
      store_row8(vc + (vpage + (size_t)h * p.block_size) * p.Dv + d, x);
    }
  }
}

// Differential attention: o = a1 - lambda a2 for the two maps of a head, divided by its root mean square, times `post`. One warp per
// (token, head); in [T, H, 2, Dv] strided by token, out [T, H * Dv] likewise. N: real columns of the Dv.
template <typename E>
__global__ void __launch_bounds__(256) diff_combine_kernel(const E* __restrict__ in, long long in_tok, E* out, long long out_tok, int T, int H,
                                                           int Dv, int N, float lambda, float eps, float post) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long gw = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (gw >= (long long)T * H) return;
  const int t = (int)(gw / H), h = (int)(gw % H);
  const E* a = in + t * in_tok + (long long)h * 2 * Dv;
  E* o = out + t * out_tok + (long long)h * Dv;
  float ss = 0.f;
  for (int d = lane; d < Dv; d += 32) {
    const float x = to_f(a[d]) - lambda * to_f(a[Dv + d]);
    ss = fmaf(x, x, ss);
  }
  const float r = rsqrtf(warp_sum(ss) / (float)N + eps) * post;
  for (int d = lane; d < Dv; d += 32) from_f(o[d], (to_f(a[d]) - lambda * to_f(a[Dv + d])) * r);
}

// Heads that exchange their attention weights: with a[t, g, c] the weights of query head g applied to the values of key/value head c,
//     out[t, h] = sigmoid(gate[t, h]) sum_g talk[h, g] a[t, g, c(h)],   c(h) = h / (H / G)
// because the weighted sum over the heads' weights passes through the (linear) application to the values. A thread owns four columns of
// one c for TT tokens and HM of its query heads.
constexpr int MIX_PAD = 8;
struct HeadMixParams {
  const void* a;              // [T, H, G, Dv] (a token's part contiguous), a_tok apart
  long long a_tok;
  const float* talk;          // [H (g), G (c), HP]: talk[c * H / G + i, g] at i, HP = H / G rounded up to MIX_PAD, zeros behind
  const void* gate;           // optional logits [T, >= H], gate_tok apart
  long long gate_tok;
  void* out;                  // [T, H * Dv], out_tok apart
  long long out_tok;
  int T, H, G, Dv;
};

template <typename E, int TT, int HM>
__global__ void __launch_bounds__(128) head_mix_kernel(const HeadMixParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int col = (blockIdx.x * 128 + threadIdx.x) * 4, width = p.G * p.Dv, t0 = blockIdx.y * TT;
  if (col >= width) return;
  const int c = col / p.Dv, per = p.H / p.G, hp = (per + MIX_PAD - 1) / MIX_PAD * MIX_PAD, h0 = blockIdx.z * HM;
  const E* a[TT];
#pragma unroll
  for (int i = 0; i < TT; ++i) a[i] = reinterpret_cast<const E*>(p.a) + min(t0 + i, p.T - 1) * p.a_tok + col;
  const float* talk = p.talk + (size_t)c * hp + h0;
  float4 acc[TT][HM];
#pragma unroll
  for (int i = 0; i < TT; ++i)
#pragma unroll
    for (int h = 0; h < HM; ++h) acc[i][h] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
  for (int g = 0; g < p.H; ++g) {
    float w[HM];
#pragma unroll
    for (int h = 0; h < HM; ++h) w[h] = __ldg(talk + (size_t)g * p.G * hp + h);
#pragma unroll
    for (int i = 0; i < TT; ++i) {
      const float4 x = load_row4(a[i] + (size_t)g * width);
#pragma unroll
      for (int h = 0; h < HM; ++h) {
        acc[i][h].x = fmaf(w[h], x.x, acc[i][h].x), acc[i][h].y = fmaf(w[h], x.y, acc[i][h].y);
        acc[i][h].z = fmaf(w[h], x.z, acc[i][h].z), acc[i][h].w = fmaf(w[h], x.w, acc[i][h].w);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < TT; ++i) {
    const int t = t0 + i;
    if (t >= p.T) break;
#pragma unroll
    for (int h = 0; h < HM; ++h) {
      if (h0 + h >= per) break;
      const int head = c * per + h0 + h;
      const float s = p.gate ? 1.f / (1.f + expf(-to_f(reinterpret_cast<const E*>(p.gate)[t * p.gate_tok + head]))) : 1.f;
      const float4 v = acc[i][h];
      store_row4(reinterpret_cast<E*>(p.out) + t * p.out_tok + (size_t)head * p.Dv + col % p.Dv, make_float4(v.x * s, v.y * s, v.z * s, v.w * s));
    }
  }
}

template <typename E>
int launch_head_mix(const HeadMixParams& p, cudaStream_t s) {
  const int per = p.H / p.G;
  const unsigned x = (p.G * p.Dv / 4 + 127) / 128;
  auto go = [&](auto one, auto two, int hm) {
    const unsigned z = (per + hm - 1) / hm;
    return p.T < 512 ? launch_kernel(one, dim3(x, p.T, z), dim3(128), 0, s, p) : launch_kernel(two, dim3(x, (p.T + 1) / 2, z), dim3(128), 0, s, p);
  };
  if (per <= 1) return go(head_mix_kernel<E, 1, 1>, head_mix_kernel<E, 2, 1>, 1);
  if (per <= 2) return go(head_mix_kernel<E, 1, 2>, head_mix_kernel<E, 2, 2>, 2);
  if (per <= 4) return go(head_mix_kernel<E, 1, 4>, head_mix_kernel<E, 2, 4>, 4);
  return go(head_mix_kernel<E, 1, 8>, head_mix_kernel<E, 2, 8>, 8);
}

__device__ __forceinline__ float gated_act(float g, bool gelu, bool exact) {
  if (gelu) return gelu_tanh_f(g);
  return exact ? g / (1.f + expf(-g)) : silu_f(g);
}

// out[t, f] = act(gu[t, f]) * gu[t, F + f]; act 1 = SiLU (SwiGLU), 2 = tanh-GELU (GeGLU). act 3 / 4: the same two
// activations on a pair-interleaved projection output, out[t, f] = act(gu[t, 2f]) * gu[t, 2f + 1]. act 5 / 6: the gated unit with both
// parts clamped at `limit`, side by side / interleaved. row_gate (fp32 logits, one per
// row, `gate_ld` apart): the row is scaled by its sigmoid.
template <typename E>
__global__ void __launch_bounds__(256) gated_act_mul_kernel(const E* __restrict__ gu, int ld_gu, E* out, int ldo, int T, int F, int act, float limit,
                                                           const float* __restrict__ row_gate, int gate_ld) {
  pdl_launch_dependents();
  pdl_wait(TL_GATED_ACT);
  const int nvec = F / 8;
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= (long long)T * nvec) return;
  const int t = (int)(idx / nvec);
  const int v = (int)(idx % nvec);
  float g[8], u[8], o[8];
  if (act == 3 || act == 4 || act == 6) {
    float lo[8], hi[8];
    load_row8(gu + (size_t)t * ld_gu + v * 16, lo);
    load_row8(gu + (size_t)t * ld_gu + v * 16 + 8, hi);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      g[j] = lo[2 * j];
      u[j] = lo[2 * j + 1];
      g[4 + j] = hi[2 * j];
      u[4 + j] = hi[2 * j + 1];
    }
  } else {
    load_row8(gu + (size_t)t * ld_gu + v * 8, g);
    load_row8(gu + (size_t)t * ld_gu + F + v * 8, u);
  }
  const bool gelu = act == 2 || act == 4;
#pragma unroll
  for (int j = 0; j < 8; ++j)
    o[j] = act >= 5 ? clamped_gate_f<sizeof(E) == 4>(g[j], u[j], limit) : gated_act(g[j], gelu, sizeof(E) == 4) * u[j];
  if (row_gate) {
    const float s = 1.f / (1.f + expf(-row_gate[(size_t)t * gate_ld]));
#pragma unroll
    for (int j = 0; j < 8; ++j) o[j] *= s;
  }
  store_row8(out + (size_t)t * ldo + v * 8, o);
}

// out = a N(z) + b N(z^2) + c N(z^3) + e with the powers taken element by element and N(y) = y / sqrt(mean(y^2) + eps) over
// a row's F values; coef = (a, b, c, e). One CTA per row, statistics in fp32. Rows of at most THREADS * VPT * 8 values stay in
// registers (VPT > 0), longer ones are read twice.
template <typename E, int THREADS, int VPT>
__global__ void __launch_bounds__(THREADS) poly_norm_kernel(const E* __restrict__ z, int ldz, E* out, int ldo, int F, int Fp,
                                                            const float* __restrict__ coef, float eps) {
  pdl_launch_dependents();
  pdl_wait(TL_GATED_ACT);
  __shared__ float red[3][THREADS / 32];
  const E* zr = z + (size_t)blockIdx.x * ldz;
  const int nvec = Fp / 8, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float keep[VPT > 0 ? VPT : 1][8];
  float s2 = 0.f, s4 = 0.f, s6 = 0.f;
  auto add = [&](const float* v) {       // padding columns hold zeros
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float q = v[j] * v[j];
      s2 += q;
      s4 = fmaf(q, q, s4);
      s6 = fmaf(q * q, q, s6);
    }
  };
  if constexpr (VPT > 0) {
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * THREADS;
      if (c < nvec) load_row8(zr + c * 8, keep[i]);
      else
#pragma unroll
        for (int j = 0; j < 8; ++j) keep[i][j] = 0.f;
    }
#pragma unroll
    for (int i = 0; i < VPT; ++i) add(keep[i]);
  } else {
    for (int c = threadIdx.x; c < nvec; c += THREADS) {
      load_row8(zr + c * 8, keep[0]);
      add(keep[0]);
    }
  }
  s2 = warp_sum(s2), s4 = warp_sum(s4), s6 = warp_sum(s6);
  if (lane == 0) red[0][warp] = s2, red[1][warp] = s4, red[2][warp] = s6;
  __syncthreads();
  s2 = s4 = s6 = 0.f;
#pragma unroll
  for (int w = 0; w < THREADS / 32; ++w) s2 += red[0][w], s4 += red[1][w], s6 += red[2][w];
  const float n = (float)F;
  const float a = coef[0] * rsqrtf(s2 / n + eps), b = coef[1] * rsqrtf(s4 / n + eps), c3 = coef[2] * rsqrtf(s6 / n + eps), e = coef[3];
  E* orow = out + (size_t)blockIdx.x * ldo;
  auto put = [&](int c, float* v) {
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = fmaf(fmaf(fmaf(c3, v[j], b), v[j], a), v[j], e);
    store_row8(orow + c * 8, v);
  };
  if constexpr (VPT > 0) {
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * THREADS;
      if (c < nvec) put(c, keep[i]);
    }
  } else {
    for (int c = threadIdx.x; c < nvec; c += THREADS) {
      load_row8(zr + c * 8, keep[0]);
      put(c, keep[0]);
    }
  }
}

template <typename E>
int launch_poly_norm(const E* z, int ldz, E* out, int ldo, int T, int F, int Fp, const float* coef, float eps, cudaStream_t s) {
  const int nvec = Fp / 8;
  const dim3 grid((unsigned)T);
  auto go = [&](auto kernel, int threads) {
    return launch_kernel(kernel, grid, dim3(threads), 0, s, z, ldz, out, ldo, F, Fp, coef, eps);
  };
  switch ((nvec + 255) / 256) {
    case 1: return go(poly_norm_kernel<E, 256, 1>, 256);
    case 2: return go(poly_norm_kernel<E, 256, 2>, 256);
    case 3: return go(poly_norm_kernel<E, 256, 3>, 256);
    case 4: return go(poly_norm_kernel<E, 256, 4>, 256);
    case 5: return go(poly_norm_kernel<E, 256, 5>, 256);
    case 6: return go(poly_norm_kernel<E, 256, 6>, 256);
    case 7: case 8: return go(poly_norm_kernel<E, 512, 4>, 512);
    default: return go(poly_norm_kernel<E, 512, 0>, 512);
  }
}

__global__ void __launch_bounds__(256) embedding_kernel(const long long* __restrict__ ids, const bf16* __restrict__ table,
                                                       bf16* out, int T, int H, int vocab_start, int vocab_end,
                                                       float scale) {
  pdl_launch_dependents();
  pdl_wait(TL_EMBED);
  const int nvec = H / 8;
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= (long long)T * nvec) return;
  const int t = (int)(idx / nvec);
  const int v = (int)(idx % nvec);
  const long long id = ids[t];
  uint4 u = make_uint4(0, 0, 0, 0);
  if (id >= vocab_start && id < vocab_end) {
    u = __ldg(reinterpret_cast<const uint4*>(table + (size_t)(id - vocab_start) * H + v * 8));
    if (scale != 1.f) {
      float f[8];
      unpack8(u, f);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] *= scale;
      u = pack8(f);
    }
  }
  *reinterpret_cast<uint4*>(out + (size_t)t * H + v * 8) = u;
}

// out = a + gate * b (gate per batch row-vector), or out = a + b when gate == nullptr.
__global__ void __launch_bounds__(256) gated_residual_kernel(const bf16* __restrict__ a, const bf16* __restrict__ b,
                                                            const bf16* __restrict__ gate, int ld_gate,
                                                            int rows_per_batch, bf16* out, int T, int H) {
  pdl_launch_dependents();
  pdl_wait();
  const int nvec = H / 8;
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= (long long)T * nvec) return;
  const int t = (int)(idx / nvec);
  const int v = (int)(idx % nvec);
  float fa[8], fb[8], o[8];
  unpack8(*reinterpret_cast<const uint4*>(a + (size_t)t * H + v * 8), fa);
  unpack8(*reinterpret_cast<const uint4*>(b + (size_t)t * H + v * 8), fb);
  if (gate) {
    float g[8];
    const int bi = rows_per_batch > 0 ? t / rows_per_batch : 0;
    unpack8(*reinterpret_cast<const uint4*>(gate + (size_t)bi * ld_gate + v * 8), g);
#pragma unroll
    for (int j = 0; j < 8; ++j) o[j] = fa[j] + g[j] * fb[j];
  } else {
#pragma unroll
    for (int j = 0; j < 8; ++j) o[j] = fa[j] + fb[j];
  }
  *reinterpret_cast<uint4*>(out + (size_t)t * H + v * 8) = pack8(o);
}

template <typename F>
int launch_norm(int H, F&& f) {
  const int nvec = H / 8;
  if (nvec <= 128) return f(std::integral_constant<int, 128>{}, std::integral_constant<int, 1>{});
  if (nvec <= 256) return f(std::integral_constant<int, 256>{}, std::integral_constant<int, 1>{});
  if (nvec <= 512) return f(std::integral_constant<int, 256>{}, std::integral_constant<int, 2>{});
  if (nvec <= 1024) return f(std::integral_constant<int, 256>{}, std::integral_constant<int, 4>{});
  if (nvec <= 2048) return f(std::integral_constant<int, 512>{}, std::integral_constant<int, 4>{});
  return -3;
}

static thread_local int launch_rc = 0;
inline int last_err() { return launch_rc; }

}  // namespace
}  // namespace swb

extern "C" {

int swb_rmsnorm_prefetch(const void* x, int ldx, void* residual, int ldr, const void* w, void* out, int ldo, int T,
                         int H, float eps, float w_offset, const void* prefetch_ptr, long long prefetch_bytes,
                         void* stream);

int swb_rmsnorm(const void* x, int ldx, void* residual, int ldr, const void* w, void* out, int ldo, int T, int H,
                float eps, float w_offset, void* stream) {
  return swb_rmsnorm_prefetch(x, ldx, residual, ldr, w, out, ldo, T, H, eps, w_offset, nullptr, 0, stream);
}

// As swb_rmsnorm; additionally asks L2 to fetch prefetch_bytes (16-byte aligned start) of the next kernel's weights.
int swb_rmsnorm_prefetch(const void* x, int ldx, void* residual, int ldr, const void* w, void* out, int ldo, int T,
                         int H, float eps, float w_offset, const void* prefetch_ptr, long long prefetch_bytes,
                         void* stream) {
  using namespace swb;
  if (T <= 0) return 0;
  if (H % 8 != 0 || ldx % 8 != 0 || ldo % 8 != 0 || (residual && ldr % 8 != 0)) return -3;
  if (prefetch_ptr && ((reinterpret_cast<uintptr_t>(prefetch_ptr) & 15) || prefetch_bytes < 0)) return -3;
  const uint8_t* pf = prefetch_bytes > 0 ? reinterpret_cast<const uint8_t*>(prefetch_ptr) : nullptr;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return launch_norm(H, [&](auto TH, auto VP) {
    constexpr int THREADS = decltype(TH)::value, VPT = decltype(VP)::value;
    launch_rc = launch_kernel(rmsnorm_kernel<THREADS, VPT>, dim3(T), dim3(THREADS), 0, s, reinterpret_cast<const bf16*>(x), ldx,
                                                        reinterpret_cast<bf16*>(residual), ldr,
                                                        reinterpret_cast<const bf16*>(w), reinterpret_cast<bf16*>(out),
                                                        ldo, H, eps, w_offset, pf, prefetch_bytes);
    return last_err();
  });
}

int swb_layernorm_mod(const void* x, int ldx, const void* scale, const void* shift, int ld_mod, int rows_per_batch,
                      const void* gamma, const void* beta, void* out, int ldo, int T, int H, float eps,
                      void* stream) {
  using namespace swb;
  if (T <= 0) return 0;
  if (H % 8 != 0 || ldx % 8 != 0 || ldo % 8 != 0 || ld_mod % 8 != 0) return -3;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return launch_norm(H, [&](auto TH, auto VP) {
    constexpr int THREADS = decltype(TH)::value, VPT = decltype(VP)::value;
    launch_rc = launch_kernel(layernorm_mod_kernel<THREADS, VPT>, dim3(T), dim3(THREADS), 0, s, reinterpret_cast<const bf16*>(x), ldx, reinterpret_cast<const bf16*>(scale),
        reinterpret_cast<const bf16*>(shift), ld_mod, rows_per_batch, reinterpret_cast<const bf16*>(gamma),
        reinterpret_cast<const bf16*>(beta), reinterpret_cast<bf16*>(out), ldo, H, eps);
    return last_err();
  });
}

// fp32 = 1: qkv and both caches hold floats (q_norm_w / k_norm_w stay bf16). Dv: width of the v heads and of the v cache.
int swb_rope_kv_write_ex(void* qkv, int ld_qkv, const int* positions, const long long* slot_mapping,
                         const float* cos_tab, const float* sin_tab, int rot_dim, int interleaved, const void* q_norm_w,
                         const void* k_norm_w, float norm_eps, float norm_w_offset, void* kcache, void* vcache,
                         int block_size, int T, int Hq, int Hkv, int D, int Dv, int fp32, void* stream) {
  using namespace swb;
  if (T <= 0) return 0;
  if (D > 512 || Dv > 512 || rot_dim > D || (rot_dim & 1)) return -3;
  const int wpb = 8;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const bf16* qn = reinterpret_cast<const bf16*>(q_norm_w);
  const bf16* kn = reinterpret_cast<const bf16*>(k_norm_w);
  if (!fp32 && D == 128 && Dv == 128 && rot_dim == 128 && (ld_qkv % 2) == 0 && (reinterpret_cast<uintptr_t>(qkv) & 3) == 0) {
    const int heads_active = Hq + Hkv + (vcache ? Hkv : 0);   // V stays where it is unless it goes to a cache
    const long long nblk = ((long long)T * heads_active + wpb - 1) / wpb;
    auto kern = interleaved ? rope_kv_write_d128_kernel<true> : rope_kv_write_d128_kernel<false>;
    launch_rc = launch_kernel(kern, dim3((unsigned)nblk), dim3(wpb * 32), 0, st, reinterpret_cast<bf16*>(qkv), ld_qkv,
                              positions, slot_mapping, cos_tab, sin_tab, qn, kn, norm_eps, norm_w_offset,
                              reinterpret_cast<bf16*>(kcache), reinterpret_cast<bf16*>(vcache), block_size, T, Hq, Hkv,
                              heads_active);
    return last_err();
  }
  const long long warps = (long long)T * (Hq + 2 * Hkv);
  const dim3 grid((unsigned)((warps + wpb - 1) / wpb)), block(wpb * 32);
  const bool wide = D > 256 || Dv > 256;
  if (fp32) {
    auto kern = wide ? rope_kv_write_kernel<float, 16> : rope_kv_write_kernel<float, 8>;
    launch_rc = launch_kernel(kern, grid, block, 0, st, reinterpret_cast<float*>(qkv), ld_qkv, positions, slot_mapping,
                              cos_tab, sin_tab, rot_dim, interleaved, qn, kn, norm_eps, norm_w_offset,
                              reinterpret_cast<float*>(kcache), reinterpret_cast<float*>(vcache), block_size, T, Hq, Hkv, D,
                              Dv);
  } else {
    auto kern = wide ? rope_kv_write_kernel<bf16, 16> : rope_kv_write_kernel<bf16, 8>;
    launch_rc = launch_kernel(kern, grid, block, 0, st, reinterpret_cast<bf16*>(qkv), ld_qkv, positions, slot_mapping,
                              cos_tab, sin_tab, rot_dim, interleaved, qn, kn, norm_eps, norm_w_offset,
                              reinterpret_cast<bf16*>(kcache), reinterpret_cast<bf16*>(vcache), block_size, T, Hq, Hkv, D,
                              Dv);
  }
  return last_err();
}

int swb_rope_kv_write(void* qkv, int ld_qkv, const int* positions, const long long* slot_mapping,
                      const float* cos_tab, const float* sin_tab, int rot_dim, int interleaved, const void* q_norm_w,
                      const void* k_norm_w, float norm_eps, float norm_w_offset, void* kcache, void* vcache,
                      int block_size, int T, int Hq, int Hkv, int D, void* stream) {
  return swb_rope_kv_write_ex(qkv, ld_qkv, positions, slot_mapping, cos_tab, sin_tab, rot_dim, interleaved, q_norm_w,
                              k_norm_w, norm_eps, norm_w_offset, kcache, vcache, block_size, T, Hq, Hkv, D, D, 0, stream);
}

// Fp: padded row width (a multiple of 8), F <= Fp values enter the statistics; fp32 selects the element type of z and out.
int swb_poly_norm(const void* z, int ldz, void* out, int ldo, int T, int F, int Fp, const float* coef, float eps, int fp32,
                  void* stream) {
  using namespace swb;
  if (T <= 0) return 0;
  if (F <= 0 || F > Fp || (Fp % 8) || (ldz % 8) || (ldo % 8) || !coef) return -3;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (fp32) return launch_poly_norm(reinterpret_cast<const float*>(z), ldz, reinterpret_cast<float*>(out), ldo, T, F, Fp, coef, eps, s);
  return launch_poly_norm(reinterpret_cast<const bf16*>(z), ldz, reinterpret_cast<bf16*>(out), ldo, T, F, Fp, coef, eps, s);
}
// row_gate: see gated_act_mul_kernel; fp32 selects the element type of gate_up and out.
int swb_gated_act_mul_ex(const void* gate_up, int ld_gu, void* out, int ldo, int T, int F, int act, float limit, const float* row_gate, int gate_ld,
                         int fp32, void* stream) {
  using namespace swb;
  if (T <= 0) return 0;
  if (F % 8 != 0 || ld_gu % 8 != 0 || ldo % 8 != 0) return -3;
  const long long n = (long long)T * (F / 8);
  const dim3 grid((unsigned)((n + 255) / 256)), block(256);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (fp32)
    return launch_kernel(gated_act_mul_kernel<float>, grid, block, 0, s, reinterpret_cast<const float*>(gate_up), ld_gu,
                         reinterpret_cast<float*>(out), ldo, T, F, act, limit, row_gate, gate_ld);
  return launch_kernel(gated_act_mul_kernel<bf16>, grid, block, 0, s, reinterpret_cast<const bf16*>(gate_up), ld_gu,
                       reinterpret_cast<bf16*>(out), ldo, T, F, act, limit, row_gate, gate_ld);
}
int swb_gated_act_mul(const void* gate_up, int ld_gu, void* out, int ldo, int T, int F, int act, void* stream) {
  return swb_gated_act_mul_ex(gate_up, ld_gu, out, ldo, T, F, act, 0.f, nullptr, 0, 0, stream);
}

// See RowRopeParams. D, Dv, ld and v_col multiples of 8, buffers 16-byte aligned (32 in fp32). GV 0: as many value heads as key heads.
int swb_row_rope_kv_write(void* buf, int ld, int v_col, int H, int G, int D, int Dv, int rot, const float* wq, const float* wk, int nq, int nk,
                          float eps, const float* cos, const float* sin, const int* positions, const long long* slots, void* kcache,
                          void* vcache, int block_size, int v_from_k, int store_v, int GV, int unit, int T, int fp32, void* stream) {
  using namespace swb;
  if (T <= 0) return 0;
  if (GV <= 0) GV = G;
  if (unit < 0 || unit > D || (unit && wk) || (v_from_k && GV != G)) return -3;
  if (H < 0 || G < 1 || D < 8 || Dv < 8 || ((D | Dv | ld | v_col) % 8) || rot < 0 || rot > D || (rot % 2) || block_size < 1 || !kcache || !vcache ||
      !slots || (wk && (nk < 1 || (H > 0 && (!wq || nq < 1)))) || (v_from_k && Dv != D))
    return -3;
  const RowRopeParams p{buf, ld, v_col, H, G, D, Dv, rot, wq, wk, nq > 0 ? nq : 1, nk > 0 ? nk : 1, eps, cos, sin, positions, slots, kcache,
                        vcache, block_size, v_from_k, store_v, GV, unit};
  const int work = (H + G) * D / 8;
  const dim3 grid((unsigned)T), block(work <= 64 ? 64 : work <= 128 ? 128 : 256);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const size_t smem = unit ? (size_t)work * sizeof(float) : 0;
  if (smem > 48 * 1024) return -3;
  return fp32 ? launch_kernel(row_rope_kv_kernel<float>, grid, block, smem, s, p) : launch_kernel(row_rope_kv_kernel<bf16>, grid, block, smem, s, p);
}

// See HeadMixParams. Dv and the strides multiples of 4, rows 8-byte (fp32: 16-byte) aligned.
int swb_head_mix(const void* a, long long a_tok, const float* talk, const void* gate, long long gate_tok, void* out, long long out_tok, int T,
                 int H, int G, int Dv, int fp32, void* stream) {
  using namespace swb;
  if (T <= 0) return 0;
  if (H < 1 || G < 1 || H % G || Dv < 4 || ((Dv | a_tok | out_tok) % 4) || !talk) return -3;
  const HeadMixParams p{a, a_tok, talk, gate, gate_tok, out, out_tok, T, H, G, Dv};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return fp32 ? launch_head_mix<float>(p, s) : launch_head_mix<bf16>(p, s);
}

int swb_diff_combine(const void* in, long long in_tok, void* out, long long out_tok, int T, int H, int Dv, int N, float lambda, float eps,
                     float post, int fp32, void* stream) {
  using namespace swb;
  if (T <= 0) return 0;
  if (H < 1 || Dv < 1 || N < 1 || N > Dv) return -3;
  const dim3 grid((unsigned)(((long long)T * H + 7) / 8)), block(256);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (fp32)
    return launch_kernel(diff_combine_kernel<float>, grid, block, 0, s, reinterpret_cast<const float*>(in), in_tok,
                         reinterpret_cast<float*>(out), out_tok, T, H, Dv, N, lambda, eps, post);
  return launch_kernel(diff_combine_kernel<bf16>, grid, block, 0, s, reinterpret_cast<const bf16*>(in), in_tok,
                       reinterpret_cast<bf16*>(out), out_tok, T, H, Dv, N, lambda, eps, post);
}

int swb_embedding(const long long* ids, const void* table, void* out, int T, int H, int vocab_start, int vocab_end,
                  float scale, void* stream) {
  using namespace swb;
  if (T <= 0) return 0;
  if (H % 8 != 0) return -3;
  const long long n = (long long)T * (H / 8);
  launch_rc = launch_kernel(embedding_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, reinterpret_cast<cudaStream_t>(stream), ids, reinterpret_cast<const bf16*>(table), reinterpret_cast<bf16*>(out), T, H, vocab_start, vocab_end, scale);
  return last_err();
}

int swb_gated_residual(const void* a, const void* b, const void* gate, int ld_gate, int rows_per_batch, void* out,
                       int T, int H, void* stream) {
  using namespace swb;
  if (T <= 0) return 0;
  if (H % 8 != 0 || (gate && ld_gate % 8 != 0)) return -3;
  const long long n = (long long)T * (H / 8);
  launch_rc = launch_kernel(gated_residual_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, reinterpret_cast<cudaStream_t>(stream), reinterpret_cast<const bf16*>(a), reinterpret_cast<const bf16*>(b), reinterpret_cast<const bf16*>(gate), ld_gate,
      rows_per_batch, reinterpret_cast<bf16*>(out), T, H);
  return last_err();
}

}  // extern "C"
