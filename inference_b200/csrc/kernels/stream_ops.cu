// Kernels around a 32-bit residual stream: embedding into the stream and the fused step between two sublayers.
//
// stream_norm_kernel is that step in one pass over a row:
//     x   += norm1(branch)            branch = a projection output row, or the mean of a token's expert output rows
//     out  = norm2(x) * out_scale     or the stream itself, for a projection that reads it un-normalised
// A layer with norms before and after each sublayer then needs one such launch per sublayer. Both norms are layer norms
// (mean removed, weight and bias) or RMS norms, computed in fp32 on the row held in registers (squared deviations from the
// mean, never a difference of large sums). The output is stored once per token, or to every row of an expert-sorted buffer that the token's
// routing names, so the gather in front of a grouped GEMM costs no launch of its own.
// The EXT instantiations add what some designs need on top: RMS norms over equal groups of columns, a stream that is read
// from another buffer than it is written to, the depth average, in which the joined stream is filed as one more result
// and x becomes a weighted sum of all results so far, and a second part of the branch: weighted expert output rows beside a
// dense row (parallel sublayers join the stream together).
// Rows are padded to a multiple of 8 columns; padding columns of the stream, the weights and the outputs are zero and do
// not enter the statistics.
#include "common.cuh"

namespace swb {

SWB_REGISTER_STATUS_UNIT(stream_ops);

namespace {

struct StreamNormParams {
  float* x;                  // [T, ldx] residual stream
  int ldx;
  const long long* rows;     // optional: process row rows[i] of x as output row i (then no branch)
  const void* branch;        // optional bf16 / fp32 [*, ld_branch]
  int ld_branch, branch_fp32;
  const int* branch_rows;    // optional [T, branch_top]: the branch is the weighted sum of these rows
  int branch_top;
  float branch_weight;
  const float *w1, *b1;      // norm of the branch (b1 optional; w1 null: the branch is added as it is)
  const float *w2, *b2;      // norm of the stream (w2 null: the stream itself is stored)
  void* out;                 // optional bf16 / fp32 [*, ldo]
  int ldo, out_fp32;
  const int* out_rows;       // optional [T, out_top]: the output row goes to all of these rows
  int out_top;
  int H, Hp;
  float eps, out_scale;
  int center;                // 1: layer norm, 0: RMS norm
  // EXT only
  int groups;                // RMS norms over `groups` equal parts of the H columns
  const float* x_in;         // optional: the stream is read here (row stride ldx) and written to x
  float* hist;               // optional depth average: results 0 .. n_hist - 1, [T, ldx] each, `hist_stride` apart
  long long hist_stride;
  int n_hist;
  const float* mix;          // [n_hist + 1]: x <- sum_j mix[j] hist[j] + mix[n_hist] x; the joined x becomes hist[n_hist]
  const void* extra;         // optional bf16 / fp32 [*, ld_extra]: rows extra_rows[t, k] times extra_weights[t, k] join the branch
  int ld_extra, extra_fp32;
  const int* extra_rows;     // [T, extra_top]
  const float* extra_weights;
  int extra_top;
};

__device__ __forceinline__ float4 load4(const void* base, size_t off, int fp32) {
  if (fp32) return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(base) + off);
  const uint2 u = *reinterpret_cast<const uint2*>(reinterpret_cast<const bf16*>(base) + off);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(void* base, size_t off, int fp32, float4 v) {
  if (fp32) {
    *reinterpret_cast<float4*>(reinterpret_cast<float*>(base) + off) = v;
    return;
  }
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(reinterpret_cast<bf16*>(base) + off) =
      make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
}

// Sum over the block; `red` alternates between two slots so that one barrier per reduction is enough.
template <int THREADS>
__device__ __forceinline__ float block_total(float v, float* red) {
  v = warp_sum(v);
  if constexpr (THREADS == 32) return v;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (lane == 0) red[warp] = v;
  __syncthreads();
  return warp_sum(lane < THREADS / 32 ? red[lane] : 0.f);
}

// Mean and sum of squared deviations of a row whose threads hold N values each: every thread takes those of its own
// values, then equal-sized groups are merged pairwise (M2 = M2a + M2b + (mean_a - mean_b)^2 n / 2), so one barrier serves
// both and no large sums cancel.
template <int THREADS, int N>
__device__ __forceinline__ float2 block_moments(const float* v, float* red) {
  float m = 0.f, q = 0.f, n = (float)N;
#pragma unroll
  for (int i = 0; i < N; ++i) m += v[i];
  m *= 1.f / N;
#pragma unroll
  for (int i = 0; i < N; ++i) q += (v[i] - m) * (v[i] - m);
  auto merge = [&](int o) {
    const float mo = __shfl_xor_sync(0xffffffffu, m, o), qo = __shfl_xor_sync(0xffffffffu, q, o), d = m - mo;
    q += qo + d * d * (0.5f * n);
    m = 0.5f * (m + mo);
    n *= 2.f;
  };
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) merge(o);
  constexpr int WARPS = THREADS / 32;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (lane == 0) red[warp] = m, red[32 + warp] = q;
  __syncthreads();
  m = red[lane % WARPS], q = red[32 + lane % WARPS];
#pragma unroll
  for (int o = WARPS / 2; o > 0; o >>= 1) merge(o);
  return make_float2(m, q);
}

// v <- norm(v) * w + b over the first H columns of the row (thread t owns float4 columns t, t + THREADS, ...)
template <int THREADS, int VPT>
__device__ __forceinline__ void norm_row(float4* v, const float* __restrict__ w, const float* __restrict__ b, int H, int nvec,
                                         float eps, int center, float* red) {
  float mean = 0.f, ss = 0.f;
  const bool full = center && H == THREADS * VPT * 4;     // every thread holds the same number of columns
  if (full) {
    const float2 mq = block_moments<THREADS, VPT * 4>(reinterpret_cast<const float*>(v), red);
    mean = mq.x, ss = mq.y;
  } else if (center) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) s += (v[i].x + v[i].y) + (v[i].z + v[i].w);   // padding columns hold zeros
    mean = block_total<THREADS>(s, red) / (float)H;
    red += 32;
  }
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (threadIdx.x + i * THREADS) * 4;
    v[i].x -= mean, v[i].y -= mean, v[i].z -= mean, v[i].w -= mean;
    if (full) continue;
    if (c < H) ss += v[i].x * v[i].x;
    if (c + 1 < H) ss += v[i].y * v[i].y;
    if (c + 2 < H) ss += v[i].z * v[i].z;
    if (c + 3 < H) ss += v[i].w * v[i].w;
  }
  if (!full) ss = block_total<THREADS>(ss, red);
  const float r = rsqrtf(ss / (float)H + eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c4 = threadIdx.x + i * THREADS;
    if (c4 < nvec) {
      const float4 ww = __ldg(reinterpret_cast<const float4*>(w) + c4);
      const float4 bb = b ? __ldg(reinterpret_cast<const float4*>(b) + c4) : make_float4(0.f, 0.f, 0.f, 0.f);
      v[i] = make_float4(v[i].x * r * ww.x + bb.x, v[i].y * r * ww.y + bb.y, v[i].z * r * ww.z + bb.z,
                         v[i].w * r * ww.w + bb.w);
    }
  }
}

// RMS norm in groups of gs columns. Groups of whole 128-column chunks (the columns of one warp and one i) sum per chunk;
// other sizes sum through a row of squares in shared memory. `part` holds Hp / 4 + H / gs floats at least (Hp + H / gs then).
template <int THREADS, int VPT>
__device__ __forceinline__ void group_norm_row(float4* v, const float* __restrict__ w, int H, int nvec, int groups, float eps,
                                               float* part) {
  const int gs = H / groups, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  __syncthreads();                                   // an earlier norm may still be reading `part`
  if (gs % 128 == 0) {
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const float q = warp_sum((v[i].x * v[i].x + v[i].y * v[i].y) + (v[i].z * v[i].z + v[i].w * v[i].w));
      if (lane == 0) part[warp + i * (THREADS / 32)] = q;
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c4 = threadIdx.x + i * THREADS;
      if (c4 >= nvec) continue;
      const int g = c4 * 4 / gs, per = gs / 128;
      float ss = 0.f;
      if (g < groups)
        for (int k = 0; k < per; ++k) ss += part[g * per + k];
      const float r = rsqrtf(ss / (float)gs + eps);
      const float4 ww = __ldg(reinterpret_cast<const float4*>(w) + c4);
      v[i] = make_float4(v[i].x * r * ww.x, v[i].y * r * ww.y, v[i].z * r * ww.z, v[i].w * r * ww.w);
    }
    return;
  }
  float* sums = part + nvec * 4;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c4 = threadIdx.x + i * THREADS;
    if (c4 < nvec)
      reinterpret_cast<float4*>(part)[c4] = make_float4(v[i].x * v[i].x, v[i].y * v[i].y, v[i].z * v[i].z, v[i].w * v[i].w);
  }
  __syncthreads();
  for (int g = warp; g < groups; g += THREADS / 32) {
    float ss = 0.f;
    for (int c = lane; c < gs; c += 32) ss += part[g * gs + c];
    ss = warp_sum(ss);
    if (lane == 0) sums[g] = rsqrtf(ss / (float)gs + eps);
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c4 = threadIdx.x + i * THREADS, c = c4 * 4;
    if (c4 >= nvec) continue;
    const float4 ww = __ldg(reinterpret_cast<const float4*>(w) + c4);
    auto r = [&](int k) { return sums[min((c + k) / gs, groups - 1)]; };
    v[i] = make_float4(v[i].x * r(0) * ww.x, v[i].y * r(1) * ww.y, v[i].z * r(2) * ww.z, v[i].w * r(3) * ww.w);
  }
}

template <int THREADS, int VPT, bool EXT>
__global__ void __launch_bounds__(THREADS) stream_norm_kernel(const StreamNormParams p) {
  pdl_launch_dependents();
  pdl_wait(TL_RMSNORM);
  __shared__ float red[4 * 32];
  extern __shared__ float part[];      // EXT: scratch of the group norms
  const int row = blockIdx.x;
  const int nvec = p.Hp / 4;
  const size_t xo = (size_t)(p.rows ? p.rows[row] : row) * p.ldx;
  float* xr = p.x + xo;
  const float* xi = (EXT && p.x_in) ? p.x_in + xo : xr;
  float4 x[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * THREADS;
    x[i] = c < nvec ? *reinterpret_cast<const float4*>(xi + c * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  if (p.branch) {
    float4 v[VPT];
#pragma unroll
    for (int i = 0; i < VPT; ++i) v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    const int terms = p.branch_rows ? p.branch_top : 1;
    for (int k = 0; k < terms; ++k) {
      const size_t br = p.branch_rows ? (size_t)p.branch_rows[row * p.branch_top + k] : (size_t)row;
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + i * THREADS;
        if (c < nvec) {
          const float4 y = load4(p.branch, br * p.ld_branch + c * 4, p.branch_fp32);
          v[i].x += y.x, v[i].y += y.y, v[i].z += y.z, v[i].w += y.w;
        }
      }
    }
    if (p.branch_rows) {
#pragma unroll
      for (int i = 0; i < VPT; ++i)
        v[i].x *= p.branch_weight, v[i].y *= p.branch_weight, v[i].z *= p.branch_weight, v[i].w *= p.branch_weight;
    }
    if constexpr (EXT) {
      if (p.extra) {
#pragma unroll 4
        for (int k = 0; k < p.extra_top; ++k) {
          const size_t er = (size_t)p.extra_rows[row * p.extra_top + k] * p.ld_extra;
          const float w = p.extra_weights[row * p.extra_top + k];
#pragma unroll
          for (int i = 0; i < VPT; ++i) {
            const int c = threadIdx.x + i * THREADS;
            if (c < nvec) {
              const float4 y = load4(p.extra, er + c * 4, p.extra_fp32);
              v[i].x = fmaf(w, y.x, v[i].x), v[i].y = fmaf(w, y.y, v[i].y);
              v[i].z = fmaf(w, y.z, v[i].z), v[i].w = fmaf(w, y.w, v[i].w);
            }
          }
        }
      }
    }
    if (p.w1) {
      if (EXT && p.groups > 1) group_norm_row<THREADS, VPT>(v, p.w1, p.H, nvec, p.groups, p.eps, part);
      else norm_row<THREADS, VPT>(v, p.w1, p.b1, p.H, nvec, p.eps, p.center, red);
    }
    float* to = (EXT && p.hist) ? p.hist + p.n_hist * p.hist_stride + xo : xr;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * THREADS;
      if (c < nvec) {
        x[i].x += v[i].x, x[i].y += v[i].y, x[i].z += v[i].z, x[i].w += v[i].w;
        *reinterpret_cast<float4*>(to + c * 4) = x[i];
      }
    }
  }
  if constexpr (EXT) {
    if (p.hist) {
      const float own = __ldg(p.mix + p.n_hist);
#pragma unroll
      for (int i = 0; i < VPT; ++i) x[i].x *= own, x[i].y *= own, x[i].z *= own, x[i].w *= own;
#pragma unroll 4
      for (int j = 0; j < p.n_hist; ++j) {
        const float m = __ldg(p.mix + j);
        const float* h = p.hist + j * p.hist_stride + xo;
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
          const int c = threadIdx.x + i * THREADS;
          if (c < nvec) {
            const float4 y = *reinterpret_cast<const float4*>(h + c * 4);
            x[i].x = fmaf(m, y.x, x[i].x), x[i].y = fmaf(m, y.y, x[i].y);
            x[i].z = fmaf(m, y.z, x[i].z), x[i].w = fmaf(m, y.w, x[i].w);
          }
        }
      }
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + i * THREADS;
        if (c < nvec) *reinterpret_cast<float4*>(xr + c * 4) = x[i];
      }
    }
  }
  if (!p.out) return;
  if (p.w2) {
    if (EXT && p.groups > 1) group_norm_row<THREADS, VPT>(x, p.w2, p.H, nvec, p.groups, p.eps, part);
    else norm_row<THREADS, VPT>(x, p.w2, p.b2, p.H, nvec, p.eps, p.center, red + 64);
  }
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * THREADS;
    if (c < nvec) {
      x[i].x *= p.out_scale, x[i].y *= p.out_scale, x[i].z *= p.out_scale, x[i].w *= p.out_scale;
      if (!p.out_rows) {
        store4(p.out, (size_t)row * p.ldo + c * 4, p.out_fp32, x[i]);
      } else {
        for (int k = 0; k < p.out_top; ++k)
          store4(p.out, (size_t)p.out_rows[row * p.out_top + k] * p.ldo + c * 4, p.out_fp32, x[i]);
      }
    }
  }
}

// x[t] = scale * table[ids[t]] as fp32; optional copies of the row in the activation type (out_a / out_b, strides ld_a / ld_b).
// Ids outside [0, vocab) read as a zero row.
__global__ void __launch_bounds__(256) stream_embed_kernel(const long long* __restrict__ ids, const void* table, int table_fp32,
                                                           int vocab, float* x, int ldx, void* out_a, int ld_a, void* out_b,
                                                           int ld_b, int out_fp32, float scale, int T, int Hp) {
  pdl_launch_dependents();
  pdl_wait(TL_EMBED);
  const int nvec = Hp / 4;
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= (long long)T * nvec) return;
  const int t = (int)(idx / nvec), c = (int)(idx % nvec) * 4;
  const long long id = ids[t];
  float4 v = (id >= 0 && id < vocab) ? load4(table, (size_t)id * Hp + c, table_fp32) : make_float4(0.f, 0.f, 0.f, 0.f);
  v.x *= scale, v.y *= scale, v.z *= scale, v.w *= scale;
  *reinterpret_cast<float4*>(x + (size_t)t * ldx + c) = v;
  if (out_a) store4(out_a, (size_t)t * ld_a + c, out_fp32, v);
  if (out_b) store4(out_b, (size_t)t * ld_b + c, out_fp32, v);
}

// Token pair embedding: x[t] = table[id] + pairs[row], row = (previous id * mul_prev + id * mul_cur) mod buckets, or `buckets` at
// the first position of a sequence. Every token files its id in the paged token cache; a sequence's first token of a step finds
// its predecessor there, the others in `ids`.
struct PairEmbedParams {
  const long long* ids;
  const void *table, *pairs;       // [vocab, Hp], [buckets + 1, Hp], both fp32 or bf16
  int fp32, vocab;
  long long mul_prev, mul_cur, buckets;
  const int* positions;
  const long long* slots;          // row of the token cache, < 0: none
  int* tokens;                     // [blocks * block_size]
  const int* block_table;
  int max_blocks, block_size;
  const int* cu_q;                 // [num_seqs + 1] or null (uniform_q tokens each)
  int num_seqs, uniform_q;
  float* x;
  int T, Hp;
};

__global__ void __launch_bounds__(128) stream_embed_pairs_kernel(const PairEmbedParams p) {
  pdl_launch_dependents();
  pdl_wait(TL_EMBED);
  const int t = blockIdx.x, pos = p.positions[t];
  const long long id = p.ids[t];
  long long row = p.buckets;
  if (pos > 0) {
    const int seq = seq_of_token(p.cu_q, p.num_seqs, p.uniform_q, t), q0 = p.cu_q ? p.cu_q[seq] : seq * p.uniform_q;
    long long prev;
    if (t > q0) {
      prev = p.ids[t - 1];
    } else {
      const int page = p.block_table[(size_t)seq * p.max_blocks + (pos - 1) / p.block_size];
      prev = p.tokens[(size_t)page * p.block_size + (pos - 1) % p.block_size];
    }
    row = (prev * p.mul_prev + id * p.mul_cur) % p.buckets;
    if (row < 0) row += p.buckets;
  }
  if (threadIdx.x == 0 && p.slots[t] >= 0) p.tokens[p.slots[t]] = (int)id;
  const bool known = id >= 0 && id < p.vocab;
  for (int c = threadIdx.x * 4; c < p.Hp; c += 512) {
    const float4 a = known ? load4(p.table, (size_t)id * p.Hp + c, p.fp32) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float4 b = load4(p.pairs, (size_t)row * p.Hp + c, p.fp32);
    *reinterpret_cast<float4*>(p.x + (size_t)t * p.Hp + c) = make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w);
  }
}

template <int THREADS, int VPT>
int launch_sn(const StreamNormParams& p, int T, cudaStream_t s) {
  if (p.groups <= 1 && !p.x_in && !p.hist && !p.extra)
    return launch_kernel(stream_norm_kernel<THREADS, VPT, false>, dim3((unsigned)T), dim3(THREADS), 0, s, p);
  size_t smem = 0;
  if (p.groups > 1) smem = (p.H / p.groups) % 128 == 0 ? THREADS / 32 * VPT * sizeof(float) : (size_t)(p.Hp + p.groups) * sizeof(float);
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(stream_norm_kernel<THREADS, VPT, true>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               (int)smem);
    if (e != cudaSuccess) return -(int)e;
  }
  return launch_kernel(stream_norm_kernel<THREADS, VPT, true>, dim3((unsigned)T), dim3(THREADS), smem, s, p);
}

}  // namespace
}  // namespace swb

extern "C" {

// See StreamNormParams. All pointers 16-byte aligned (8 for bf16 rows), strides multiples of 4 elements, Hp a multiple of
// 8 up to 32768, H <= Hp.
int swb_stream_norm(void* x, int ldx, const long long* rows, const void* branch, int ld_branch, int branch_fp32,
                    const int* branch_rows, int branch_top, float branch_weight, const float* w1, const float* b1,
                    const float* w2, const float* b2, void* out, int ldo, int out_fp32, const int* out_rows, int out_top,
                    int T, int H, int Hp, float eps, float out_scale, int center, int groups, const void* x_in, void* hist,
                    long long hist_stride, int n_hist, const float* mix, const void* extra, int ld_extra, int extra_fp32,
                    const int* extra_rows, const float* extra_weights, int extra_top, void* stream) {
  using namespace swb;
  if (T <= 0) return 0;
  if (extra && (!branch || (ld_extra % 4) || !extra_rows || !extra_weights || extra_top <= 0)) return -3;
  if (groups < 1 || H % groups || (groups > 1 && (center || b1 || b2)) || (hist && (!mix || !branch || n_hist < 0 || (hist_stride % 4))) ||
      (rows && (x_in || hist)))
    return -3;
  if (H <= 0 || H > Hp || (Hp % 8) || (ldx % 4) || (branch && (ld_branch % 4)) || (out && (ldo % 4)) || (rows && branch) ||
      (branch_rows && branch_top <= 0) || (out_rows && out_top <= 0))
    return -3;
  StreamNormParams p{};
  p.x = reinterpret_cast<float*>(x);
  p.ldx = ldx;
  p.rows = rows;
  p.branch = branch;
  p.ld_branch = ld_branch;
  p.branch_fp32 = branch_fp32;
  p.branch_rows = branch_rows;
  p.branch_top = branch_top;
  p.branch_weight = branch_weight;
  p.w1 = w1, p.b1 = b1, p.w2 = w2, p.b2 = b2;
  p.out = out;
  p.ldo = ldo;
  p.out_fp32 = out_fp32;
  p.out_rows = out_rows;
  p.out_top = out_top;
  p.H = H, p.Hp = Hp;
  p.eps = eps;
  p.out_scale = out_scale;
  p.center = center;
  p.groups = groups;
  p.x_in = reinterpret_cast<const float*>(x_in);
  p.hist = reinterpret_cast<float*>(hist);
  p.hist_stride = hist_stride;
  p.n_hist = n_hist;
  p.mix = mix;
  p.extra = extra, p.ld_extra = ld_extra, p.extra_fp32 = extra_fp32;
  p.extra_rows = extra_rows, p.extra_weights = extra_weights, p.extra_top = extra_top;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const int nvec = Hp / 4;
  if (nvec <= 128) return launch_sn<128, 1>(p, T, s);
  if (nvec <= 256) return launch_sn<256, 1>(p, T, s);
  if (nvec <= 512) return launch_sn<256, 2>(p, T, s);
  if (nvec <= 1024) return launch_sn<256, 4>(p, T, s);
  if (nvec <= 2048) return launch_sn<512, 4>(p, T, s);
  if (nvec <= 4096) return launch_sn<1024, 4>(p, T, s);
  if (nvec <= 8192) return launch_sn<1024, 8>(p, T, s);
  return -3;
}

int swb_stream_embed(const long long* ids, const void* table, int table_fp32, int vocab, void* x, int ldx, void* out_a,
                     int ld_a, void* out_b, int ld_b, int out_fp32, float scale, int T, int Hp, void* stream) {
  using namespace swb;
  if (T <= 0) return 0;
  if ((Hp % 8) || (ldx % 4) || (out_a && (ld_a % 4)) || (out_b && (ld_b % 4))) return -3;
  const long long n = (long long)T * (Hp / 4);
  return launch_kernel(stream_embed_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0,
                       reinterpret_cast<cudaStream_t>(stream), ids, table, table_fp32, vocab,
                       reinterpret_cast<float*>(x), ldx, out_a, ld_a, out_b, ld_b, out_fp32, scale, T, Hp);
}

// See PairEmbedParams; x [T, Hp] fp32, rows 16-byte aligned, Hp a multiple of 8.
int swb_stream_embed_pairs(const long long* ids, const void* table, const void* pairs, int fp32, int vocab, long long mul_prev,
                           long long mul_cur, long long buckets, const int* positions, const long long* slots, int* tokens,
                           const int* block_table, int max_blocks, int block_size, const int* cu_q, int num_seqs, int uniform_q,
                           float* x, int T, int Hp, void* stream) {
  using namespace swb;
  if (T <= 0) return 0;
  if ((Hp % 8) || buckets < 1 || num_seqs < 1 || block_size < 1 || !tokens || !block_table || !slots || (!cu_q && (long long)num_seqs * uniform_q != T))
    return -3;
  const PairEmbedParams p{ids, table, pairs, fp32, vocab, mul_prev, mul_cur, buckets, positions, slots, tokens, block_table, max_blocks,
                          block_size, cu_q, num_seqs, uniform_q, x, T, Hp};
  return launch_kernel(stream_embed_pairs_kernel, dim3((unsigned)T), dim3(128), 0, reinterpret_cast<cudaStream_t>(stream), p);
}

}  // extern "C"
