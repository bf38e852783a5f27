// 32-bit mode and unrestricted shapes: an fp32 GEMM (dense or grouped rows) and a paged attention kernel for any head
// widths, both on the ordinary FMA pipes with true fp32 products. They serve models that run in float32 (numerical
// checks), and the attention kernel also serves bf16 models whose head widths the tensor-core kernels do not cover.
#include "common.cuh"
#include "gemm_tcgen05.cuh"

namespace swb {

SWB_REGISTER_STATUS_UNIT(f32_ops);

namespace {

constexpr int TM = 64, TN = 64, TK = 16;

// out[r, n] = act(sum_k a[src ? src[r] : r, k] w[e, n, k] + bias[n]); 64 x 64 tile, 4 x 4 per thread. Grouped: blockIdx.z = expert.
__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ a, int lda, const int* __restrict__ src,
                                                       const int* __restrict__ offsets, const float* __restrict__ w, int ldw,
                                                       float* out, int ldo, int T, int N, int K, int act, float act_a, float act_b,
                                                       const float* __restrict__ bias) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float sa[TK][TM + 4], sw[TK][TN + 4];
  const int lo = offsets ? offsets[blockIdx.z] : 0, hi = offsets ? offsets[blockIdx.z + 1] : T;
  const int r0 = lo + blockIdx.y * TM, n0 = blockIdx.x * TN;
  if (r0 >= hi) return;
  const float* we = w + (size_t)blockIdx.z * N * ldw;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;   // 64 rows x 16 columns, four per thread
  const int arow = r0 + lr;
  const float* ap = arow < hi ? a + (size_t)(src ? src[arow] : arow) * lda : nullptr;
  const float* wp = n0 + lr < N ? we + (size_t)(n0 + lr) * ldw : nullptr;
  for (int k0 = 0; k0 < K; k0 += TK) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int k = k0 + lk + j;
      sa[lk + j][lr] = (ap && k < K) ? ap[k] : 0.f;
      sw[lk + j][lr] = (wp && k < K) ? wp[k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < TK; ++k) {
      float x[4], y[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) x[i] = sa[k][ty * 4 + i], y[i] = sw[k][tx * 4 + i];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], y[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = r0 + ty * 4 + i;
    if (r >= hi) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= N) continue;
      float v = acc[i][j];
      if (bias) v += bias[n];
      if (act == SWB_ACT_RELU2) v = relu2_f(v);
      else if (act == SWB_ACT_SILU) v = silu_f(v);
      else if (act == SWB_ACT_GELU_TANH) v = gelu_tanh_f(v);
      else if (act == SWB_ACT_XIELU) v = xielu_exact_f(v, act_a, act_b);
      out[(size_t)r * ldo + n] = v;
    }
  }
}

constexpr int AW = 4;          // warps per CTA: keys are dealt out to them
constexpr int MAX_PER_LANE = 32;   // head widths up to 1024

// What a query sees and how its scores are formed, beyond scale and causality.
struct SimpleAttnParams {
  long long q_stride_tok, out_stride_tok;
  const int* block_table;
  int max_blocks, block_size;
  const int *cu_q, *kv_lens;
  int num_seqs, uniform_q, Hq, Hkv, D, Dv;
  int k_row, v_row;          // elements between the key / value rows of consecutive tokens of a page
  float scale;
  int chunk;                 // > 0: only keys of the query's own run of `chunk` positions
  int window;                // > 0: only the last `window` keys, the query's own included
  float softcap;             // > 0: score <- softcap tanh(score / softcap)
  const float* q_temp;       // optional, by position: factor of the scores in front of the cap
  const float* sink;
  int maps;                  // query heads h, h + 1, ... take turns on `maps` key parts of D columns each within a key row
  int v_heads;               // > 0: every query head is applied to all value heads; out [token, Hq, v_heads, Dv]
  const void* gate;          // optional logits in the layout of a token's output, rows gate_stride apart: out is scaled by their sigmoid
  long long gate_stride;
};

// One CTA per (query token, head) or, with v_heads, (query token, head, value head). Each warp runs an online softmax over its share of the visible keys; lanes split the
// head dimension. The sink joins the denominator when the four partial results are merged.
template <typename E, int PL>
__global__ void __launch_bounds__(AW * 32) attn_simple_kernel(const E* __restrict__ q, const E* __restrict__ kc, const E* __restrict__ vc,
                                                              E* out, const SimpleAttnParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, nv = p.v_heads > 0 ? p.v_heads : 1, head = blockIdx.y / nv, kvh = head / (p.Hq / p.Hkv);
  const int v_rows = p.v_heads > 0 ? nv : p.Hkv, vh = p.v_heads > 0 ? blockIdx.y % nv : kvh;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seq = seq_of_token(p.cu_q, p.num_seqs, p.uniform_q, t);
  const int q0 = p.cu_q ? p.cu_q[seq] : seq * p.uniform_q, q_len = p.cu_q ? p.cu_q[seq + 1] - q0 : p.uniform_q;
  const int pos = p.kv_lens[seq] - q_len + (t - q0);
  int first = p.chunk > 0 ? pos / p.chunk * p.chunk : 0;
  if (p.window > 0) first = max(first, pos - p.window + 1);
  const int* table = p.block_table + (size_t)seq * p.max_blocks;
  const E* qr = q + (size_t)t * p.q_stride_tok + (size_t)head * p.D;
  const float scale = p.scale * (p.q_temp ? p.q_temp[pos] : 1.f);
  const int k_off = p.maps > 1 ? head % p.maps * p.D : 0;
  float qv[PL], o[PL];
#pragma unroll
  for (int i = 0; i < PL; ++i) {
    const int d = lane + i * 32;
    qv[i] = d < p.D ? to_f(qr[d]) : 0.f;
    o[i] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  for (int j = first + warp; j <= pos; j += AW) {
    const size_t page = table[j / p.block_size], at = j % p.block_size;
    const E* kr = kc + ((page * p.Hkv + kvh) * p.block_size + at) * p.k_row + k_off;
    const E* vr = vc + ((page * v_rows + vh) * p.block_size + at) * p.v_row;
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < PL; ++i) {
      const int d = lane + i * 32;
      if (d < p.D) s = fmaf(qv[i], to_f(kr[d]), s);
    }
    s = warp_sum(s) * scale;
    if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
    const float mn = fmaxf(m, s), f = expf(m - mn), e = expf(s - mn);
    l = l * f + e;
    m = mn;
#pragma unroll
    for (int i = 0; i < PL; ++i) {
      const int d = lane + i * 32;
      if (d < p.Dv) o[i] = fmaf(e, to_f(vr[d]), o[i] * f);
    }
  }
  __shared__ float so[AW][32 * PL], sm[AW], sl[AW];
#pragma unroll
  for (int i = 0; i < PL; ++i) so[warp][lane + i * 32] = o[i];
  if (lane == 0) sm[warp] = m, sl[warp] = l;
  __syncthreads();
  float top = p.sink ? p.sink[head] : -INFINITY;
  for (int w = 0; w < AW; ++w) top = fmaxf(top, sm[w]);
  float den = p.sink ? expf(p.sink[head] - top) : 0.f;
  for (int w = 0; w < AW; ++w) den += sl[w] * expf(sm[w] - top);
  for (int d = threadIdx.x; d < p.Dv; d += AW * 32) {
    float v = 0.f;
    for (int w = 0; w < AW; ++w) v = fmaf(so[w][d], expf(sm[w] - top), v);
    const size_t col = (size_t)blockIdx.y * p.Dv + d;
    v /= den;
    if (p.gate) v /= 1.f + expf(-to_f(reinterpret_cast<const E*>(p.gate)[t * p.gate_stride + col]));
    from_f(out[(size_t)t * p.out_stride_tok + col], v);
  }
}

// out[t, h, n] = sigmoid(gate[t, h]) * sum_k a[t, h, k] w[h, n, k] with free strides of w, for 8 tokens per CTA (gate optional).
constexpr int HP_T = 8, HP_K = 128;
template <typename E>
__global__ void __launch_bounds__(64) head_product_kernel(const E* __restrict__ a, long long a_tok, int a_head,
                                                          const E* __restrict__ w, long long w_head, int w_n, int w_k, E* out,
                                                          long long out_tok, int out_head, const E* gate, long long gate_tok, int T,
                                                          int N, int K) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float sa[HP_T][HP_K];
  const int n = blockIdx.x * 64 + threadIdx.x, h = blockIdx.y, t0 = blockIdx.z * HP_T;
  const E* wr = w + h * w_head + (long long)min(n, N - 1) * w_n;
  float acc[HP_T] = {};
  for (int k0 = 0; k0 < K; k0 += HP_K) {
    __syncthreads();
    for (int i = threadIdx.x; i < HP_T * HP_K; i += 64) {
      const int r = i / HP_K, k = i % HP_K;
      sa[r][k] = (t0 + r < T && k0 + k < K) ? to_f(a[(t0 + r) * a_tok + (long long)h * a_head + k0 + k]) : 0.f;
    }
    __syncthreads();
    const int m = min(HP_K, K - k0);
    for (int k = 0; k < m; ++k) {
      const float x = to_f(wr[(long long)(k0 + k) * w_k]);
#pragma unroll
      for (int r = 0; r < HP_T; ++r) acc[r] = fmaf(x, sa[r][k], acc[r]);
    }
  }
  if (n >= N) return;
#pragma unroll
  for (int r = 0; r < HP_T; ++r) {
    if (t0 + r >= T) break;
    float v = acc[r];
    if (gate) v /= 1.f + expf(-to_f(gate[(t0 + r) * gate_tok + h]));
    from_f(out[(t0 + r) * out_tok + (long long)h * out_head + n], v);
  }
}

template <typename E>
int launch_attn_simple(const void* q, const void* k, const void* v, void* out, const SimpleAttnParams& p, int total_tokens, cudaStream_t s) {
  const dim3 grid((unsigned)total_tokens, p.Hq * (p.v_heads > 0 ? p.v_heads : 1)), block(AW * 32);
  auto go = [&](auto kernel) {
    return launch_kernel(kernel, grid, block, 0, s, reinterpret_cast<const E*>(q), reinterpret_cast<const E*>(k), reinterpret_cast<const E*>(v),
                         reinterpret_cast<E*>(out), p);
  };
  const int widest = max(p.D, p.Dv);
  if (widest <= 128) return go(attn_simple_kernel<E, 4>);
  if (widest <= 320) return go(attn_simple_kernel<E, 10>);
  if (widest <= 640) return go(attn_simple_kernel<E, 20>);
  return go(attn_simple_kernel<E, MAX_PER_LANE>);
}

}  // namespace
}  // namespace swb

extern "C" {

// fp32 GEMM without reduced-precision modes. Dense: offsets null, groups 1. Grouped: w [groups, N, ldw], rows of group g
// are [offsets[g], offsets[g + 1]), at most T rows in all; src (nullable) names the row of `a` for each row.
int swb_gemm_f32(const float* a, int lda, const int* src, const int* offsets, int groups, const float* w, int ldw, float* out,
                 int ldo, int T, int N, int K, int act, float act_a, float act_b, const float* bias, void* stream) {
  using namespace swb;
  if (T <= 0 || N <= 0 || K <= 0) return 0;
  if (groups < 1 || (bias && offsets) || (groups > 1 && !offsets) || gemm_act_pairs(act)) return -3;
  return launch_kernel(gemm_f32_kernel, dim3((N + TN - 1) / TN, (T + TM - 1) / TM, groups), dim3(256), 0,
                       reinterpret_cast<cudaStream_t>(stream), a, lda, src, offsets, w, ldw, out, ldo, T, N, K, act, act_a, act_b, bias);
}

// Paged attention for any head widths up to 1024 in fp32 arithmetic; elements fp32 or bf16 (fp32 flag). Arguments as in
// swb_attn_ext and SimpleAttnParams; causal, sequences from cu_q or uniform lengths of uniform_q tokens. v_row: elements between the
// value rows of consecutive tokens of a page (0: Dv), so that values may be the leading columns of wider rows. Key rows are maps * D
// wide (D up to 1024 each).
int swb_attn_simple(const void* q, long long q_stride_tok, const void* k, const void* v, void* out, long long out_stride_tok,
                    const int* block_table, int max_blocks, int block_size, const int* cu_q, const int* kv_lens, int num_seqs,
                    int uniform_q, int total_tokens, int Hq, int Hkv, int D, int Dv, int v_row, float scale, int chunk,
                    const float* sink, int window, float softcap, const float* q_temp, int maps, int v_heads, const void* gate,
                    long long gate_stride, int fp32, void* stream) {
  using namespace swb;
  if (total_tokens <= 0 || num_seqs <= 0) return 0;
  if (Hkv <= 0 || Hq % Hkv || D < 1 || Dv < 1 || D > 32 * MAX_PER_LANE || Dv > 32 * MAX_PER_LANE || block_size <= 0 ||
      !block_table || !kv_lens || chunk < 0 || window < 0 || softcap < 0.f || maps < 1 || v_heads < 0 || (maps > 1 && v_heads) || (Hq / Hkv) % maps ||
      (!cu_q && (uniform_q <= 0 || num_seqs * uniform_q != total_tokens)) || (v_row && v_row < Dv))
    return -3;
  const SimpleAttnParams p{q_stride_tok, out_stride_tok, block_table, max_blocks, block_size, cu_q, kv_lens, num_seqs, uniform_q, Hq, Hkv, D, Dv,
                           maps * D, v_row ? v_row : Dv, scale, chunk, window, softcap, q_temp, sink, maps, v_heads, gate, gate_stride};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return fp32 ? launch_attn_simple<float>(q, k, v, out, p, total_tokens, s) : launch_attn_simple<bf16>(q, k, v, out, p, total_tokens, s);
}

// Per-head products of any sizes and strides (elements): out[t, h, n] = sigmoid(gate[t, h]) sum_k a[t, h, k] w[h, n, k].
int swb_head_product_simple(const void* a, long long a_tok, int a_head, const void* w, long long w_head, int w_n, int w_k, void* out,
                            long long out_tok, int out_head, const void* gate, long long gate_tok, int T, int H, int N, int K, int fp32,
                            void* stream) {
  using namespace swb;
  if (T <= 0 || H <= 0 || N <= 0 || K <= 0) return 0;
  const dim3 grid((N + 63) / 64, H, (T + HP_T - 1) / HP_T), block(64);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (fp32)
    return launch_kernel(head_product_kernel<float>, grid, block, 0, s, reinterpret_cast<const float*>(a), a_tok, a_head,
                         reinterpret_cast<const float*>(w), w_head, w_n, w_k, reinterpret_cast<float*>(out), out_tok, out_head,
                         reinterpret_cast<const float*>(gate), gate_tok, T, N, K);
  return launch_kernel(head_product_kernel<bf16>, grid, block, 0, s, reinterpret_cast<const bf16*>(a), a_tok, a_head,
                       reinterpret_cast<const bf16*>(w), w_head, w_n, w_k, reinterpret_cast<bf16*>(out), out_tok, out_head,
                       reinterpret_cast<const bf16*>(gate), gate_tok, T, N, K);
}

}  // extern "C"
