// Gated delta rule with a decay per head and key channel, over a flat ragged batch of sequences:
//     S <- g * S          (rows of S are key channels)
//     u  = beta (v - S^T k),   S <- S + k u^T,   o = S^T q
// Three launches around the projections:
//   delta_prep   short causal convolutions with silu, unit q / k, decays, step sizes (a warp per token and head);
//   delta_scan   the recurrence. A column of S (one value channel) never meets the others, so LPC lanes own one column with
//                DPL key channels each in registers; q, k, g stream through shared memory in blocks of tokens. Both dots run
//                on the decayed state, o = (g S)^T q + (k . q) u, so one cross-lane reduction per token is on the critical
//                path. Arithmetic is fp32 in token order: results do not depend on how a prompt was cut.
//   delta_post   RMS norm over a head's value channels, weight and gate; moves the convolution windows on.
// States and windows live in slots; a sequence's state is zero at position 0, a slot below 0 is neither read nor written.
#include "common.cuh"

namespace swb {

SWB_REGISTER_STATUS_UNIT(delta_rule);

namespace {

struct DeltaShape {
  int T, num_seqs, uniform_q;
  const int* cu_q;           // [num_seqs + 1] or null
  const int* positions;      // [T]
  const int* slots;          // [num_seqs]
  int H, G, dim, dp, vdim, vp, taps;   // dp / vp: padded widths
};

struct PrepParams {
  DeltaShape s;
  const void* buf;           // projections [T, ld]: q (G dp) at 0, k, v (H vp), then beta logits at col_b
  int ld, col_b;
  const void* decay;         // [T, ld_decay]: decay logits, H dp
  int ld_decay;
  const float* conv;         // [2 G dp + H vp, taps]
  const void* window;        // [slots, taps - 1, 2 G dp + H vp]
  const float *a_log, *dt_bias;
  float *qk, *kq, *g, *v, *beta;       // [T, G, 2, dp] (k, q), [T, G], [T, H, dp], [T, H, vp], [T, H]
  int tokens_per_cta;
};

__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }

template <typename E>
struct ConvIn {
  const E* buf;
  const E* window;           // of this sequence's slot, or null (no history)
  int ld, C, taps, start, t; // start: flat index of the sequence's first token of this step
  // silu(sum_j w[c, taps - 1 - j] x[t - j])
  __device__ __forceinline__ float operator()(const float* __restrict__ conv, int c) const {
    const float* w = conv + (size_t)c * taps;
    float y = 0.f;
    for (int j = 0; j < taps; ++j) {
      const int r = t - (taps - 1 - j);
      float x = 0.f;
      if (r >= start) x = to_f(buf[(size_t)r * ld + c]);
      else if (window) x = to_f(window[(size_t)(taps - 1 + r - start) * C + c]);
      y = fmaf(w[j], x, y);
    }
    return y * sigmoid_f(y);
  }
};

// Warp task of a token: [0, G) unit q and k of a key head; [G, G + H) decays, step size; [G + H, G + 2 H) values.
template <typename E>
__global__ void __launch_bounds__(256) delta_prep_kernel(const PrepParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const DeltaShape& s = p.s;
  const int task = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (task >= s.G + 2 * s.H) return;
  const int nq = s.G * s.dp, C = 2 * nq + s.H * s.vp;
  const E* buf = reinterpret_cast<const E*>(p.buf);
  for (int i = 0; i < p.tokens_per_cta; ++i) {
    const int t = blockIdx.x * p.tokens_per_cta + i;
    if (t >= s.T) return;
    if (task >= s.G && task < s.G + s.H) {
      const int h = task - s.G;
      const float rate = -expf(p.a_log[h]);
      const E* x = reinterpret_cast<const E*>(p.decay) + (size_t)t * p.ld_decay + h * s.dp;
      float* g = p.g + ((size_t)t * s.H + h) * s.dp;
      for (int c = lane; c < s.dp; c += 32) g[c] = expf(rate * softplus_f(to_f(x[c]) + p.dt_bias[h * s.dp + c]));
      if (lane == 0) p.beta[(size_t)t * s.H + h] = sigmoid_f(to_f(buf[(size_t)t * p.ld + p.col_b + h]));
      continue;
    }
    const int seq = seq_of_token(s.cu_q, s.num_seqs, s.uniform_q, t);
    const int start = s.cu_q ? s.cu_q[seq] : seq * s.uniform_q, slot = s.slots[seq];
    const bool fresh = s.positions[start] == 0 || slot < 0;
    const ConvIn<E> conv{buf, fresh ? nullptr : reinterpret_cast<const E*>(p.window) + (size_t)slot * (s.taps - 1) * C,
                         p.ld, C, s.taps, start, t};
    if (task < s.G) {
      float kk = 0.f, qq = 0.f, kq = 0.f;
      float kv[16], qv[16];            // dp <= 512
#pragma unroll
      for (int j = 0; j < 16; ++j) {
        const int c = lane + j * 32;
        kv[j] = qv[j] = 0.f;
        if (c < s.dp) {
          qv[j] = conv(p.conv, task * s.dp + c);
          kv[j] = conv(p.conv, nq + task * s.dp + c);
        }
        qq = fmaf(qv[j], qv[j], qq);
        kk = fmaf(kv[j], kv[j], kk);
        kq = fmaf(kv[j], qv[j], kq);
      }
      qq = warp_sum(qq), kk = warp_sum(kk), kq = warp_sum(kq);
      const float rk = rsqrtf(kk + 1e-6f), rq = rsqrtf(qq + 1e-6f) * rsqrtf((float)s.dim);
      float* out = p.qk + ((size_t)t * s.G + task) * 2 * s.dp;
#pragma unroll
      for (int j = 0; j < 16; ++j) {
        const int c = lane + j * 32;
        if (c < s.dp) out[c] = kv[j] * rk, out[s.dp + c] = qv[j] * rq;
      }
      if (lane == 0) p.kq[(size_t)t * s.G + task] = kq * rk * rq;
    } else {
      const int h = task - s.G - s.H;
      float* out = p.v + ((size_t)t * s.H + h) * s.vp;
      for (int c = lane; c < s.vp; c += 32) out[c] = conv(p.conv, 2 * nq + h * s.vp + c);
    }
  }
}

struct ScanParams {
  DeltaShape s;
  const float *qk, *kq, *g, *v, *beta;
  float* state;              // [slots, H, vp, dp]
  float* o;                  // [T, H, vp]
};

__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t dup2(float x) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %1};" : "=l"(d) : "f"(x));
  return d;
}
__device__ __forceinline__ float sum2(uint64_t a) {
  float x, y;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(a));
  return x + y;
}
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async4(void* dst, const void* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

constexpr int SCAN_WARPS = 4;

// TB tokens per staged block; layout of one token in shared memory: k [dp], q [dp], g [dp], v [COLS], (kq, beta, -, -)
template <int DPL, int LPC, int TB>
__global__ void __launch_bounds__(SCAN_WARPS * 32) delta_scan_kernel(const ScanParams p) {
  constexpr int DP = DPL * LPC, COLS = SCAN_WARPS * 32 / LPC, TOK = 3 * DP + COLS + 4, N2 = DPL / 2;
  extern __shared__ __align__(16) float sm[];        // 2 blocks of TB tokens
  pdl_launch_dependents();
  pdl_wait();
  const DeltaShape& s = p.s;
  const int seq = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * COLS, kvh = h / (s.H / s.G);
  const int tid = threadIdx.x, sub = tid % LPC, lc = tid / LPC, col = c0 + lc;
  const int start = s.cu_q ? s.cu_q[seq] : seq * s.uniform_q, n = s.cu_q ? s.cu_q[seq + 1] - start : s.uniform_q;
  if (n <= 0) return;
  const int slot = s.slots[seq];
  const bool live = col < s.vp;
  float* st = p.state + (((size_t)max(slot, 0) * s.H + h) * s.vp + (live ? col : 0)) * DP;
  uint64_t S[N2];
  if (slot >= 0 && live && s.positions[start] != 0) {
#pragma unroll
    for (int i = 0; i < DPL / 4; ++i) {
      const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(st + (i * LPC + sub) * 4);
      S[2 * i] = v.x, S[2 * i + 1] = v.y;
    }
  } else {
#pragma unroll
    for (int i = 0; i < N2; ++i) S[i] = 0ull;
  }
  const int ncols = min(COLS, s.vp - c0);            // vp % 8 == 0, so whole 16-byte pieces
  auto stage = [&](int b) {
    float* dst0 = sm + (b & 1) * TB * TOK;
    const int t0 = b * TB, m = min(TB, n - t0);
    for (int i = tid; i < m * (DP / 4); i += SCAN_WARPS * 32) {
      const int r = i / (DP / 4), c = (i % (DP / 4)) * 4;
      const size_t t = start + t0 + r;
      const float* qk = p.qk + (t * s.G + kvh) * 2 * DP + c;
      float* d = dst0 + r * TOK + c;
      cp_async16(d, qk);
      cp_async16(d + DP, qk + DP);
      cp_async16(d + 2 * DP, p.g + (t * s.H + h) * DP + c);
    }
    for (int i = tid; i < m * (COLS / 4); i += SCAN_WARPS * 32) {
      const int r = i / (COLS / 4), c = (i % (COLS / 4)) * 4;
      if (c < ncols) cp_async16(dst0 + r * TOK + 3 * DP + c, p.v + ((size_t)(start + t0 + r) * s.H + h) * s.vp + c0 + c);
    }
    for (int r = tid; r < m; r += SCAN_WARPS * 32) {
      cp_async4(dst0 + r * TOK + 3 * DP + COLS, p.kq + (size_t)(start + t0 + r) * s.G + kvh);
      cp_async4(dst0 + r * TOK + 3 * DP + COLS + 1, p.beta + (size_t)(start + t0 + r) * s.H + h);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const int blocks = (n + TB - 1) / TB;
  stage(0);
  float* orow = p.o + ((size_t)start * s.H + h) * s.vp + col;
  for (int b = 0; b < blocks; ++b) {
    if (b + 1 < blocks) {
      stage(b + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const float* tok = sm + (b & 1) * TB * TOK;
    const int m = min(TB, n - b * TB);
    for (int r = 0; r < m; ++r, tok += TOK, orow += (size_t)s.H * s.vp) {
      const ulonglong2* k4 = reinterpret_cast<const ulonglong2*>(tok);
      const ulonglong2* q4 = reinterpret_cast<const ulonglong2*>(tok + DP);
      const ulonglong2* g4 = reinterpret_cast<const ulonglong2*>(tok + 2 * DP);
      uint64_t ak[2] = {0ull, 0ull}, aq[2] = {0ull, 0ull}, kk[N2];
#pragma unroll
      for (int i = 0; i < DPL / 4; ++i) {
        const ulonglong2 g = g4[i * LPC + sub], k = k4[i * LPC + sub], q = q4[i * LPC + sub];
        S[2 * i] = mul2(S[2 * i], g.x);
        S[2 * i + 1] = mul2(S[2 * i + 1], g.y);
        ak[0] = fma2(S[2 * i], k.x, ak[0]);
        ak[1] = fma2(S[2 * i + 1], k.y, ak[1]);
        aq[0] = fma2(S[2 * i], q.x, aq[0]);
        aq[1] = fma2(S[2 * i + 1], q.y, aq[1]);
        kk[2 * i] = k.x, kk[2 * i + 1] = k.y;
      }
      float dk = sum2(ak[0]) + sum2(ak[1]), dq = sum2(aq[0]) + sum2(aq[1]);
#pragma unroll
      for (int o = 1; o < LPC; o <<= 1) {
        dk += __shfl_xor_sync(0xffffffffu, dk, o);
        dq += __shfl_xor_sync(0xffffffffu, dq, o);
      }
      const float u = tok[3 * DP + COLS + 1] * (tok[3 * DP + lc] - dk);
      const uint64_t uu = dup2(u);
#pragma unroll
      for (int i = 0; i < N2; ++i) S[i] = fma2(kk[i], uu, S[i]);
      if (sub == 0 && live) *orow = fmaf(tok[3 * DP + COLS], u, dq);
    }
    __syncthreads();
  }
  if (slot >= 0 && live) {
#pragma unroll
    for (int i = 0; i < DPL / 4; ++i)
      *reinterpret_cast<ulonglong2*>(st + (i * LPC + sub) * 4) = make_ulonglong2(S[2 * i], S[2 * i + 1]);
  }
}

struct PostParams {
  DeltaShape s;
  const float* o;            // [T, H, vp]
  const void* gate;          // [T, ld_gate]: gate logits, H vp
  int ld_gate;
  const float* w;            // [vp]
  float eps;
  void* out;                 // [T, H vp]
  const void* buf;           // projections, for the windows
  int ld;
  void* window;
  int norm_ctas;
};

template <typename E>
__global__ void __launch_bounds__(256) delta_post_kernel(const PostParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const DeltaShape& s = p.s;
  if ((int)blockIdx.x >= p.norm_ctas) {              // one CTA per sequence and 1024 channels: the last taps - 1 inputs
    const int C = 2 * s.G * s.dp + s.H * s.vp, pieces = (C + 1023) / 1024;
    const int id = blockIdx.x - p.norm_ctas, seq = id / pieces;
    const int start = s.cu_q ? s.cu_q[seq] : seq * s.uniform_q, n = s.cu_q ? s.cu_q[seq + 1] - start : s.uniform_q;
    const int slot = s.slots[seq], keep = s.taps - 1;
    if (slot < 0 || n <= 0) return;
    const bool fresh = s.positions[start] == 0;
    E* win = reinterpret_cast<E*>(p.window) + (size_t)slot * keep * C;
    for (int c = id % pieces * 1024 + threadIdx.x; c < min(C, (id % pieces + 1) * 1024); c += 256)
      for (int j = 0; j < keep; ++j) {               // ascending: an old entry is read before it is overwritten
        const int r = n - keep + j;
        E x;
        from_f(x, 0.f);
        if (r >= 0) x = reinterpret_cast<const E*>(p.buf)[(size_t)(start + r) * p.ld + c];
        else if (!fresh) x = win[(size_t)(j + n) * C + c];
        win[(size_t)j * C + c] = x;
      }
    return;
  }
  const long long id = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (id >= (long long)s.T * s.H) return;
  const int t = (int)(id / s.H), h = (int)(id % s.H);
  const float* o = p.o + id * s.vp;
  float ss = 0.f;
  for (int c = lane; c < s.vp; c += 32) ss = fmaf(o[c], o[c], ss);      // padding columns are zero
  const float r = rsqrtf(warp_sum(ss) / (float)s.vdim + p.eps);
  const E* gate = reinterpret_cast<const E*>(p.gate) + (size_t)t * p.ld_gate + h * s.vp;
  E* out = reinterpret_cast<E*>(p.out) + id * s.vp;
  for (int c = lane; c < s.vp; c += 32) from_f(out[c], o[c] * r * p.w[c] * sigmoid_f(to_f(gate[c])));
}

template <int DPL, int LPC, int TB>
int launch_scan(const ScanParams& p, cudaStream_t st) {
  constexpr int DP = DPL * LPC, COLS = SCAN_WARPS * 32 / LPC;
  constexpr size_t smem = 2 * TB * (3 * DP + COLS + 4) * sizeof(float);
  if (smem > 48 * 1024) {
    static bool configured[64] = {false};
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev < 0 || dev >= 64 || !configured[dev]) {
      const cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<DPL, LPC, TB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return -(int)e;
      if (dev >= 0 && dev < 64) configured[dev] = true;
    }
  }
  return launch_kernel(delta_scan_kernel<DPL, LPC, TB>, dim3((p.s.vp + COLS - 1) / COLS, p.s.H, p.s.num_seqs), dim3(SCAN_WARPS * 32),
                       smem, st, p);
}

bool shape_ok(const DeltaShape& s) {
  return s.T > 0 && s.num_seqs > 0 && s.H > 0 && s.G > 0 && s.H % s.G == 0 && s.dim > 0 && s.dim <= s.dp && s.dp % 32 == 0 &&
         s.dp <= 512 && s.vdim > 0 && s.vdim <= s.vp && s.vp % 8 == 0 && s.taps >= 1 && s.positions && s.slots &&
         (s.cu_q || (long long)s.num_seqs * s.uniform_q == s.T);
}

DeltaShape make_shape(const int* dims, const int* cu_q, const int* positions, const int* slots) {
  // dims: T, num_seqs, uniform_q, H, G, dim, dp, vdim, vp, taps
  return DeltaShape{dims[0], dims[1], dims[2], cu_q, positions, slots, dims[3], dims[4], dims[5], dims[6], dims[7], dims[8], dims[9]};
}

}  // namespace
}  // namespace swb

extern "C" {

// dims: host int[10] = T, num_seqs, uniform_q (cu_q null), H, G, dim, dp, vdim, vp, taps. fp32 selects the element type of
// the projections, windows and decay logits.
int swb_delta_prep(const int* dims, const int* cu_q, const int* positions, const int* slots, const void* buf, int ld, int col_b,
                   const void* decay, int ld_decay, const float* conv, const void* window, const float* a_log, const float* dt_bias,
                   float* qk, float* kq, float* g, float* v, float* beta, int fp32, void* stream) {
  using namespace swb;
  PrepParams p{make_shape(dims, cu_q, positions, slots), buf, ld, col_b, decay, ld_decay, conv, window, a_log, dt_bias, qk, kq, g, v,
               beta, dims[0] >= 2048 ? 8 : 1};
  if (dims[0] <= 0) return 0;
  if (!shape_ok(p.s)) return -3;
  const dim3 grid((p.s.T + p.tokens_per_cta - 1) / p.tokens_per_cta, (p.s.G + 2 * p.s.H + 7) / 8);
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return fp32 ? launch_kernel(delta_prep_kernel<float>, grid, dim3(256), 0, st, p)
              : launch_kernel(delta_prep_kernel<bf16>, grid, dim3(256), 0, st, p);
}

int swb_delta_scan(const int* dims, const int* cu_q, const int* positions, const int* slots, const float* qk, const float* kq,
                   const float* g, const float* v, const float* beta, float* state, float* o, void* stream) {
  using namespace swb;
  ScanParams p{make_shape(dims, cu_q, positions, slots), qk, kq, g, v, beta, state, o};
  if (dims[0] <= 0) return 0;
  if (!shape_ok(p.s)) return -3;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  switch (p.s.dp) {
    case 32: return launch_scan<8, 4, 16>(p, st);
    case 64: return launch_scan<16, 4, 16>(p, st);
    case 96: return launch_scan<24, 4, 16>(p, st);
    case 128: return launch_scan<32, 4, 16>(p, st);
    case 192: return launch_scan<24, 8, 8>(p, st);
    case 256: return launch_scan<32, 8, 8>(p, st);
    case 512: return launch_scan<32, 16, 4>(p, st);
    default: return -3;
  }
}

int swb_delta_post(const int* dims, const int* cu_q, const int* positions, const int* slots, const float* o, const void* gate,
                   int ld_gate, const float* w, float eps, void* out, const void* buf, int ld, void* window, int fp32, void* stream) {
  using namespace swb;
  PostParams p{make_shape(dims, cu_q, positions, slots), o, gate, ld_gate, w, eps, out, buf, ld, window, 0};
  if (dims[0] <= 0) return 0;
  if (!shape_ok(p.s)) return -3;
  p.norm_ctas = (int)(((long long)p.s.T * p.s.H + 7) / 8);
  const int C = 2 * p.s.G * p.s.dp + p.s.H * p.s.vp;
  const dim3 grid(p.norm_ctas + (p.s.taps > 1 ? p.s.num_seqs * ((C + 1023) / 1024) : 0));
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return fp32 ? launch_kernel(delta_post_kernel<float>, grid, dim3(256), 0, st, p)
              : launch_kernel(delta_post_kernel<bf16>, grid, dim3(256), 0, st, p);
}

}  // extern "C"
