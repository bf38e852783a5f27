// Gated delta rule with a decay per head and key channel, or one per head, over a flat ragged batch of sequences:
//     S <- g * S          (rows of S are key channels)
//     u  = beta (v - S^T k),   S <- S + k u^T,   o = S^T q
// Three launches around the projections:
//   delta_prep   short causal convolutions with silu, unit q / k, decays, step sizes. A warp takes one head of one token, the
//                warps of a CTA consecutive tokens, so that all but one of a convolution's rows come from L1;
//   delta_scan   the recurrence. A column of S (one value channel) never meets the others: sixteen lanes own NC columns, DPL key
//                channels of each in registers, so that every q, k, g value read from shared memory serves NC columns (reading
//                them is what bounds the kernel otherwise). Both dots run on the decayed state, o = (g S)^T q + (k . q) u, so one
//                cross-lane reduction per token is on the critical path; it folds the 2 NC sums into different lanes on the way.
//                Arithmetic is fp32 in token order: results do not depend on how a prompt was cut.
//   delta_post   RMS norm over a head's value channels, weight and gate; moves the convolution windows on.
// With one decay per head the dots run on the state as it is, a factor g behind them, and the decay joins the update.
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
  int head_decay;            // 1: one decay per head
};

struct PrepParams {
  DeltaShape s;
  const void* buf;           // projections [T, ld]: q (G dp) at 0, k, v (H vp), then beta logits at col_b
  int ld, col_b;
  const void* decay;         // [T, ld_decay]: decay logits, H dp (H with one per head, as are dt_bias and g)
  int ld_decay;
  const float* conv;         // [taps, 2 G dp + H vp]
  const void* window;        // [slots, taps - 1, 2 G dp + H vp]
  const float *a_log, *dt_bias;
  float *qk, *kq, *g, *v, *beta;       // [T, G, 2, dp] (k, q), [T, G], [T, H, dp], [T, H, vp], [T, H]
  int heads_per_cta;
};

__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
// for activations and output gates, which do not enter the recurrence as they are
__device__ __forceinline__ float fast_sigmoid(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }

// Four channels of the convolution at token t: silu(sum_j w[taps - 1 - j] x[t - j]). TAPS 0: any number of taps.
template <typename E, int TAPS>
struct Conv {
  const E *buf, *window;     // window: of this sequence's slot, or null (no history)
  const float* w;            // [taps, C]
  int ld, C, taps, start, t;

  __device__ __forceinline__ float4 operator()(int c) const {
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
    auto input = [&](int r) {
      if (r >= start) return load_row4(buf + (size_t)r * ld + c);
      if (window) return load_row4(window + (size_t)(taps - 1 + r - start) * C + c);
      return make_float4(0.f, 0.f, 0.f, 0.f);
    };
    auto mac = [&](int j, float4 x) {
      const float4 b = __ldg(reinterpret_cast<const float4*>(w + (size_t)j * C + c));
      y.x = fmaf(x.x, b.x, y.x), y.y = fmaf(x.y, b.y, y.y), y.z = fmaf(x.z, b.z, y.z), y.w = fmaf(x.w, b.w, y.w);
    };
    if constexpr (TAPS > 0) {
      float4 x[TAPS];
#pragma unroll
      for (int j = 0; j < TAPS; ++j) x[j] = input(t - (TAPS - 1) + j);
#pragma unroll
      for (int j = 0; j < TAPS; ++j) mac(j, x[j]);
    } else {
      for (int j = 0; j < taps; ++j) mac(j, input(t - (taps - 1) + j));
    }
    y.x *= fast_sigmoid(y.x), y.y *= fast_sigmoid(y.y), y.z *= fast_sigmoid(y.z), y.w *= fast_sigmoid(y.w);
    return y;
  }
};

__device__ __forceinline__ float dot4(float4 a, float4 b) { return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, a.w * b.w))); }
__device__ __forceinline__ float4 scale4(float4 a, float r) { return make_float4(a.x * r, a.y * r, a.z * r, a.w * r); }

// Tasks of a token: [0, G) unit q and k of a key head; [G, G + H) decays and step size of a head; [G + H, G + 2 H) its values.
// blockIdx.y takes heads_per_cta of them. NI: 128-channel pieces of a key head.
template <typename E, int TAPS, int NI>
__global__ void __launch_bounds__(256) delta_prep_kernel(const PrepParams p) {
  pdl_wait();
  const DeltaShape& s = p.s;
  const int t = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int nq = s.G * s.dp, C = 2 * nq + s.H * s.vp;
  const E* buf = reinterpret_cast<const E*>(p.buf);
  if (t >= s.T) return;
  const int seq = seq_of_token(s.cu_q, s.num_seqs, s.uniform_q, t);
  const int start = s.cu_q ? s.cu_q[seq] : seq * s.uniform_q, slot = s.slots[seq];
  const E* window = s.positions[start] == 0 || slot < 0 ? nullptr
                                                         : reinterpret_cast<const E*>(p.window) + (size_t)slot * (s.taps - 1) * C;
  const Conv<E, TAPS> conv{buf, window, p.conv, p.ld, C, s.taps, start, t};
  const float q_scale = rsqrtf((float)s.dim);
  const int first = blockIdx.y * p.heads_per_cta, last = min(first + p.heads_per_cta, s.G + 2 * s.H);
#pragma unroll 1
  for (int task = first; task < last; ++task) {
    if (task < s.G) {
      float4 q[NI], k[NI];
      float qq = 0.f, kk = 0.f, kq = 0.f;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int c = lane * 4 + i * 128;
        q[i] = k[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < s.dp) q[i] = conv(task * s.dp + c), k[i] = conv(nq + task * s.dp + c);
        qq += dot4(q[i], q[i]), kk += dot4(k[i], k[i]), kq += dot4(k[i], q[i]);
      }
      qq = warp_sum(qq), kk = warp_sum(kk), kq = warp_sum(kq);
      const float rk = rsqrtf(kk + 1e-6f), rq = rsqrtf(qq + 1e-6f) * q_scale;
      float* out = p.qk + ((size_t)t * s.G + task) * 2 * s.dp;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int c = lane * 4 + i * 128;
        if (c >= s.dp) continue;
        *reinterpret_cast<float4*>(out + c) = scale4(k[i], rk);
        *reinterpret_cast<float4*>(out + s.dp + c) = scale4(q[i], rq);
      }
      if (lane == 0) p.kq[(size_t)t * s.G + task] = kq * rk * rq;
    } else if (task < s.G + s.H) {
      const int h = task - s.G;
      const float rate = -expf(p.a_log[h]);
      if (s.head_decay) {
        if (lane == 0)
          p.g[(size_t)t * s.H + h] =
              expf(rate * softplus_f(to_f(reinterpret_cast<const E*>(p.decay)[(size_t)t * p.ld_decay + h]) + p.dt_bias[h]));
      } else for (int c = lane * 4; c < s.dp; c += 128) {
        const float4 b = *reinterpret_cast<const float4*>(p.dt_bias + h * s.dp + c);
        float4 x = load_row4(reinterpret_cast<const E*>(p.decay) + (size_t)t * p.ld_decay + h * s.dp + c);
        x.x = expf(rate * softplus_f(x.x + b.x)), x.y = expf(rate * softplus_f(x.y + b.y));
        x.z = expf(rate * softplus_f(x.z + b.z)), x.w = expf(rate * softplus_f(x.w + b.w));
        *reinterpret_cast<float4*>(p.g + ((size_t)t * s.H + h) * s.dp + c) = x;
      }
      if (lane == 0) p.beta[(size_t)t * s.H + h] = sigmoid_f(to_f(buf[(size_t)t * p.ld + p.col_b + h]));
    } else {
      const int h = task - s.G - s.H;
      for (int c = lane * 4; c < s.vp; c += 128)
        *reinterpret_cast<float4*>(p.v + ((size_t)t * s.H + h) * s.vp + c) = conv(2 * nq + h * s.vp + c);
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

constexpr int SCAN_WARPS = 4, SCAN_LANES = 16;

// DPL key channels per lane in pieces of V (2 or 4); `at(i)` is the first channel of piece i of lane `sub`.
template <int DPL>
struct Lane {
  static constexpr int V = DPL % 4 ? 2 : 4, N = DPL / V;
  static __device__ __forceinline__ int at(int i, int sub) { return (i * SCAN_LANES + sub) * V; }
  static __device__ __forceinline__ void load(const float* p, int sub, uint64_t* v) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      if constexpr (V == 4) {
        const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(p + at(i, sub));
        v[2 * i] = x.x, v[2 * i + 1] = x.y;
      } else {
        v[i] = *reinterpret_cast<const uint64_t*>(p + at(i, sub));
      }
    }
  }
  static __device__ __forceinline__ void store(float* p, int sub, const uint64_t* v) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      if constexpr (V == 4) *reinterpret_cast<ulonglong2*>(p + at(i, sub)) = make_ulonglong2(v[2 * i], v[2 * i + 1]);
      else *reinterpret_cast<uint64_t*>(p + at(i, sub)) = v[i];
    }
  }
};

// TB tokens per staged block; layout of one token in shared memory: k [dp], q [dp], g [dp], v [COLS], (kq, beta, -, -). HEAD: one decay
// per head, no g [dp] but (kq, beta, g, -).
template <int DPL, int NC, int TB, bool HEAD>
__global__ void __launch_bounds__(SCAN_WARPS * 32) delta_scan_kernel(const ScanParams p) {
  constexpr int DP = DPL * SCAN_LANES, COLS = SCAN_WARPS * 2 * NC, VO = HEAD ? 2 * DP : 3 * DP, TAIL = VO + COLS, TOK = TAIL + 4, N2 = DPL / 2;
  constexpr bool AHEAD = DPL <= 16;                  // operands of the next token are read while this one is computed
  using L = Lane<DPL>;
  extern __shared__ __align__(16) float sm[];        // 2 blocks of TB tokens
  pdl_wait();
  const DeltaShape& s = p.s;
  const int seq = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * COLS, kvh = h / (s.H / s.G);
  const int tid = threadIdx.x, sub = tid % SCAN_LANES, lc = tid / SCAN_LANES * NC;   // first of this lane's NC columns
  const int start = s.cu_q ? s.cu_q[seq] : seq * s.uniform_q, n = s.cu_q ? s.cu_q[seq + 1] - start : s.uniform_q;
  if (n <= 0) return;
  const int slot = s.slots[seq];
  float* st = p.state + (((size_t)max(slot, 0) * s.H + h) * s.vp + c0 + lc) * DP;
  const bool carried = slot >= 0 && s.positions[start] != 0;
  uint64_t S[NC][N2];
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    if (carried && c0 + lc + c < s.vp) {
      L::load(st + c * DP, sub, S[c]);
    } else {
#pragma unroll
      for (int i = 0; i < N2; ++i) S[c][i] = 0ull;
    }
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
      if constexpr (!HEAD) cp_async16(d + 2 * DP, p.g + (t * s.H + h) * DP + c);
    }
    for (int i = tid; i < m * (COLS / 4); i += SCAN_WARPS * 32) {
      const int r = i / (COLS / 4), c = (i % (COLS / 4)) * 4;
      if (c < ncols) cp_async16(dst0 + r * TOK + VO + c, p.v + ((size_t)(start + t0 + r) * s.H + h) * s.vp + c0 + c);
    }
    for (int r = tid; r < m; r += SCAN_WARPS * 32) {
      cp_async4(dst0 + r * TOK + TAIL, p.kq + (size_t)(start + t0 + r) * s.G + kvh);
      cp_async4(dst0 + r * TOK + TAIL + 1, p.beta + (size_t)(start + t0 + r) * s.H + h);
      if constexpr (HEAD) cp_async4(dst0 + r * TOK + TAIL + 2, p.g + (size_t)(start + t0 + r) * s.H + h);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const int blocks = (n + TB - 1) / TB;
  // which of the 2 NC sums this lane ends up with: dots with k (upper bit 0) or q (1), of column `mine`
  const int mine = NC == 4 ? (sub >> 1) & 3 : NC == 2 ? (sub >> 2) & 1 : 0;
  const bool is_q = sub & 8, writes = is_q && (sub & (NC == 4 ? 1 : NC == 2 ? 3 : 7)) == 0 && c0 + lc + mine < s.vp;
  stage(0);
  float* orow = p.o + ((size_t)start * s.H + h) * s.vp + c0 + lc + mine;
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
    // one token: operands in (k, q, g), those of the next token are read into (kn, qn, gn) meanwhile
    auto step = [&](const float* tok, float* o_to, uint64_t* k, uint64_t* q, uint64_t* g, uint64_t* kn, uint64_t* qn, uint64_t* gn,
                    bool more) {
      const float kq = tok[TAIL], beta = tok[TAIL + 1], v = tok[VO + lc + mine], gh = HEAD ? tok[TAIL + 2] : 1.f;
      const uint64_t gg = dup2(gh);
      if (AHEAD && more) {
        L::load(tok + TOK, sub, kn), L::load(tok + TOK + DP, sub, qn);
        if constexpr (!HEAD) L::load(tok + TOK + 2 * DP, sub, gn);
      }
      float a[2 * NC];
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        uint64_t ak = 0ull, aq = 0ull;
#pragma unroll
        for (int i = 0; i < N2; ++i) {
          if constexpr (!HEAD) S[c][i] = mul2(S[c][i], g[i]);
          ak = i ? fma2(S[c][i], k[i], ak) : mul2(S[c][i], k[i]);
          aq = i ? fma2(S[c][i], q[i], aq) : mul2(S[c][i], q[i]);
        }
        a[c] = sum2(ak), a[NC + c] = sum2(aq);
      }
      // fold: each step halves the number of sums a lane still carries, then plain sums over the remaining lane bits
      int o = 8;
#pragma unroll
      for (int w = NC; w >= 1; w >>= 1, o >>= 1) {
        const bool hi = sub & o;
#pragma unroll
        for (int i = 0; i < w; ++i) {
          const float keep = hi ? a[i + w] : a[i], send = hi ? a[i] : a[i + w];
          a[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
        }
      }
#pragma unroll
      for (; o > 0; o >>= 1) a[0] += __shfl_xor_sync(0xffffffffu, a[0], o);
      if constexpr (HEAD) a[0] *= gh;
      const float u_mine = beta * (v - a[0]);        // meaningful in the lanes that hold a dot with k
      float u_out = 0.f;
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        const float u = __shfl_sync(0xffffffffu, u_mine, (tid & 16) | (NC == 4 ? c << 1 : NC == 2 ? c << 2 : 0));
        if (c == mine) u_out = u;
        const uint64_t uu = dup2(u);
#pragma unroll
        for (int i = 0; i < N2; ++i) S[c][i] = fma2(k[i], uu, HEAD ? mul2(S[c][i], gg) : S[c][i]);
      }
      if (writes) *o_to = fmaf(kq, u_out, a[0]);
    };
    const size_t o_step = (size_t)s.H * s.vp;
    if constexpr (AHEAD) {
      uint64_t k0[N2], q0[N2], g0[N2], k1[N2], q1[N2], g1[N2];
      L::load(tok, sub, k0), L::load(tok + DP, sub, q0);
      if constexpr (!HEAD) L::load(tok + 2 * DP, sub, g0);
      int r = 0;
      for (; r + 2 <= m; r += 2, tok += 2 * TOK, orow += 2 * o_step) {
        step(tok, orow, k0, q0, g0, k1, q1, g1, true);
        step(tok + TOK, orow + o_step, k1, q1, g1, k0, q0, g0, r + 2 < m);
      }
      if (r < m) {
        step(tok, orow, k0, q0, g0, k1, q1, g1, false);
        orow += o_step;
      }
    } else {
      for (int r = 0; r < m; ++r, tok += TOK, orow += o_step) {
        uint64_t k[N2], q[N2], g[N2];
        L::load(tok, sub, k), L::load(tok + DP, sub, q);
        if constexpr (!HEAD) L::load(tok + 2 * DP, sub, g);
        step(tok, orow, k, q, g, k, q, g, false);
      }
    }
    __syncthreads();
  }
  pdl_launch_dependents();
  if (slot >= 0) {
#pragma unroll
    for (int c = 0; c < NC; ++c)
      if (c0 + lc + c < s.vp) L::store(st + c * DP, sub, S[c]);
  }
}

struct PostParams {
  DeltaShape s;
  const float* o;            // [T, H, vp]
  const void* gate;          // [T, ld_gate]: gate logits, H vp
  int ld_gate;
  const float* w;            // [vp]
  float eps;
  int gate_silu;             // the gate is silu of its logits (else their sigmoid)
  void* out;                 // [T, H vp]
  const void* buf;           // projections, for the windows
  int ld;
  void* window;
  int norm_ctas, rows_per_warp;
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
  const int lane = threadIdx.x & 31;
  const long long rows = (long long)s.T * s.H, id0 = ((long long)blockIdx.x * 8 + (threadIdx.x >> 5)) * p.rows_per_warp;
  auto finish = [&](long long id, int c, float4 x, float4 z, float r) {
    const float4 w = __ldg(reinterpret_cast<const float4*>(p.w + c));
    if (p.gate_silu) x = make_float4(x.x * z.x, x.y * z.y, x.z * z.z, x.w * z.w);
    store_row4(reinterpret_cast<E*>(p.out) + id * s.vp + c,
               make_float4(x.x * r * w.x * fast_sigmoid(z.x), x.y * r * w.y * fast_sigmoid(z.y), x.z * r * w.z * fast_sigmoid(z.z),
                           x.w * r * w.w * fast_sigmoid(z.w)));
  };
  auto gate = [&](long long id, int c) {
    return load_row4(reinterpret_cast<const E*>(p.gate) + (size_t)(id / s.H) * p.ld_gate + (id % s.H) * s.vp + c);
  };
  if (s.vp <= 128) {                                 // one piece per lane, the loads of all rows in flight together
    const int c = lane * 4;
    constexpr int R = 4;                             // rows_per_warp is 1 or R
    float4 x[R], z[R];
#pragma unroll
    for (int i = 0; i < R; ++i) {
      x[i] = z[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i < p.rows_per_warp && id0 + i < rows && c < s.vp) x[i] = load_row4(p.o + (id0 + i) * s.vp + c), z[i] = gate(id0 + i, c);
    }
#pragma unroll
    for (int i = 0; i < R; ++i) {
      if (i >= p.rows_per_warp || id0 + i >= rows) return;
      const float r = rsqrtf(warp_sum(dot4(x[i], x[i])) / (float)s.vdim + p.eps);    // padding columns are zero
      if (c < s.vp) finish(id0 + i, c, x[i], z[i], r);
    }
    return;
  }
  for (long long id = id0; id < min(rows, id0 + p.rows_per_warp); ++id) {
    const float* o = p.o + id * s.vp;
    float ss = 0.f;
    for (int c = lane * 4; c < s.vp; c += 128) {
      const float4 x = load_row4(o + c);
      ss += dot4(x, x);
    }
    const float r = rsqrtf(warp_sum(ss) / (float)s.vdim + p.eps);
    for (int c = lane * 4; c < s.vp; c += 128) finish(id, c, load_row4(o + c), gate(id, c), r);
  }
}

template <int DPL, int NC, int TB, bool HEAD>
int launch_scan(const ScanParams& p, cudaStream_t st) {
  constexpr int DP = DPL * SCAN_LANES, COLS = SCAN_WARPS * 2 * NC;
  constexpr size_t smem = 2 * TB * ((HEAD ? 2 : 3) * DP + COLS + 4) * sizeof(float);
  if (smem > 48 * 1024) {
    static bool configured[64] = {false};
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev < 0 || dev >= 64 || !configured[dev]) {
      const cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<DPL, NC, TB, HEAD>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return -(int)e;
      if (dev >= 0 && dev < 64) configured[dev] = true;
    }
  }
  return launch_kernel(delta_scan_kernel<DPL, NC, TB, HEAD>, dim3((p.s.vp + COLS - 1) / COLS, p.s.H, p.s.num_seqs), dim3(SCAN_WARPS * 32),
                       smem, st, p);
}
template <int DPL, int NC, int TB>
int launch_scan(const ScanParams& p, cudaStream_t st) {
  return p.s.head_decay ? launch_scan<DPL, NC, TB, true>(p, st) : launch_scan<DPL, NC, TB, false>(p, st);
}

bool shape_ok(const DeltaShape& s) {
  return s.T > 0 && s.num_seqs > 0 && s.H > 0 && s.G > 0 && s.H % s.G == 0 && s.dim > 0 && s.dim <= s.dp && s.dp % 32 == 0 &&
         s.dp <= 512 && s.vdim > 0 && s.vdim <= s.vp && s.vp % 8 == 0 && s.taps >= 1 && s.positions && s.slots &&
         (s.cu_q || (long long)s.num_seqs * s.uniform_q == s.T);
}

DeltaShape make_shape(const int* dims, const int* cu_q, const int* positions, const int* slots) {
  // dims: T, num_seqs, uniform_q, H, G, dim, dp, vdim, vp, taps, head_decay
  return DeltaShape{dims[0], dims[1], dims[2], cu_q, positions, slots, dims[3], dims[4], dims[5], dims[6], dims[7], dims[8], dims[9], dims[10]};
}

}  // namespace
}  // namespace swb

extern "C" {

}  // extern "C"
namespace swb {
namespace {
template <typename E, int NI>
int launch_prep(const PrepParams& p, cudaStream_t st) {
  const dim3 grid((p.s.T + 7) / 8, (p.s.G + 2 * p.s.H + p.heads_per_cta - 1) / p.heads_per_cta);
  if constexpr (NI > 2) return launch_kernel(delta_prep_kernel<E, 0, NI>, grid, dim3(256), 0, st, p);
  else switch (p.s.taps) {
    case 1: return launch_kernel(delta_prep_kernel<E, 1, NI>, grid, dim3(256), 0, st, p);
    case 2: return launch_kernel(delta_prep_kernel<E, 2, NI>, grid, dim3(256), 0, st, p);
    case 3: return launch_kernel(delta_prep_kernel<E, 3, NI>, grid, dim3(256), 0, st, p);
    case 4: return launch_kernel(delta_prep_kernel<E, 4, NI>, grid, dim3(256), 0, st, p);
    default: return launch_kernel(delta_prep_kernel<E, 0, NI>, grid, dim3(256), 0, st, p);
  }
}
template <typename E>
int launch_prep(const PrepParams& p, cudaStream_t st) {
  return p.s.dp <= 128 ? launch_prep<E, 1>(p, st) : p.s.dp <= 256 ? launch_prep<E, 2>(p, st) : launch_prep<E, 4>(p, st);
}
}  // namespace
}  // namespace swb
extern "C" {

// dims: host int[11] = T, num_seqs, uniform_q (cu_q null), H, G, dim, dp, vdim, vp, taps, head_decay. fp32 selects the element type of
// the projections, windows and decay logits.
int swb_delta_prep(const int* dims, const int* cu_q, const int* positions, const int* slots, const void* buf, int ld, int col_b,
                   const void* decay, int ld_decay, const float* conv, const void* window, const float* a_log, const float* dt_bias,
                   float* qk, float* kq, float* g, float* v, float* beta, int fp32, void* stream) {
  using namespace swb;
  PrepParams p{make_shape(dims, cu_q, positions, slots), buf, ld, col_b, decay, ld_decay, conv, window, a_log, dt_bias, qk, kq, g, v,
               beta, dims[0] >= 4096 ? 8 : dims[0] >= 1024 ? 4 : 1};
  if (dims[0] <= 0) return 0;
  if (!shape_ok(p.s) || (ld % 4) || (!p.s.head_decay && ld_decay % 4)) return -3;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return fp32 ? launch_prep<float>(p, st) : launch_prep<bf16>(p, st);
}

int swb_delta_scan(const int* dims, const int* cu_q, const int* positions, const int* slots, const float* qk, const float* kq,
                   const float* g, const float* v, const float* beta, float* state, float* o, void* stream) {
  using namespace swb;
  ScanParams p{make_shape(dims, cu_q, positions, slots), qk, kq, g, v, beta, state, o};
  if (dims[0] <= 0) return 0;
  if (!shape_ok(p.s)) return -3;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  switch (p.s.dp) {
    case 32: return launch_scan<2, 4, 16>(p, st);
    case 64: return launch_scan<4, 4, 16>(p, st);
    case 96: return launch_scan<6, 4, 16>(p, st);
    case 128: return launch_scan<8, 4, 16>(p, st);
    case 192: return launch_scan<12, 4, 8>(p, st);
    case 256: return launch_scan<16, 4, 8>(p, st);
    case 512: return launch_scan<32, 2, 4>(p, st);
    default: return -3;
  }
}

int swb_delta_post(const int* dims, const int* cu_q, const int* positions, const int* slots, const float* o, const void* gate,
                   int ld_gate, const float* w, float eps, int gate_silu, void* out, const void* buf, int ld, void* window, int fp32,
                   void* stream) {
  using namespace swb;
  PostParams p{make_shape(dims, cu_q, positions, slots), o, gate, ld_gate, w, eps, gate_silu, out, buf, ld, window, 0,
               dims[0] >= 1024 ? 4 : 1};
  if (dims[0] <= 0) return 0;
  if (!shape_ok(p.s)) return -3;
  p.norm_ctas = (int)(((long long)p.s.T * p.s.H + 8 * p.rows_per_warp - 1) / (8 * p.rows_per_warp));
  const int C = 2 * p.s.G * p.s.dp + p.s.H * p.s.vp;
  const dim3 grid(p.norm_ctas + (p.s.taps > 1 ? p.s.num_seqs * ((C + 1023) / 1024) : 0));
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return fp32 ? launch_kernel(delta_post_kernel<float>, grid, dim3(256), 0, st, p)
              : launch_kernel(delta_post_kernel<bf16>, grid, dim3(256), 0, st, p);
}

}  // extern "C"
