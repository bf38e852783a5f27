// Residual streams side by side (hyper-connections) in 32-bit, and the short convolution behind each sublayer's norm.
//
// hyper_step_kernel is what lies between two sublayers, in one pass over a token:
//     x_t <- sum_s mix[s, t] x_s + put[t] y      (all t at once; y: one projection row, two normed ones, or weighted expert rows)
//     h    = N(sum_t read[t] x_t) w              (RMS norm)
//     out  = h + conv(h)                         (optional: only where every sequence has one token in this step)
// A thread owns columns, so the streams of a column are mixed in registers and only the norms' statistics cross threads. For one-token
// sequences the convolution's other inputs are the sequence's window, column by column as well; prompts take short_conv_kernel.
// Padding columns (from H to Hp) of the streams, branches and weights are zero.
#include "common.cuh"

namespace swb {

SWB_REGISTER_STATUS_UNIT(hyper_stream);

namespace {

struct ConvParams {
  const float* w;             // [taps, Hp]: the last row is the current token's
  int taps;
  void* window;               // [slots, taps - 1, Hp]: the inputs in front of the step, oldest first
  const int* slots;           // [num_seqs], < 0: no window (zeros, nothing kept)
  const int* positions;       // [T]; a sequence that starts this step at position 0 starts from zeros
};

struct HyperParams {
  const float* x_in;          // streams as they are: token t, stream s at t * in_tok + s * in_stream
  long long in_tok, in_stream;
  float* x;                   // [T, S, Hp] (with a branch)
  const long long* rows;      // optional: output row i is token rows[i] (no branch then)
  int S;
  const float *mix, *put;     // [S (from), S (to)], [S]
  const float* read;          // [S] or null (ones)
  const void *y, *y2;         // branch: y, or N(y) w_y + N(y2) w_y2, or weighted rows of y
  int ld_y, ld_y2;
  const float *w_y, *w_y2;
  const int* pick;            // optional [T, top]: the branch is sum_k pick_weights[t, k] y[pick[t, k]]
  const float* pick_weights;
  int top;
  const float* w;             // norm of what is read
  void* out;                  // optional [*, ldo]
  int ldo;
  ConvParams conv;            // w null: none
  int H, Hp;
  float eps;
};

constexpr int MAX_STREAMS = 16;

// Sums over the block of two values; one barrier per call, `red` is used by one call only.
template <int THREADS>
__device__ __forceinline__ float2 block_total2(float a, float b, float2* red) {
  a = warp_sum(a), b = warp_sum(b);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (lane == 0) red[warp] = make_float2(a, b);
  __syncthreads();
  const float2 v = lane < THREADS / 32 ? red[lane] : make_float2(0.f, 0.f);
  return make_float2(warp_sum(v.x), warp_sum(v.y));
}

__device__ __forceinline__ float sq4(float4 a) { return fmaf(a.x, a.x, fmaf(a.y, a.y, fmaf(a.z, a.z, a.w * a.w))); }
__device__ __forceinline__ float4 fma4(float w, float4 a, float4 b) {
  return make_float4(fmaf(w, a.x, b.x), fmaf(w, a.y, b.y), fmaf(w, a.z, b.z), fmaf(w, a.w, b.w));
}
__device__ __forceinline__ float4 fma4(float4 w, float4 a, float4 b) {
  return make_float4(fmaf(w.x, a.x, b.x), fmaf(w.y, a.y, b.y), fmaf(w.z, a.z, b.z), fmaf(w.w, a.w, b.w));
}
__device__ __forceinline__ float4 mul4(float4 a, float4 b, float r) {
  return make_float4(a.x * b.x * r, a.y * b.y * r, a.z * b.z * r, a.w * b.w * r);
}
// the value as it is stored
template <typename E>
__device__ __forceinline__ float4 rounded4(float4 v) {
  if constexpr (sizeof(E) == 4) return v;
  return make_float4(__bfloat162float(__float2bfloat16(v.x)), __bfloat162float(__float2bfloat16(v.y)),
                     __bfloat162float(__float2bfloat16(v.z)), __bfloat162float(__float2bfloat16(v.w)));
}

// SM >= S bounds the streams a thread holds.
template <typename E, int THREADS, int VPT, int SM>
__global__ void __launch_bounds__(THREADS) hyper_step_kernel(const HyperParams p) {
  pdl_launch_dependents();
  __shared__ float coef[SM * SM + 2 * SM];      // mix, put, read
  __shared__ float2 red[2][32];
  const int S = p.S, nvec = p.Hp / 4;
  for (int i = threadIdx.x; i < SM * SM + 2 * SM; i += THREADS) {      // weights: they do not depend on the kernel in front
    float v = 0.f;
    if (i < SM * SM) {
      const int s = i / SM, t = i % SM;
      if (p.y && s < S && t < S) v = p.mix[s * S + t];
    } else if (i < SM * SM + SM) {
      const int t = i - SM * SM;
      if (p.y && t < S) v = p.put[t];
    } else {
      const int t = i - SM * SM - SM;
      if (t < S) v = p.read ? p.read[t] : 1.f;
    }
    coef[i] = v;
  }
  pdl_wait(TL_RMSNORM);
  const int row = blockIdx.x;
  const long long tok = p.rows ? p.rows[row] : row;
  const float* xi = p.x_in + tok * p.in_tok;
  float4 x[VPT][SM], v[VPT];
  auto load_x = [&] {
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * THREADS;
#pragma unroll
      for (int s = 0; s < SM; ++s)
        x[i][s] = c < nvec && s < S ? *reinterpret_cast<const float4*>(xi + s * p.in_stream + c * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  load_x();
  if (p.y) {
    const E* y = reinterpret_cast<const E*>(p.y);
    float4 v2[VPT];
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * THREADS;
      v[i] = v2[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < nvec && !p.pick) v[i] = load_row4(y + (size_t)row * p.ld_y + c * 4);
      if (c < nvec && p.y2) v2[i] = load_row4(reinterpret_cast<const E*>(p.y2) + (size_t)row * p.ld_y2 + c * 4);
    }
    if (p.pick) {
#pragma unroll 4
      for (int k = 0; k < p.top; ++k) {
        const E* yr = y + (size_t)p.pick[row * p.top + k] * p.ld_y;
        const float w = p.pick_weights[row * p.top + k];
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
          const int c = threadIdx.x + i * THREADS;
          if (c < nvec) v[i] = fma4(w, load_row4(yr + c * 4), v[i]);
        }
      }
    }
    if (p.w_y) {
      float a = 0.f, b = 0.f;
#pragma unroll
      for (int i = 0; i < VPT; ++i) a += sq4(v[i]), b += sq4(v2[i]);
      const float2 ss = block_total2<THREADS>(a, b, red[0]);
      const float r = rsqrtf(ss.x / (float)p.H + p.eps), r2 = rsqrtf(ss.y / (float)p.H + p.eps);
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + i * THREADS;
        if (c >= nvec) continue;
        v[i] = mul4(v[i], __ldg(reinterpret_cast<const float4*>(p.w_y) + c), r);
        if (p.y2) {
          const float4 u = mul4(v2[i], __ldg(reinterpret_cast<const float4*>(p.w_y2) + c), r2);
          v[i].x += u.x, v[i].y += u.y, v[i].z += u.z, v[i].w += u.w;
        }
      }
    } else {
      __syncthreads();                         // coef
    }
    float* xo = p.x + (size_t)row * S * p.Hp;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * THREADS;
      float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int t = 0; t < SM; ++t) {
        if (t >= S) break;
        const float w = coef[SM * SM + t];
        float4 z = make_float4(v[i].x * w, v[i].y * w, v[i].z * w, v[i].w * w);
#pragma unroll
        for (int s = 0; s < SM; ++s) {
          if (s >= S) break;
          z = fma4(coef[s * SM + t], x[i][s], z);
        }
        if (c < nvec) *reinterpret_cast<float4*>(xo + (size_t)t * p.Hp + c * 4) = z;
        u = fma4(coef[SM * SM + SM + t], z, u);
      }
      v[i] = u;
    }
  } else {
    __syncthreads();
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int s = 0; s < SM; ++s) {
        if (s >= S) break;
        v[i] = fma4(coef[SM * SM + SM + s], x[i][s], v[i]);
      }
    }
  }
  if (!p.out) return;
  float a = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) a += sq4(v[i]);
  const float r = rsqrtf(block_total2<THREADS>(a, 0.f, red[1]).x / (float)p.H + p.eps);
  E* out = reinterpret_cast<E*>(p.out) + (size_t)row * p.ldo;
  const ConvParams& cv = p.conv;
  const int slot = cv.w ? cv.slots[row] : -1, keep = cv.taps - 1;
  E* win = slot >= 0 && keep > 0 ? reinterpret_cast<E*>(cv.window) + (size_t)slot * keep * p.Hp : nullptr;
  const bool carried = win && cv.positions[row] != 0;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = threadIdx.x + i * THREADS;
    if (c >= nvec) continue;
    float4 h = mul4(v[i], __ldg(reinterpret_cast<const float4*>(p.w) + c), r);
    if (cv.w) {
      h = rounded4<E>(h);
      const float4* wc = reinterpret_cast<const float4*>(cv.w) + c;
      float4 y = fma4(__ldg(wc + (size_t)keep * nvec), h, h);
      for (int j = 0; j < keep; ++j) {         // ascending: an old entry is read before it is overwritten
        const float4 old = carried ? load_row4(win + (size_t)j * p.Hp + c * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
        y = fma4(__ldg(wc + (size_t)j * nvec), old, y);
        if (win && j > 0) store_row4(win + (size_t)(j - 1) * p.Hp + c * 4, old);
      }
      if (win) store_row4(win + (size_t)(keep - 1) * p.Hp + c * 4, h);
      h = y;
    }
    store_row4(out + c * 4, h);
  }
}

// out = h + conv(h) over a ragged batch of sequences: a thread owns eight channels of up to `chunk` consecutive tokens. The first piece of
// a sequence alone reads its window (chunk >= taps - 1), and moves it on.
struct ShortConvParams {
  const void* h;              // [T, ldh]
  void* out;                  // [T, ldo]
  int ldh, ldo;
  ConvParams conv;
  const int* cu_q;            // [num_seqs + 1] or null (uniform_q tokens each)
  int uniform_q, Hp, chunk;
};

// TAPS 0: any number.
template <typename E, int TAPS>
__global__ void __launch_bounds__(128) short_conv_kernel(const ShortConvParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const ConvParams& cv = p.conv;
  const int seq = blockIdx.z, start = p.cu_q ? p.cu_q[seq] : seq * p.uniform_q, n = p.cu_q ? p.cu_q[seq + 1] - start : p.uniform_q;
  const int first = blockIdx.y * p.chunk, last = min(first + p.chunk, n), c8 = (blockIdx.x * 128 + threadIdx.x) * 8;
  if (first >= n || c8 >= p.Hp) return;
  const int taps = TAPS > 0 ? TAPS : cv.taps, keep = taps - 1, slot = cv.slots[seq];
  E* win = slot >= 0 && keep > 0 ? reinterpret_cast<E*>(cv.window) + (size_t)slot * keep * p.Hp + c8 : nullptr;
  const bool carried = win && cv.positions[start] != 0;
  const E* h = reinterpret_cast<const E*>(p.h) + (size_t)start * p.ldh + c8;
  E* out = reinterpret_cast<E*>(p.out) + (size_t)start * p.ldo + c8;
  auto weights = [&](int j, float* w) { load_row8(cv.w + (size_t)j * p.Hp + c8, w); };
  auto input = [&](int r, float* x) {          // input of token r of this step, r < 0: in front of it
    if (r >= 0) load_row8(h + (size_t)r * p.ldh, x);
    else if (carried) load_row8(win + (size_t)(keep + r) * p.Hp, x);
    else
#pragma unroll
      for (int k = 0; k < 8; ++k) x[k] = 0.f;
  };
  if constexpr (TAPS > 0) {
    constexpr int B = 4;                       // tokens whose loads are in flight together
    float w[TAPS][8], x[TAPS - 1 + B][8];      // x[j]: input of token t - keep + j
#pragma unroll
    for (int j = 0; j < TAPS; ++j) weights(j, w[j]);
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) input(first - keep + j, x[j]);
    for (int t = first; t < last; t += B) {
#pragma unroll
      for (int i = 0; i < B; ++i) load_row8(h + (size_t)min(t + i, last - 1) * p.ldh, x[TAPS - 1 + i]);
#pragma unroll
      for (int i = 0; i < B; ++i) {
        if (t + i >= last) break;
        float y[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          y[k] = x[TAPS - 1 + i][k];
#pragma unroll
          for (int j = 0; j < TAPS; ++j) y[k] = fmaf(w[j][k], x[i + j][k], y[k]);
        }
        store_row8(out + (size_t)(t + i) * p.ldo, y);
      }
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
        for (int k = 0; k < 8; ++k) x[j][k] = x[j + B][k];
    }
  } else {
    for (int t = first; t < last; ++t) {
      float y[8], x[8], w[8];
      input(t, y);
      for (int j = 0; j < taps; ++j) {
        input(t - keep + j, x), weights(j, w);
#pragma unroll
        for (int k = 0; k < 8; ++k) y[k] = fmaf(w[k], x[k], y[k]);
      }
      store_row8(out + (size_t)t * p.ldo, y);
    }
  }
  if (blockIdx.y == 0 && win)
    for (int j = 0; j < keep; ++j) {           // ascending, as above
      float x[8];
      input(n - keep + j, x);
      store_row8(win + (size_t)j * p.Hp, x);
    }
}

template <typename E, int THREADS, int VPT>
int launch_hyper(const HyperParams& p, int T, cudaStream_t s) {
  const dim3 grid((unsigned)T), block(THREADS);
  if (p.S == 1) return launch_kernel(hyper_step_kernel<E, THREADS, VPT, 1>, grid, block, 0, s, p);
  if (p.S == 2) return launch_kernel(hyper_step_kernel<E, THREADS, VPT, 2>, grid, block, 0, s, p);
  if (p.S <= 4) return launch_kernel(hyper_step_kernel<E, THREADS, VPT, 4>, grid, block, 0, s, p);
  if (p.S <= 8) return launch_kernel(hyper_step_kernel<E, THREADS, VPT, 8>, grid, block, 0, s, p);
  return launch_kernel(hyper_step_kernel<E, THREADS, VPT, MAX_STREAMS>, grid, block, 0, s, p);
}

template <typename E>
int launch_hyper(const HyperParams& p, int T, cudaStream_t s) {
  const int nvec = p.Hp / 4;
  if (nvec <= 128) return launch_hyper<E, 128, 1>(p, T, s);
  if (nvec <= 256) return launch_hyper<E, 256, 1>(p, T, s);
  if (nvec <= 512) return launch_hyper<E, 256, 2>(p, T, s);
  if (nvec <= 1024) return launch_hyper<E, 512, 2>(p, T, s);
  if (nvec <= 2048) return launch_hyper<E, 1024, 2>(p, T, s);
  return launch_hyper<E, 1024, 4>(p, T, s);
}

}  // namespace
}  // namespace swb

extern "C" {

// See HyperParams and ConvParams. dims: host int[8] = T, S, H, Hp, top, taps, fp32, number of sequences. fp32 selects the element type of
// the branches, out and the window. Hp a multiple of 8 up to 16384, rows of 16-byte (bf16: 8-byte) alignment, S up to 16.
int swb_hyper_step(const int* dims, const float* x_in, long long in_tok, long long in_stream, float* x, const long long* rows,
                   const float* mix, const float* put, const float* read, const void* y, int ld_y, const float* w_y, const void* y2,
                   int ld_y2, const float* w_y2, const int* pick, const float* pick_weights, const float* w, void* out, int ldo, float eps,
                   const float* conv_w, void* window, const int* slots, const int* positions, void* stream) {
  using namespace swb;
  const int T = dims[0], S = dims[1], H = dims[2], Hp = dims[3], top = dims[4], taps = dims[5], fp32 = dims[6], seqs = dims[7];
  if (T <= 0) return 0;
  if (S < 1 || S > MAX_STREAMS || H < 1 || H > Hp || (Hp % 8) || Hp > 16384 || !x_in || ((in_tok | in_stream) % 4) || (out && (!w || ldo % 4)))
    return -3;
  if (y ? (!x || !mix || !put || rows || (ld_y % 4) || (y2 && (!w_y || !w_y2 || ld_y2 % 4)) || (pick && (!pick_weights || top < 1 || w_y)))
        : (!out || y2 || pick))
    return -3;
  if (conv_w && (rows || taps < 1 || !slots || !positions || seqs != T || (taps > 1 && !window) || !out)) return -3;
  const HyperParams p{x_in, in_tok, in_stream, x, rows, S, mix, put, read, y, y2, ld_y, ld_y2, w_y, w_y2, pick, pick_weights, top, w, out, ldo,
                      ConvParams{conv_w, conv_w ? taps : 1, window, slots, positions}, H, Hp, eps};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return fp32 ? launch_hyper<float>(p, T, s) : launch_hyper<bf16>(p, T, s);
}

// See ShortConvParams. max_q bounds a sequence's tokens (all have max_q without cu_q).
int swb_short_conv(const void* h, int ldh, void* out, int ldo, const float* conv_w, int taps, void* window, const int* slots,
                   const int* positions, const int* cu_q, int num_seqs, int max_q, int Hp, int fp32, void* stream) {
  using namespace swb;
  if (num_seqs <= 0 || max_q <= 0) return 0;
  if (Hp < 8 || (Hp % 8) || ((ldh | ldo) % 8) || taps < 1 || !conv_w || !slots || !positions || (taps > 1 && !window) || h == out) return -3;
  const int chunk = taps > 17 ? taps - 1 : 16;
  const ShortConvParams p{h, out, ldh, ldo, ConvParams{conv_w, taps, window, slots, positions}, cu_q, max_q, Hp, chunk};
  const dim3 grid((Hp / 8 + 127) / 128, (max_q + chunk - 1) / chunk, num_seqs), block(128);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  auto go = [&](auto bk, auto fk) { return fp32 ? launch_kernel(fk, grid, block, 0, s, p) : launch_kernel(bk, grid, block, 0, s, p); };
  switch (taps) {
    case 2: return go(short_conv_kernel<bf16, 2>, short_conv_kernel<float, 2>);
    case 3: return go(short_conv_kernel<bf16, 3>, short_conv_kernel<float, 3>);
    case 4: return go(short_conv_kernel<bf16, 4>, short_conv_kernel<float, 4>);
    default: return go(short_conv_kernel<bf16, 0>, short_conv_kernel<float, 0>);
  }
}

}  // extern "C"
