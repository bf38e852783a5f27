// Latent attention: a token's keys and values of all heads are projections of one cached row [c | k_rot], c the normed latent
// (rank numbers) and k_rot the rotated key part shared by the heads.
//   latent_prep   norm of c, rotation of k_rot and of every head's rotated query part, cache write.
#include "common.cuh"

namespace swb {

SWB_REGISTER_STATUS_UNIT(latent_attention);

namespace {

struct LatentPrepParams {
  void* buf;                 // projections [T, ld]: q (H heads of dn + rp) at 0, c (rk) at col_c, k_rot (rp) behind it
  int ld, col_c;
  const float* w;            // [rk]
  float eps;
  const float *cos, *sin;    // [positions, rot / 2]
  const int* positions;
  const long long* slots;    // row of the cache, < 0: none
  void* cache;               // [rows, rk + rp]
  void* q_abs;               // optional [T, H, rk + rp]: receives the rotated query part at column rk
  int T, H, dn, rot, rp, rank, rk;
};

template <typename E>
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentPrepParams p) {
  pdl_launch_dependents();
  pdl_wait(TL_ROPE_KV);
  __shared__ float red[8];
  const int t = blockIdx.x, pos = p.positions[t], half = p.rp / 2, width = p.rk + p.rp;
  E* row = reinterpret_cast<E*>(p.buf) + (size_t)t * p.ld;
  E* c = row + p.col_c;
  const long long slot = p.slots[t];
  E* dst = slot >= 0 ? reinterpret_cast<E*>(p.cache) + (size_t)slot * width : nullptr;
  float ss = 0.f;
  for (int i = threadIdx.x; i < p.rank; i += 256) ss = fmaf(to_f(c[i]), to_f(c[i]), ss);
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) ss += red[w];
  const float r = rsqrtf(ss / (float)p.rank + p.eps);
  for (int i = threadIdx.x; i < p.rk; i += 256) {
    E x;
    from_f(x, i < p.rank ? to_f(c[i]) * r * p.w[i] : 0.f);
    c[i] = x;
    if (dst) dst[i] = x;
  }
  const float* cs = p.cos + (size_t)pos * (p.rot / 2);
  const float* sn = p.sin + (size_t)pos * (p.rot / 2);
  for (int i = threadIdx.x; i < (p.H + 1) * half; i += 256) {       // pairs of the heads' queries, then of the shared key
    const int h = i / half, k = i % half;
    E* x = (h < p.H ? row + h * (p.dn + p.rp) + p.dn : c + p.rk) + 2 * k;
    E y[2] = {x[0], x[1]};
    if (2 * k < p.rot) {
      const float u = to_f(x[0]), v = to_f(x[1]), a = cs[k], b = sn[k];
      from_f(y[0], u * a - v * b);
      from_f(y[1], v * a + u * b);
      x[0] = y[0], x[1] = y[1];
    }
    E* to = h < p.H ? (p.q_abs ? reinterpret_cast<E*>(p.q_abs) + ((size_t)t * p.H + h) * width : nullptr) : dst;
    if (to) to[p.rk + 2 * k] = y[0], to[p.rk + 2 * k + 1] = y[1];
  }
}

}  // namespace
}  // namespace swb

extern "C" {

int swb_latent_prep(void* buf, int ld, int col_c, const float* w, float eps, const float* cos, const float* sin, const int* positions,
                    const long long* slots, void* cache, void* q_abs, int T, int H, int dn, int rot, int rp, int rank, int rk, int fp32,
                    void* stream) {
  using namespace swb;
  if (T <= 0) return 0;
  if (H <= 0 || dn <= 0 || rot <= 0 || (rot % 2) || rot > rp || (rp % 2) || rank <= 0 || rank > rk || !cache || !slots) return -3;
  const LatentPrepParams p{buf, ld, col_c, w, eps, cos, sin, positions, slots, cache, q_abs, T, H, dn, rot, rp, rank, rk};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return fp32 ? launch_kernel(latent_prep_kernel<float>, dim3((unsigned)T), dim3(256), 0, s, p)
              : launch_kernel(latent_prep_kernel<bf16>, dim3((unsigned)T), dim3(256), 0, s, p);
}

}  // extern "C"
