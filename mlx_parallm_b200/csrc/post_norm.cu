// Row-wise step of designs whose sublayers read the residual stream itself and are normed on their OUTPUT only, and whose stream
// may be replaced after a layer by a weighted sum of the embedding output and every layer's result so far ("depth average").
// One pass over a token's row closes a sublayer and writes what comes next:
//   x = (y given) h + rms_norm(y) w,  or  rms_norm(h) w  (the embedding's norm)
//   stack[slot] = x                     (slot >= 0: x is one of the vectors the averages read)
//   h = sum_{j < n - 1} a_j stack[j] + a_{n-1} x     (a given; otherwise h = x)
//   raw_out = h in the storage type     (what the next sublayer multiplies)
// Everything is fp32 except raw_out.  The stack lies token by token, [M, slots, W]: `slot` is none of the slots that
// the average reads.
#include "common.cuh"

namespace b200p {

// V neighbouring channels per access (4: 16 bytes), ITEMS accesses per thread; the row stays in registers between the norm's
// sum of squares and the result
template <typename T, int V, int ITEMS>
__global__ void __launch_bounds__(ITEMS <= 2 ? 1024 : 512)
post_norm_step_kernel(const float* __restrict__ y, const float* __restrict__ w, float* __restrict__ h, float* __restrict__ stack,
                      int64_t slots, int slot, const float* __restrict__ a, int n, T* __restrict__ raw_out, int64_t W, float eps) {
  __shared__ float red[32];
  const int64_t t = blockIdx.x;
  float* hr = h + t * W;
  const float* src = y ? y + t * W : hr;
  float x[ITEMS][V], hv[ITEMS][V], acc[ITEMS][V], ss = 0.f;
  auto load = [&](const float* p, float (&r)[V]) {
    if constexpr (V == 4) {
      const float4 q = *reinterpret_cast<const float4*>(p);
      r[0] = q.x; r[1] = q.y; r[2] = q.z; r[3] = q.w;
    } else {
      r[0] = *p;
    }
  };
  auto store = [&](float* p, const float (&r)[V]) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r[0], r[1], r[2], r[3]);
    else *p = r[0];
  };
  // everything that does not wait for the norm's sum is read before it: the row, the stream, the weighted vectors of the stack
#pragma unroll
  for (int i = 0; i < ITEMS; ++i) {
    const int64_t c = ((int64_t)i * blockDim.x + threadIdx.x) * V;
#pragma unroll
    for (int k = 0; k < V; ++k) acc[i][k] = hv[i][k] = x[i][k] = 0.f;
    if (c >= W) continue;
    load(src + c, x[i]);
    if (y) load(hr + c, hv[i]);
    if (a) {
      const float* st = stack + t * slots * W + c;
#pragma unroll 4
      for (int j = 0; j < n - 1; ++j) {
        float v[V];
        load(st + (int64_t)j * W, v);
#pragma unroll
        for (int k = 0; k < V; ++k) acc[i][k] = fmaf(a[j], v[k], acc[i][k]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < ITEMS; ++i)
#pragma unroll
    for (int k = 0; k < V; ++k) ss = fmaf(x[i][k], x[i][k], ss);
  ss = warp_sum(ss);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  float total = 0.f;
  for (int i = 0; i < nw; ++i) total += red[i];      // same order in every thread
  const float inv = 1.f / sqrtf(total / (float)W + eps), last = a ? a[n - 1] : 1.f;
#pragma unroll
  for (int i = 0; i < ITEMS; ++i) {
    const int64_t c = ((int64_t)i * blockDim.x + threadIdx.x) * V;
    if (c >= W) continue;
    float wv[V];
    load(w + c, wv);
#pragma unroll
    for (int k = 0; k < V; ++k) x[i][k] = hv[i][k] + x[i][k] * inv * wv[k];          // hv is zero without y
    if (slot >= 0) store(stack + (t * slots + slot) * W + c, x[i]);
    if (a) {
#pragma unroll
      for (int k = 0; k < V; ++k) x[i][k] = fmaf(last, x[i][k], acc[i][k]);
    }
    store(hr + c, x[i]);
    if (raw_out) {
      T* o = raw_out + t * W + c;
      if constexpr (V == 4 && sizeof(T) == 2) {
        T q[4] = {Tr<T>::from_f(x[i][0]), Tr<T>::from_f(x[i][1]), Tr<T>::from_f(x[i][2]), Tr<T>::from_f(x[i][3])};
        *reinterpret_cast<uint2*>(o) = *reinterpret_cast<const uint2*>(q);
      } else {
#pragma unroll
        for (int k = 0; k < V; ++k) o[k] = Tr<T>::from_f(x[i][k]);
      }
    }
  }
}

constexpr int POST_NORM_MAX_ITEMS = 8;

template <typename T, int V>
static int post_norm_step_launch(const float* y, const float* w, float* h, float* stack, int64_t slots, int slot, const float* a, int n,
                                 void* raw_out, int64_t M, int64_t W, float eps, cudaStream_t st) {
  const int64_t pieces = (W + V - 1) / V;
  // many tokens: CTAs of at most 256 threads with several pieces each; few tokens (a decode step): a row over more threads
  int64_t threads = M >= 512 ? 256 : 1024;
  if (pieces < threads) threads = (pieces + 31) / 32 * 32;
  while ((pieces + threads - 1) / threads > 4 && threads < 512) threads *= 2;
  if ((pieces + threads - 1) / threads > 2 && threads > 512) threads = 512;          // what the kernels of 4 and 8 pieces take
  const int64_t items = (pieces + threads - 1) / threads;
  B200P_REQUIRE(items <= POST_NORM_MAX_ITEMS, B200P_ERR_ARG, "rows of %lld values are not built", (long long)W);
#define PN_CASE(I_)                                                                                                          \
  if (items <= I_) {                                                                                                         \
    post_norm_step_kernel<T, V, I_><<<(unsigned)M, (unsigned)threads, 0, st>>>(y, w, h, stack, slots, slot, a, n, (T*)raw_out, W, eps); \
  } else
  PN_CASE(1) PN_CASE(2) PN_CASE(4) PN_CASE(8) {}
#undef PN_CASE
  B200P_LAUNCH_CHECK("post_norm_step_kernel");
  return B200P_OK;
}

}  // namespace b200p

using namespace b200p;

extern "C" int b200p_post_norm_step(const float* y, const float* w, float* h, float* stack, int64_t slots, int slot, const float* a,
                                    int n, void* raw_out, int64_t M, int64_t W, float eps, int dtype, void* stream) {
  B200P_REQUIRE(w && h && W > 0, B200P_ERR_ARG, "null pointer");
  B200P_REQUIRE(slot < 0 || (stack && slot < slots), B200P_ERR_ARG, "the stack has no slot %d", slot);
  B200P_REQUIRE(a == nullptr || (n >= 1 && (n == 1 || (stack && n - 1 <= slots))), B200P_ERR_ARG, "an average over %d vectors needs as many slots less one", n);
  if (M == 0) return B200P_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const bool vec = W % 4 == 0 && aligned(y, 16) && aligned(w, 16) && aligned(h, 16) && aligned(stack, 16) && aligned(raw_out, dtype == B200P_F32 ? 16 : 8);
#define PN_DTYPE(T)                                                                                                  \
  return vec ? post_norm_step_launch<T, 4>(y, w, h, stack, slots, slot, a, n, raw_out, M, W, eps, st)               \
             : post_norm_step_launch<T, 1>(y, w, h, stack, slots, slot, a, n, raw_out, M, W, eps, st)
  switch (raw_out ? dtype : B200P_F32) {
    case B200P_F32: PN_DTYPE(float);
    case B200P_F16: PN_DTYPE(__half);
    case B200P_BF16: PN_DTYPE(__nv_bfloat16);
    default: set_error("bad dtype %d", dtype); return B200P_ERR_ARG;
  }
#undef PN_DTYPE
}
