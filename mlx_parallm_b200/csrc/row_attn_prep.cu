// Preparation of grouped attention whose projections are biased and whose q and k are rms-normed as WHOLE rows, all heads at once:
//   row_attn_prep_kernel   biases on q, k, v; the two row norms; half-split or pairwise rotation of the first dimensions of every
//                          head; a query temperature 1 + coef ln(floor((p + 1) / every) + 1); values blended with an earlier
//                          layer's values of the same token; q scaled into fp32, k and v into the cache at (row, position)
//                          (per token)
// Every option is a parameter (no bias, no norm, no rotation, no temperature, no blending); everything is fp32 up to the caches.
#include "common.cuh"
#include "mma_util.cuh"

namespace b200p {

// V fp32 values into V neighbouring cache elements (V == 4: one 8- or 16-byte store)
template <typename T, int V>
__device__ __forceinline__ void store_cache(T* d, const float (&x)[V]) {
  if constexpr (V == 4 && sizeof(T) == 2) {
    *reinterpret_cast<uint2*>(d) = make_uint2(pack2<T>(x[0], x[1]), pack2<T>(x[2], x[3]));
  } else {
#pragma unroll
    for (int k = 0; k < V; ++k) d[k] = Tr<T>::from_f(x[k]);
  }
}

// V neighbouring channels per access (4: every head starts on a 16-byte boundary and a rotated group of 4 stays inside its half)
template <typename T, int V>
__global__ void __launch_bounds__(256)
row_attn_prep_kernel(const float* __restrict__ proj, int64_t ldp, int64_t col_q, int64_t col_k, int64_t col_v,
                     const float* __restrict__ bias, const float* __restrict__ wq, const float* __restrict__ wk, float eps,
                     const float* __restrict__ rates, int n_rot, float mag, int pairs, float scale, float temp_coef, float temp_every,
                     const float* __restrict__ v_first, float v_lambda, float* __restrict__ v_keep, float* __restrict__ q_out,
                     T* __restrict__ kcache, T* __restrict__ vcache, int64_t Tcap, const int32_t* __restrict__ t_row,
                     const int32_t* __restrict__ t_pos, int H, int G, int dk, int dv, int buffered) {
  // the biased q | k row (buffered: read once from memory, afterwards from here), cos and sin of this position ([n_rot] each)
  extern __shared__ __align__(16) float mp_sm[];
  __shared__ float red[2][8];
  float* rowbuf = mp_sm;
  float* cs = mp_sm + (buffered ? (H + G) * dk : 0);
  float* sn = cs + n_rot;
  const int64_t t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const int64_t pos = t_pos[t], row = t_row[t];
  const float* pt = proj + t * ldp;
  for (int i = threadIdx.x; i < n_rot; i += blockDim.x) {
    float s, c;
    sincosf((float)pos * rates[i], &s, &c);
    cs[i] = c * mag;
    sn[i] = s * mag;
  }
  if (temp_coef != 0.f) scale *= 1.f + temp_coef * logf(floorf((float)(pos + 1) / temp_every) + 1.f);
  auto load = [&](int64_t col, float (&r)[V]) {                    // biased projection columns
    if constexpr (V == 4) {
      const float4 q = *reinterpret_cast<const float4*>(pt + col);
      r[0] = q.x; r[1] = q.y; r[2] = q.z; r[3] = q.w;
      if (bias) {
        const float4 b = *reinterpret_cast<const float4*>(bias + col);
        r[0] += b.x; r[1] += b.y; r[2] += b.z; r[3] += b.w;
      }
    } else {
      r[0] = pt[col] + (bias ? bias[col] : 0.f);
    }
  };
  const int nq = H * dk, nk = G * dk;
  float sq = 0.f, sk = 0.f;
  if (wq || wk || buffered) {
#pragma unroll 4
    for (int c = threadIdx.x * V; c < nq + nk; c += blockDim.x * V) {
      float r[V], ss = 0.f;
      load(c < nq ? col_q + c : col_k + c - nq, r);
      if (buffered) {
        if constexpr (V == 4) *reinterpret_cast<float4*>(rowbuf + c) = make_float4(r[0], r[1], r[2], r[3]);
        else rowbuf[c] = r[0];
      }
#pragma unroll
      for (int k = 0; k < V; ++k) ss = fmaf(r[k], r[k], ss);
      if (c < nq) sq += ss;
      else sk += ss;
    }
  }
  const bool in_cache = pos < Tcap;                                // the host sizes the cache first; never write outside it
  if (in_cache || v_keep)                                          // the values need no norm: their reads overlap the reduction
    for (int c = threadIdx.x * V; c < G * dv; c += blockDim.x * V) {
      float r[V];
      load(col_v + c, r);
      const int64_t at = t * G * dv + c;
      if (v_first) {                                               // blended with the same token's values of an earlier layer
#pragma unroll
        for (int k = 0; k < V; ++k) r[k] = (1.f - v_lambda) * r[k] + v_lambda * v_first[at + k];
      }
      if (v_keep) {
#pragma unroll
        for (int k = 0; k < V; ++k) v_keep[at + k] = r[k];
      }
      if (in_cache) store_cache<T, V>(vcache + ((row * G + c / dv) * Tcap + pos) * dv + c % dv, r);
    }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if (lane == 0) { red[0][warp] = sq; red[1][warp] = sk; }
  __syncthreads();
  sq = sk = 0.f;
  for (int i = 0; i < nw; ++i) { sq += red[0][i]; sk += red[1][i]; }
  const float inv_q = wq ? 1.f / sqrtf(sq / (float)nq + eps) : 1.f, inv_k = wk ? 1.f / sqrtf(sk / (float)nk + eps) : 1.f;
  auto take = [&](int c, float (&r)[V]) {                          // entry c of the q | k row
    if (!buffered) load(c < nq ? col_q + c : col_k + c - nq, r);
    else if constexpr (V == 4) {
      const float4 q4 = *reinterpret_cast<const float4*>(rowbuf + c);
      r[0] = q4.x; r[1] = q4.y; r[2] = q4.z; r[3] = q4.w;
    } else r[0] = rowbuf[c];
  };
  for (int c = threadIdx.x * V; c < nq + nk; c += blockDim.x * V) {
    const bool is_q = c < nq;
    const int cc = is_q ? c : c - nq;
    const int head = cc / dk, i = cc % dk;
    const float* w = is_q ? wq : wk;
    const float inv = is_q ? inv_q : inv_k;
    float x[V];
    take(c, x);
    auto normed = [&](int col, float (&r)[V]) {
      if (!w) return;
      if constexpr (V == 4) {
        const float4 w4 = *reinterpret_cast<const float4*>(w + col);
        r[0] *= inv * w4.x; r[1] *= inv * w4.y; r[2] *= inv * w4.z; r[3] *= inv * w4.w;
      } else r[0] *= inv * w[col];
    };
    normed(cc, x);
    if (i < 2 * n_rot) {                                           // rotated: u' = u cos - v sin, v' = v cos + u sin
      const bool first = pairs ? (i & 1) == 0 : i < n_rot;
      const int f = pairs ? i >> 1 : (first ? i : i - n_rot);
      const int other = pairs ? cc ^ 1 : (first ? cc + n_rot : cc - n_rot);     // heads start at even columns: cc ^ 1 is the partner
      float o[V];
      take(c + other - cc, o);
      normed(other, o);
#pragma unroll
      for (int k = 0; k < V; ++k) {
        x[k] = first ? x[k] * cs[f + k] - o[k] * sn[f + k] : x[k] * cs[f + k] + o[k] * sn[f + k];
      }
    }
    if (is_q) {
      float* d = q_out + t * nq + cc;
      if constexpr (V == 4) *reinterpret_cast<float4*>(d) = make_float4(x[0] * scale, x[1] * scale, x[2] * scale, x[3] * scale);
      else d[0] = x[0] * scale;
    } else if (in_cache) {
      store_cache<T, V>(kcache + ((row * G + head) * Tcap + pos) * dk + i, x);
    }
  }
}

}  // namespace b200p

using namespace b200p;

extern "C" int b200p_row_attn_prep(const float* proj, int64_t ldp, int64_t col_q, int64_t col_k, int64_t col_v, const float* bias,
                                   const float* wq, const float* wk, float eps, const float* rates, int n_rot, float mag, int pairs,
                                   float scale, float temp_coef, float temp_every, const float* v_first, float v_lambda, float* v_keep,
                                   float* q_out, void* kcache, void* vcache, int64_t Tcap, const int32_t* t_row, const int32_t* t_pos,
                                   int64_t M, int H, int G, int dk, int dv, int dtype, void* stream) {
  B200P_REQUIRE(proj && q_out && kcache && vcache && t_row && t_pos, B200P_ERR_ARG, "null pointer");
  B200P_REQUIRE(H > 0 && G > 0 && H % G == 0 && dk > 0 && dv > 0, B200P_ERR_ARG, "bad head geometry");
  B200P_REQUIRE(n_rot >= 0 && 2 * n_rot <= dk && n_rot <= 4096 && (n_rot == 0 || rates), B200P_ERR_ARG, "at most dk dimensions are rotated");
  B200P_REQUIRE(!(pairs && n_rot) || dk % 2 == 0, B200P_ERR_ARG, "pairwise rotation needs heads of an even size");
  B200P_REQUIRE(temp_coef == 0.f || temp_every > 0.f, B200P_ERR_ARG, "the query temperature needs a positive block length");
  if (M == 0) return B200P_OK;
  const bool vec = !pairs && dk % 4 == 0 && dv % 4 == 0 && n_rot % 4 == 0 && ldp % 4 == 0 && col_q % 4 == 0 && col_k % 4 == 0 && col_v % 4 == 0 &&
                   aligned(wq, 16) && aligned(wk, 16) && aligned(kcache, 16) && aligned(vcache, 16) && aligned(proj, 16) &&
                   aligned(bias, 16) && aligned(q_out, 16);
  const size_t turns = 2 * (size_t)n_rot * sizeof(float), row_bytes = (size_t)(H + G) * dk * sizeof(float);
  const int buffered = turns + row_bytes <= 47 * 1024;
  const size_t smem = turns + (buffered ? row_bytes : 0);
  cudaStream_t st = (cudaStream_t)stream;
  if (vec) {
    B200P_DISPATCH_DTYPE(dtype, T, (row_attn_prep_kernel<T, 4><<<(unsigned)M, 256, smem, st>>>(
        proj, ldp, col_q, col_k, col_v, bias, wq, wk, eps, rates, n_rot, mag, pairs, scale, temp_coef,
        temp_every, v_first, v_lambda, v_keep, q_out, (T*)kcache, (T*)vcache, Tcap, t_row, t_pos, H, G, dk, dv, buffered)));
  } else {
    B200P_DISPATCH_DTYPE(dtype, T, (row_attn_prep_kernel<T, 1><<<(unsigned)M, 256, smem, st>>>(
        proj, ldp, col_q, col_k, col_v, bias, wq, wk, eps, rates, n_rot, mag, pairs, scale, temp_coef,
        temp_every, v_first, v_lambda, v_keep, q_out, (T*)kcache, (T*)vcache, Tcap, t_row, t_pos, H, G, dk, dv, buffered)));
  }
  B200P_LAUNCH_CHECK("row_attn_prep_kernel");
  return B200P_OK;
}
