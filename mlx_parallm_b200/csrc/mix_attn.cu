// Attention whose heads' scores are mixed before the softmax: score_h = sum_g talk[h, g] (q_g . k_{kv(g)}), a matrix over the query
// heads of one layer, over a ragged batch with a sliding window and a learned sink per head (one extra term exp(sink_h) in the
// denominator).  Every head's probabilities need every head's raw scores, so one CTA holds all heads of its queries.
//   mix_attn_kernel        one token, all heads, fp32 throughout, any sizes; the keys optionally split over CTAs whose partial
//                          sums attn_merge_kernel combines (decode steps)                                                (per token)
//   mix_attn_tile_kernel   prompts of 16-bit models on mma.sync: 16 query rows per warp, one warp per head (or 8 queries of two
//                          neighbouring heads that share a key/value head); the raw scores meet in shared memory in fp32 and are
//                          mixed by a second matrix product (tf32 with the scores split in two, so that nothing is lost)
//   mix_attn_decode_kernel decode steps of 16-bit models on mma.sync: the heads of a key/value head as rows, keys split over CTAs
// Queries and caches are prepared by row_attn_prep.cu.  Raw and mixed scores and the softmax statistics are fp32; caches and matrix
// operands are in the storage type.
#include "attn_merge.cuh"
#include "common.cuh"
#include "mma_util.cuh"

namespace b200p {

// ---- one token per CTA -----------------------------------------------------------------------------------------------------
constexpr int MX_KEYS = 32;          // keys per chunk: one per lane while scores are formed
constexpr int MX_THREADS = 256;
constexpr int MX_HEADS = 4;          // query heads of one key/value head scored together (they share the key's load)
constexpr int MX_MAX_SPLITS = 16;
constexpr int MX_SMEM_MAX = 227 * 1024;

// CTA = (share of the keys blockIdx.x of gridDim.x, token blockIdx.y).  VEC elements per 16-byte piece of a cache row (1: rows that
// are not whole pieces).  kv_block key heads are staged at a time.  part_o NULL: the whole softmax, sink included, into `out`.
template <typename T, int VEC>
__global__ void __launch_bounds__(MX_THREADS)
mix_attn_kernel(const float* __restrict__ q, const T* __restrict__ kcache, const T* __restrict__ vcache, int64_t Tcap,
                const int32_t* __restrict__ t_row, const int32_t* __restrict__ t_pos, const float* __restrict__ talk,
                const float* __restrict__ sink, int64_t window, T* __restrict__ out, int64_t ld_out, int H, int G, int dk, int dv,
                float* __restrict__ part_o, float* __restrict__ part_ms, int kv_block) {
  extern __shared__ __align__(16) uint8_t mx_smem[];
  const int per = H / G, KP = VEC > 1 ? dk + VEC : dk + 1;          // padded key row
  T* kst = reinterpret_cast<T*>(mx_smem);                            // [kv_block][MX_KEYS][KP]
  float* qs = reinterpret_cast<float*>(mx_smem + ((size_t)kv_block * MX_KEYS * KP * sizeof(T) + 15) / 16 * 16);   // [H][dk]
  float* acc = qs + H * dk;                                          // [H][dv]
  float* tk = acc + H * dv;                                          // [H][H]
  float* raw = tk + H * H;                                           // [H][MX_KEYS]
  float* pr = raw + H * MX_KEYS;                                     // [H][MX_KEYS]
  float* m_s = pr + H * MX_KEYS;                                     // [H] each: running max, sum, this chunk's rescale factor
  float* l_s = m_s + H;
  float* c_s = l_s + H;
  const int64_t t = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = MX_THREADS / 32;
  const int64_t pos = t_pos[t];
  const T* kb = kcache + (int64_t)t_row[t] * G * Tcap * dk;
  const T* vb = vcache + (int64_t)t_row[t] * G * Tcap * dv;
  const bool whole = part_o == nullptr;
  for (int i = threadIdx.x; i < H * dk; i += MX_THREADS) qs[i] = q[t * H * dk + i];
  for (int i = threadIdx.x; i < H * dv; i += MX_THREADS) acc[i] = 0.f;
  for (int i = threadIdx.x; i < H * H; i += MX_THREADS) tk[i] = talk[i];
  for (int h = threadIdx.x; h < H; h += MX_THREADS) {
    m_s[h] = whole && sink ? sink[h] : -INFINITY;
    l_s[h] = whole && sink ? 1.f : 0.f;
  }
  const int64_t lo = (window > 0 && pos - window + 1 > 0) ? pos - window + 1 : 0;
  const int64_t chunks = (pos - lo) / MX_KEYS + 1, share = (chunks + gridDim.x - 1) / gridDim.x;
  const int64_t c_lo = blockIdx.x * share, c_hi = min(chunks, c_lo + share);
  for (int64_t ci = c_lo; ci < c_hi; ++ci) {
    const int64_t j0 = lo + ci * MX_KEYS;
    const int nk = (int)min((int64_t)MX_KEYS, pos + 1 - j0);
    for (int g0 = 0; g0 < G; g0 += kv_block) {
      const int ng = min(kv_block, G - g0);
      __syncthreads();                                               // the staged keys and the raw scores of the last round are used up
      if constexpr (VEC > 1) {
        const int pieces = dk / VEC;
        for (int idx = threadIdx.x; idx < ng * MX_KEYS * pieces; idx += MX_THREADS) {
          const int p = idx % pieces, kk = (idx / pieces) % MX_KEYS, gl = idx / (pieces * MX_KEYS);
          const bool ok = kk < nk;
          cp_async16((uint32_t)__cvta_generic_to_shared(kst + ((size_t)gl * MX_KEYS + kk) * KP + p * VEC),
                     kb + ((int64_t)(g0 + gl) * Tcap + j0 + (ok ? kk : 0)) * dk + p * VEC, ok);
        }
        cp_async_commit();
        cp_async_wait<0>();
      } else {
        for (int idx = threadIdx.x; idx < ng * MX_KEYS * dk; idx += MX_THREADS) {
          const int i = idx % dk, kk = (idx / dk) % MX_KEYS, gl = idx / (dk * MX_KEYS);
          kst[((size_t)gl * MX_KEYS + kk) * KP + i] = kk < nk ? kb[((int64_t)(g0 + gl) * Tcap + j0 + kk) * dk + i] : Tr<T>::from_f(0.f);
        }
      }
      __syncthreads();
      const int blocks = (per + MX_HEADS - 1) / MX_HEADS;
      for (int it = warp; it < ng * blocks; it += nw) {
        const int gl = it / blocks, h0 = (it % blocks) * MX_HEADS;   // heads h0 .. of the key head, some of which may not exist
        const T* kr = kst + ((size_t)gl * MX_KEYS + lane) * KP;
        const float* qr[MX_HEADS];
        float d[MX_HEADS];
#pragma unroll
        for (int k = 0; k < MX_HEADS; ++k) {
          qr[k] = qs + (size_t)((g0 + gl) * per + min(h0 + k, per - 1)) * dk;
          d[k] = 0.f;
        }
        for (int i = 0; i < dk; i += VEC) {
          float kv[VEC];
          if constexpr (VEC > 1) {
            const uint4 u = *reinterpret_cast<const uint4*>(kr + i);
            const T* e = reinterpret_cast<const T*>(&u);
#pragma unroll
            for (int k = 0; k < VEC; ++k) kv[k] = Tr<T>::to_f(e[k]);
          } else {
            kv[0] = Tr<T>::to_f(kr[i]);
          }
#pragma unroll
          for (int k = 0; k < MX_HEADS; ++k)
#pragma unroll
            for (int x = 0; x < VEC; ++x) d[k] = fmaf(qr[k][i + x], kv[x], d[k]);
        }
#pragma unroll
        for (int k = 0; k < MX_HEADS; ++k)
          if (h0 + k < per) raw[((g0 + gl) * per + h0 + k) * MX_KEYS + lane] = d[k];
      }
    }
    __syncthreads();
    for (int h = warp; h < H; h += nw) {                             // mix and soften: lane = key
      float s = 0.f;
      for (int g = 0; g < H; ++g) s = fmaf(tk[h * H + g], raw[g * MX_KEYS + lane], s);
      if (lane >= nk) s = -INFINITY;
      const float mo = m_s[h], mn = fmaxf(mo, warp_max(s));          // finite: every chunk holds a visible key
      const float p = lane < nk ? expf(s - mn) : 0.f, sum = warp_sum(p), corr = expf(mo - mn);
      pr[h * MX_KEYS + lane] = p;
      __syncwarp();
      if (lane == 0) { m_s[h] = mn; l_s[h] = l_s[h] * corr + sum; c_s[h] = corr; }
    }
    __syncthreads();
    const int vpieces = dv / VEC;
    for (int idx = threadIdx.x; idx < H * vpieces; idx += MX_THREADS) {
      const int h = idx / vpieces, p = idx % vpieces;
      float a[VEC];
      const float corr = c_s[h];
#pragma unroll
      for (int x = 0; x < VEC; ++x) a[x] = acc[h * dv + p * VEC + x] * corr;
      const T* vr = vb + ((int64_t)(h / per) * Tcap + j0) * dv + p * VEC;
#pragma unroll 8
      for (int kk = 0; kk < nk; ++kk) {
        const float w = pr[h * MX_KEYS + kk];
        if constexpr (VEC > 1) {
          const uint4 u = *reinterpret_cast<const uint4*>(vr + (int64_t)kk * dv);
          const T* e = reinterpret_cast<const T*>(&u);
#pragma unroll
          for (int x = 0; x < VEC; ++x) a[x] = fmaf(w, Tr<T>::to_f(e[x]), a[x]);
        } else {
          a[0] = fmaf(w, Tr<T>::to_f(vr[(int64_t)kk * dv]), a[0]);
        }
      }
#pragma unroll
      for (int x = 0; x < VEC; ++x) acc[h * dv + p * VEC + x] = a[x];
    }
  }
  __syncthreads();
  if (whole) {
    for (int i = threadIdx.x; i < H * dv; i += MX_THREADS) out[t * ld_out + i] = Tr<T>::from_f(acc[i] / l_s[i / dv]);
    return;
  }
  for (int h = threadIdx.x; h < H; h += MX_THREADS) {
    float* ms = part_ms + ((t * H + h) * gridDim.x + blockIdx.x) * 2;
    ms[0] = m_s[h] * LOG2E;                                          // a share without keys leaves (-inf, 0)
    ms[1] = l_s[h];
  }
  if (c_lo < c_hi)
    for (int i = threadIdx.x; i < H * dv; i += MX_THREADS)
      part_o[((t * H + i / dv) * gridDim.x + blockIdx.x) * dv + i % dv] = acc[i];
}

// ---- prompts on the tensor cores ---------------------------------------------------------------------------------------------
__device__ __forceinline__ void mma1688_tf32(float (&d)[4], const float4& a, float b0, float b1) {
  asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(__float_as_uint(a.x)), "r"(__float_as_uint(a.y)), "r"(__float_as_uint(a.z)), "r"(__float_as_uint(a.w)),
                 "r"(__float_as_uint(b0)), "r"(__float_as_uint(b1)));
}
// x = hi + lo: hi the leading 11 bits (what tf32 keeps), lo the rest, of which tf32 keeps 11 more
__device__ __forceinline__ float tf32_head(float x) { return __uint_as_float(__float_as_uint(x) & 0xffffe000u); }
__device__ __forceinline__ float ex2_approx(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }

// `talk` as the A operand of the mixing product, in the order a lane's registers want it: [row block][8-head step][lane] float4
__device__ __forceinline__ void stage_talk(const float* __restrict__ talk, float4* frag, int mb_n, int ks_n, int H, int tid, int nt) {
  for (int i = tid; i < mb_n * ks_n * 32; i += nt) {
    const int lane = i & 31, s = (i >> 5) % ks_n, mb = (i >> 5) / ks_n;
    const int r = mb * 16 + (lane >> 2), c = s * 8 + (lane & 3);
    auto at = [&](int a, int b) { return (a < H && b < H) ? talk[a * H + b] : 0.f; };
    frag[i] = make_float4(at(r, c), at(r + 8, c), at(r, c + 4), at(r + 8, c + 4));
  }
}

constexpr int MT_MAX_WARPS = 16;
constexpr int MT_PAD = 16;           // bytes behind every staged row: ldmatrix then reads 8 rows without bank conflicts

// shared floats: one head's raw scores (QB queries x KT keys; the paddings keep fragment accesses free of bank conflicts)
constexpr int mt_pitch(int kt) { return kt + 8; }
constexpr int mt_head(int hb, int kt) { return 16 / hb * mt_pitch(kt) + 8; }
static size_t mt_smem(int H, int G, int dk, int dv, int hb, int kt) {
  const int hp = (H + 7) / 8 * 8;
  return (size_t)G * kt * ((dk + dv) * 2 + 2 * MT_PAD) + (size_t)hp * mt_head(hb, kt) * 4 + (size_t)hb * 2 * hb * 32 * 16;
}

// CTA = QB = 16 / HB consecutive queries of entry blockIdx.y, all H heads; warp w owns the heads w HB .. w HB + HB-1 (HB = 2: two
// heads of one key/value head fill the 16 rows of a fragment with 8 queries each).  The last query tiles, which see the most
// keys, start first.  Per chunk of KT keys:
//   raw scores of the warp's heads -> shared; all heads of 8 key positions at a time mixed in place by any warp; mixed scores of
//   the warp's heads -> window, online softmax in registers (base-2 units, opened by the sink), O += P V.
// Keys and values of all key/value heads sit in one buffer each: values arrive while scores are formed, the next keys while
// scores are mixed and values multiplied.
template <typename T, int DK, int DV, int HB, int KT>
__global__ void __launch_bounds__(MT_MAX_WARPS * 32, 1)
mix_attn_tile_kernel(const float* __restrict__ q, const T* __restrict__ kc, const T* __restrict__ vc, int64_t Tcap,
                     const int32_t* __restrict__ cu, const int32_t* __restrict__ rows, const int32_t* __restrict__ t_pos,
                     const float* __restrict__ talk, const float* __restrict__ sink, int window, T* __restrict__ out, int64_t ld_out,
                     int H, int G) {
  constexpr int QB = 16 / HB, PITCH = mt_pitch(KT), HS = mt_head(HB, KT), MB = HB, KS = 2 * HB;
  constexpr int KROW = DK * 2 + MT_PAD, VROW = DV * 2 + MT_PAD, KCH = DK / 8, VCH = DV / 8;
  extern __shared__ __align__(128) uint8_t mt_sm[];
  const int e = blockIdx.y;
  const int t_first = cu[e], n_e = cu[e + 1] - t_first;
  const int q0 = (gridDim.x - 1 - blockIdx.x) * QB;
  if (q0 >= n_e) return;                                             // the same for every thread of the CTA
  const int NT = blockDim.x, NW = NT >> 5;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, quad_row = lane >> 2, qc = lane & 3;
  const int HP = (H + 7) / 8 * 8;
  const int h0 = warp * HB, h1 = HB == 2 ? h0 + 1 : h0;              // heads of the fragment's rows 0-7 and 8-15
  const int g = h0 / (H / G);
  const int l0 = q0 + quad_row, l1 = HB == 2 ? l0 : l0 + 8;          // the rows' queries (offsets in the entry)
  const int lc0 = min(l0, n_e - 1), lc1 = min(l1, n_e - 1);          // rows past the end compute a valid row, not stored
  const int p_first = t_pos[t_first];                                // positions of an entry's tokens are consecutive
  const int kend = p_first + min(n_e, q0 + QB);                      // keys any row of this CTA may see
  const int first = window > 0 ? p_first + q0 - window + 1 : 0;      // the first key the CTA's first row sees
  const int tile_lo = first > 0 ? first / KT : 0, tile_hi = (kend + KT - 1) / KT;
  const uint32_t ks = (uint32_t)__cvta_generic_to_shared(mt_sm), vs = ks + G * KT * KROW;
  float* raw = reinterpret_cast<float*>(mt_sm + (size_t)G * KT * (KROW + VROW));      // [HP][HS]
  float4* tfrag = reinterpret_cast<float4*>(raw + HP * HS);
  for (int i = threadIdx.x; i < (HP - H) * HS; i += NT) raw[H * HS + i] = 0.f;        // padded heads meet zero weights: keep them finite
  stage_talk(talk, tfrag, MB, KS, H, threadIdx.x, NT);

  uint32_t qf[DK / 16][4];
  {
    const float* p0 = q + ((int64_t)(t_first + lc0) * H + h0) * DK;
    const float* p1 = q + ((int64_t)(t_first + lc1) * H + h1) * DK;
#pragma unroll
    for (int s = 0; s < DK / 16; ++s) {
      const float2 a0 = *reinterpret_cast<const float2*>(p0 + s * 16 + 2 * qc), a1 = *reinterpret_cast<const float2*>(p1 + s * 16 + 2 * qc);
      const float2 b0 = *reinterpret_cast<const float2*>(p0 + s * 16 + 8 + 2 * qc), b1 = *reinterpret_cast<const float2*>(p1 + s * 16 + 8 + 2 * qc);
      qf[s][0] = pack2<T>(a0.x, a0.y);
      qf[s][1] = pack2<T>(a1.x, a1.y);
      qf[s][2] = pack2<T>(b0.x, b0.y);
      qf[s][3] = pack2<T>(b1.x, b1.y);
    }
  }
  // a thread stages the same 16-byte column of every NT / pieces-th row; rows past the last visible key repeat that key's row
  // (they are masked, and their values must be finite)
  const uint32_t cap = (uint32_t)Tcap;
  const int64_t row_off = (int64_t)rows[e] * G * Tcap;
  const T* kcol = kc + row_off * DK + (threadIdx.x % KCH) * 8;
  const T* vcol = vc + row_off * DV + (threadIdx.x % VCH) * 8;
  auto load_keys = [&](int tile) {
    const int key0 = tile * KT;
    for (int r = threadIdx.x / KCH; r < G * KT; r += NT / KCH)
      cp_async16(ks + r * KROW + (threadIdx.x % KCH) * 16, kcol + ((uint32_t)(r / KT) * cap + (uint32_t)min(key0 + r % KT, kend - 1)) * DK, true);
  };
  auto load_values = [&](int tile) {
    const int key0 = tile * KT;
    for (int r = threadIdx.x / VCH; r < G * KT; r += NT / VCH)
      cp_async16(vs + r * VROW + (threadIdx.x % VCH) * 16, vcol + ((uint32_t)(r / KT) * cap + (uint32_t)min(key0 + r % KT, kend - 1)) * DV, true);
  };

  float o[DV / 8][4];
#pragma unroll
  for (int j = 0; j < DV / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  // the sink opens the softmax: it is the running maximum, and its own term (one) sits in the sum of one thread of the quad
  float m0 = sink ? sink[h0] * LOG2E : -INFINITY, m1 = sink ? sink[h1] * LOG2E : -INFINITY;
  float s0 = (sink && qc == 0) ? 1.f : 0.f, s1 = s0;
  const int wnd = window > 0 ? window : 0x7fffffff;
  // per-lane ldmatrix bases: everything that changes with the unrolled loops is a constant offset
  const uint32_t kl = ks + g * KT * KROW + ((lane & 7) + ((lane >> 4) << 3)) * KROW + ((lane >> 3) & 1) * 16;
  const uint32_t vl = vs + g * KT * VROW + (lane & 15) * VROW + (lane >> 4) * 16;
  float* raw0 = raw + h0 * HS + quad_row * PITCH + 2 * qc;           // this thread's two fragment rows
  float* raw1 = HB == 2 ? raw0 + HS : raw0 + 8 * PITCH;

  load_keys(tile_lo);
  cp_async_commit();
  for (int it = tile_lo; it < tile_hi; ++it) {
    cp_async_wait<0>();                                              // this chunk's keys
    __syncthreads();                                                 // ... of every thread; the last chunk's values and scores are used up
    load_values(it);
    cp_async_commit();
    float sc[KT / 8][4];
#pragma unroll
    for (int nt = 0; nt < KT / 8; ++nt) sc[nt][0] = sc[nt][1] = sc[nt][2] = sc[nt][3] = 0.f;
#pragma unroll
    for (int s = 0; s < DK / 16; ++s) {
#pragma unroll
      for (int np = 0; np < KT / 16; ++np) {
        uint32_t bf[4];
        ldsm_x4(kl + np * 16 * KROW + s * 32, bf);
        mma16816<T>(sc[2 * np], qf[s], bf[0], bf[1]);
        mma16816<T>(sc[2 * np + 1], qf[s], bf[2], bf[3]);
      }
    }
#pragma unroll
    for (int nt = 0; nt < KT / 8; ++nt) {
      *reinterpret_cast<float2*>(raw0 + 8 * nt) = make_float2(sc[nt][0], sc[nt][1]);
      *reinterpret_cast<float2*>(raw1 + 8 * nt) = make_float2(sc[nt][2], sc[nt][3]);
    }
    __syncthreads();                                                 // raw scores of all heads; the keys are used up
    if (it + 1 < tile_hi) load_keys(it + 1);
    cp_async_commit();
    // mixed = talk x raw, twice 8 key positions of one query (columns) at a time, heads as rows and as the summed index
    for (int nt = warp; nt < QB * KT / 16; nt += NW) {
      float* base = raw + (nt / (KT / 16)) * PITCH + (nt % (KT / 16)) * 16;
      float c[2][MB][4];
#pragma unroll
      for (int i = 0; i < 2 * MB; ++i) c[i / MB][i % MB][0] = c[i / MB][i % MB][1] = c[i / MB][i % MB][2] = c[i / MB][i % MB][3] = 0.f;
#pragma unroll
      for (int s = 0; s < KS; ++s) {
        if (s * 8 < HP) {
          const float* b = base + (s * 8 + qc) * HS + quad_row;
          const float x00 = b[0], x01 = b[4 * HS], x10 = b[8], x11 = b[4 * HS + 8];
          const float g00 = tf32_head(x00), g01 = tf32_head(x01), g10 = tf32_head(x10), g11 = tf32_head(x11);
          const float r00 = x00 - g00, r01 = x01 - g01, r10 = x10 - g10, r11 = x11 - g11;
#pragma unroll
          for (int mb = 0; mb < MB; ++mb) {
            const float4 a = tfrag[(mb * KS + s) * 32 + lane];
            mma1688_tf32(c[0][mb], a, r00, r01);
            mma1688_tf32(c[1][mb], a, r10, r11);
            mma1688_tf32(c[0][mb], a, g00, g01);
            mma1688_tf32(c[1][mb], a, g10, g11);
          }
        }
      }
      __syncwarp();                                                  // every lane has read these positions
#pragma unroll
      for (int mb = 0; mb < MB; ++mb) {
        const int ha = mb * 16 + quad_row, hb = ha + 8;
        float* d = base + ha * HS + 2 * qc;
        if (ha < H) { *reinterpret_cast<float2*>(d) = make_float2(c[0][mb][0], c[0][mb][1]); *reinterpret_cast<float2*>(d + 8) = make_float2(c[1][mb][0], c[1][mb][1]); }
        d += 8 * HS;
        if (hb < H) { *reinterpret_cast<float2*>(d) = make_float2(c[0][mb][2], c[0][mb][3]); *reinterpret_cast<float2*>(d + 8) = make_float2(c[1][mb][2], c[1][mb][3]); }
      }
    }
    cp_async_wait<1>();                                              // the values (the next keys may still be on their way)
    __syncthreads();                                                 // ... of every thread, and the mixed scores
#pragma unroll
    for (int nt = 0; nt < KT / 8; ++nt) {
      const float2 a = *reinterpret_cast<const float2*>(raw0 + 8 * nt), b = *reinterpret_cast<const float2*>(raw1 + 8 * nt);
      sc[nt][0] = a.x; sc[nt][1] = a.y; sc[nt][2] = b.x; sc[nt][3] = b.y;
    }
    const int key0 = it * KT;
    if (key0 + KT - 1 > p_first + q0 || kend - 1 - key0 >= wnd) {    // some row of the CTA does not see some key of this chunk
      const int d0 = p_first + lc0 - key0 - 2 * qc, d1 = p_first + lc1 - key0 - 2 * qc;
#pragma unroll
      for (int nt = 0; nt < KT / 8; ++nt) {
        if ((unsigned)(d0 - 8 * nt) >= (unsigned)wnd) sc[nt][0] = -INFINITY;           // outside 0 <= distance < window
        if ((unsigned)(d0 - 8 * nt - 1) >= (unsigned)wnd) sc[nt][1] = -INFINITY;
        if ((unsigned)(d1 - 8 * nt) >= (unsigned)wnd) sc[nt][2] = -INFINITY;
        if ((unsigned)(d1 - 8 * nt - 1) >= (unsigned)wnd) sc[nt][3] = -INFINITY;
      }
    }
    float t0 = -INFINITY, t1 = -INFINITY;
#pragma unroll
    for (int nt = 0; nt < KT / 8; ++nt) {
      t0 = fmaxf(t0, fmaxf(sc[nt][0], sc[nt][1]));
      t1 = fmaxf(t1, fmaxf(sc[nt][2], sc[nt][3]));
    }
    t0 = fmaxf(t0, __shfl_xor_sync(0xffffffffu, t0, 1)); t0 = fmaxf(t0, __shfl_xor_sync(0xffffffffu, t0, 2));
    t1 = fmaxf(t1, __shfl_xor_sync(0xffffffffu, t1, 1)); t1 = fmaxf(t1, __shfl_xor_sync(0xffffffffu, t1, 2));
    const float keep0 = fmaxf(m0, t0 * LOG2E), keep1 = fmaxf(m1, t1 * LOG2E);
    if (__any_sync(0xffffffffu, keep0 != m0 || keep1 != m1)) {       // a running maximum moved: rescale what there is
      const float corr0 = keep0 == m0 ? 1.f : ex2_approx(m0 - keep0), corr1 = keep1 == m1 ? 1.f : ex2_approx(m1 - keep1);
      m0 = keep0; m1 = keep1;
      s0 *= corr0;
      s1 *= corr1;
#pragma unroll
      for (int j = 0; j < DV / 8; ++j) { o[j][0] *= corr0; o[j][1] *= corr0; o[j][2] *= corr1; o[j][3] *= corr1; }
    }
    // nothing seen yet (the row's window begins later and there is no sink): exponentials against 0
    const float mn0 = m0 == -INFINITY ? 0.f : m0, mn1 = m1 == -INFINITY ? 0.f : m1;
#pragma unroll
    for (int nt = 0; nt < KT / 8; ++nt) {
      sc[nt][0] = ex2_approx(fmaf(sc[nt][0], LOG2E, -mn0)); sc[nt][1] = ex2_approx(fmaf(sc[nt][1], LOG2E, -mn0));
      sc[nt][2] = ex2_approx(fmaf(sc[nt][2], LOG2E, -mn1)); sc[nt][3] = ex2_approx(fmaf(sc[nt][3], LOG2E, -mn1));
      s0 += sc[nt][0] + sc[nt][1];
      s1 += sc[nt][2] + sc[nt][3];
    }
#pragma unroll
    for (int kk = 0; kk < KT / 16; ++kk) {
      uint32_t pf[4];
      pf[0] = pack2<T>(sc[2 * kk][0], sc[2 * kk][1]);
      pf[1] = pack2<T>(sc[2 * kk][2], sc[2 * kk][3]);
      pf[2] = pack2<T>(sc[2 * kk + 1][0], sc[2 * kk + 1][1]);
      pf[3] = pack2<T>(sc[2 * kk + 1][2], sc[2 * kk + 1][3]);
#pragma unroll
      for (int jp = 0; jp < DV / 16; ++jp) {
        uint32_t bf[4];
        ldsm_x4_trans(vl + kk * 16 * VROW + jp * 32, bf);
        mma16816<T>(o[2 * jp], pf, bf[0], bf[1]);
        mma16816<T>(o[2 * jp + 1], pf, bf[2], bf[3]);
      }
    }
  }
  cp_async_wait<0>();
  s0 += __shfl_xor_sync(0xffffffffu, s0, 1); s0 += __shfl_xor_sync(0xffffffffu, s0, 2);
  s1 += __shfl_xor_sync(0xffffffffu, s1, 1); s1 += __shfl_xor_sync(0xffffffffu, s1, 2);
  const float inv0 = 1.f / s0, inv1 = 1.f / s1;
  T* o0 = out + (int64_t)(t_first + lc0) * ld_out + (int64_t)h0 * DV;
  T* o1 = out + (int64_t)(t_first + lc1) * ld_out + (int64_t)h1 * DV;
#pragma unroll
  for (int j = 0; j < DV / 8; ++j) {
    const int c = 8 * j + 2 * qc;
    if (l0 < n_e) *reinterpret_cast<uint32_t*>(o0 + c) = pack2<T>(o[j][0] * inv0, o[j][1] * inv0);
    if (l1 < n_e) *reinterpret_cast<uint32_t*>(o1 + c) = pack2<T>(o[j][2] * inv1, o[j][3] * inv1);
  }
}

// ---- decode steps on the tensor cores --------------------------------------------------------------------------------------------
// CTA = (share of the keys blockIdx.x of gridDim.x, token blockIdx.y), 8 warps.  Rows of a fragment are the query heads of one
// key/value head.  Per chunk of KT keys: raw scores (warp = key/value head x 16 keys) -> mixed scores (warp = 8 keys x 16 heads)
// -> softmax statistics and probabilities (warp = head, lane = key) -> O += P V (warp = key/value head x 64 value columns).  The
// partial sums go to attn_merge_kernel, which adds the sink.
constexpr int MD_WARPS = 8, MD_THREADS = MD_WARPS * 32;
static size_t md_smem(int H, int G, int dk, int dv, int kt) {
  const int hp = (H + 7) / 8 * 8, mb = (H + 15) / 16;
  return (size_t)G * kt * ((dk + dv) * 2 + 2 * MT_PAD) + (size_t)H * (dk * 2 + MT_PAD) + (size_t)H * (kt * 2 + MT_PAD) +
         2 * (size_t)hp * mt_pitch(kt) * 4 + (size_t)mb * 2 * mb * 32 * 16 + 3 * (size_t)hp * 4;
}

template <typename T, int DK, int DV, int MB, int KT, int ITEMS>
__global__ void __launch_bounds__(MD_THREADS)
mix_attn_decode_kernel(const float* __restrict__ q, const T* __restrict__ kc, const T* __restrict__ vc, int64_t Tcap,
                       const int32_t* __restrict__ t_row, const int32_t* __restrict__ t_pos, const float* __restrict__ talk, int64_t window,
                       int H, int G, float* __restrict__ part_o, float* __restrict__ part_ms) {
  constexpr int KROW = DK * 2 + MT_PAD, VROW = DV * 2 + MT_PAD, PROW = KT * 2 + MT_PAD, PITCH = mt_pitch(KT), KS = 2 * MB, KCH = DK / 8, VCH = DV / 8;
  extern __shared__ __align__(128) uint8_t mt_sm[];
  const int64_t t = blockIdx.y;
  const int per = H / G, HP = (H + 7) / 8 * 8;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, quad_row = lane >> 2, qc = lane & 3;
  const uint32_t sm = (uint32_t)__cvta_generic_to_shared(mt_sm);
  const uint32_t ks = sm, vs = ks + G * KT * KROW, qs = vs + G * KT * VROW, ps = qs + H * KROW;
  uint8_t* after = mt_sm + (size_t)G * KT * (KROW + VROW) + (size_t)H * (KROW + PROW);
  float4* tfrag = reinterpret_cast<float4*>(after);
  float* raw = reinterpret_cast<float*>(tfrag + MB * KS * 32);       // [HP][PITCH]
  float* mixed = raw + HP * PITCH;                                   // [HP][PITCH]
  float* m_s = mixed + HP * PITCH;                                   // [HP] each
  float* l_s = m_s + HP;
  float* c_s = l_s + HP;
  T* qsm = reinterpret_cast<T*>(mt_sm + (size_t)G * KT * (KROW + VROW));
  T* psm = reinterpret_cast<T*>(mt_sm + (size_t)G * KT * (KROW + VROW) + (size_t)H * KROW);
  const int pos = t_pos[t];
  const int lo = (window > 0 && pos - window + 1 > 0) ? (int)(pos - window + 1) : 0;
  const int chunks = (pos - lo) / KT + 1, share = (chunks + gridDim.x - 1) / gridDim.x;
  const int c_lo = blockIdx.x * share, c_hi = min(chunks, c_lo + share);
  const uint32_t cap = (uint32_t)Tcap;
  const int64_t row_off = (int64_t)t_row[t] * G * Tcap;
  const T* kcol = kc + row_off * DK + (threadIdx.x % KCH) * 8;
  const T* vcol = vc + row_off * DV + (threadIdx.x % VCH) * 8;
  auto load_keys = [&](int ci) {
    const int j0 = lo + ci * KT;
    for (int r = threadIdx.x / KCH; r < G * KT; r += MD_THREADS / KCH)
      cp_async16(ks + r * KROW + (threadIdx.x % KCH) * 16, kcol + ((uint32_t)(r / KT) * cap + (uint32_t)min(j0 + r % KT, pos)) * DK, true);
  };
  auto load_values = [&](int ci) {
    const int j0 = lo + ci * KT;
    for (int r = threadIdx.x / VCH; r < G * KT; r += MD_THREADS / VCH)
      cp_async16(vs + r * VROW + (threadIdx.x % VCH) * 16, vcol + ((uint32_t)(r / KT) * cap + (uint32_t)min(j0 + r % KT, pos)) * DV, true);
  };
  if (c_lo < c_hi) load_keys(c_lo);
  cp_async_commit();
  for (int i = threadIdx.x; i < H * (DK / 2); i += MD_THREADS) {
    const float2 v = *reinterpret_cast<const float2*>(q + t * H * DK + 2 * i);
    *reinterpret_cast<uint32_t*>(reinterpret_cast<uint8_t*>(qsm) + (i / (DK / 2)) * KROW + (i % (DK / 2)) * 4) = pack2<T>(v.x, v.y);
  }
  stage_talk(talk, tfrag, MB, KS, H, threadIdx.x, MD_THREADS);
  for (int i = threadIdx.x; i < (HP - H) * PITCH; i += MD_THREADS) raw[H * PITCH + i] = 0.f;     // padded heads meet zero weights
  for (int i = threadIdx.x; i < HP; i += MD_THREADS) { m_s[i] = -INFINITY; l_s[i] = 0.f; c_s[i] = 1.f; }

  float o[ITEMS][8][4];
#pragma unroll
  for (int i = 0; i < ITEMS; ++i)
#pragma unroll
    for (int j = 0; j < 8; ++j) o[i][j][0] = o[i][j][1] = o[i][j][2] = o[i][j][3] = 0.f;
  const int frow = min(lane & 15, per - 1);                          // this lane's ldmatrix row among the heads of a key/value head
  const int r0 = min(quad_row, per - 1), r1 = min(quad_row + 8, per - 1);

  for (int ci = c_lo; ci < c_hi; ++ci) {
    cp_async_wait<0>();
    __syncthreads();                                                 // this chunk's keys; the last chunk's values and probabilities are used up
    load_values(ci);
    cp_async_commit();
    for (int item = warp; item < G * (KT / 16); item += MD_WARPS) {
      const int g = item / (KT / 16), kb = item % (KT / 16);
      const uint32_t qa = qs + (g * per + frow) * KROW + (lane >> 4) * 16;
      const uint32_t ka = ks + (g * KT + kb * 16 + (lane & 7) + ((lane >> 4) << 3)) * KROW + ((lane >> 3) & 1) * 16;
      float sc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
      for (int s = 0; s < DK / 16; ++s) {
        uint32_t af[4], bf[4];
        ldsm_x4(qa + s * 32, af);
        ldsm_x4(ka + s * 32, bf);
        mma16816<T>(sc[0], af, bf[0], bf[1]);
        mma16816<T>(sc[1], af, bf[2], bf[3]);
      }
      float* d = raw + (g * per + quad_row) * PITCH + kb * 16 + 2 * qc;
      if (quad_row < per) { *reinterpret_cast<float2*>(d) = make_float2(sc[0][0], sc[0][1]); *reinterpret_cast<float2*>(d + 8) = make_float2(sc[1][0], sc[1][1]); }
      d += 8 * PITCH;
      if (quad_row + 8 < per) { *reinterpret_cast<float2*>(d) = make_float2(sc[0][2], sc[0][3]); *reinterpret_cast<float2*>(d + 8) = make_float2(sc[1][2], sc[1][3]); }
    }
    __syncthreads();                                                 // raw scores; the keys are used up
    if (ci + 1 < c_hi) load_keys(ci + 1);
    cp_async_commit();
    for (int item = warp; item < KT / 8 * MB; item += MD_WARPS) {
      const int nt = item / MB, mb = item % MB;
      float c[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int s = 0; s < KS; ++s) {
        if (s * 8 < HP) {
          const float* b = raw + (s * 8 + qc) * PITCH + nt * 8 + quad_row;
          const float x0 = b[0], x1 = b[4 * PITCH], g0 = tf32_head(x0), g1 = tf32_head(x1);
          const float4 a = tfrag[(mb * KS + s) * 32 + lane];
          mma1688_tf32(c, a, x0 - g0, x1 - g1);
          mma1688_tf32(c, a, g0, g1);
        }
      }
      const int ha = mb * 16 + quad_row;
      float* d = mixed + ha * PITCH + nt * 8 + 2 * qc;
      if (ha < H) *reinterpret_cast<float2*>(d) = make_float2(c[0], c[1]);
      if (ha + 8 < H) *reinterpret_cast<float2*>(d + 8 * PITCH) = make_float2(c[2], c[3]);
    }
    __syncthreads();
    const int nk = min(KT, pos + 1 - lo - ci * KT);                  // at least one: finite maxima
    for (int h = warp; h < H; h += MD_WARPS) {
      const float s = lane < nk ? mixed[h * PITCH + lane] * LOG2E : -INFINITY;
      const float mo = m_s[h], mn = fmaxf(mo, warp_max(s));
      const float p = lane < nk ? exp2f(s - mn) : 0.f, sum = warp_sum(p), corr = exp2f(mo - mn);
      if (lane < KT) *reinterpret_cast<T*>(reinterpret_cast<uint8_t*>(psm) + h * PROW + lane * 2) = Tr<T>::from_f(p);
      __syncwarp();
      if (lane == 0) { m_s[h] = mn; l_s[h] = l_s[h] * corr + sum; c_s[h] = corr; }
    }
    cp_async_wait<1>();                                              // the values (the next keys may still be on their way)
    __syncthreads();
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      const int item = warp + i * MD_WARPS;
      if (item < G * (DV / 64)) {
        const int g = item / (DV / 64), cb = item % (DV / 64);
        const float c0 = c_s[g * per + r0], c1 = c_s[g * per + r1];
#pragma unroll
        for (int j = 0; j < 8; ++j) { o[i][j][0] *= c0; o[i][j][1] *= c0; o[i][j][2] *= c1; o[i][j][3] *= c1; }
        const uint32_t pa = ps + (g * per + frow) * PROW + (lane >> 4) * 16;
        const uint32_t va = vs + (g * KT + (lane & 15)) * VROW + (lane >> 4) * 16 + cb * 128;
#pragma unroll
        for (int kk = 0; kk < KT / 16; ++kk) {
          uint32_t af[4];
          ldsm_x4(pa + kk * 32, af);
#pragma unroll
          for (int jp = 0; jp < 4; ++jp) {
            uint32_t bf[4];
            ldsm_x4_trans(va + kk * 16 * VROW + jp * 32, bf);
            mma16816<T>(o[i][2 * jp], af, bf[0], bf[1]);
            mma16816<T>(o[i][2 * jp + 1], af, bf[2], bf[3]);
          }
        }
      }
    }
  }
  cp_async_wait<0>();
  __syncthreads();
  for (int h = threadIdx.x; h < H; h += MD_THREADS) {
    float* ms = part_ms + ((t * H + h) * gridDim.x + blockIdx.x) * 2;
    ms[0] = m_s[h];                                                  // base-2 units; a share without keys leaves (-inf, 0)
    ms[1] = l_s[h];
  }
  if (c_lo >= c_hi) return;
#pragma unroll
  for (int i = 0; i < ITEMS; ++i) {
    const int item = warp + i * MD_WARPS;
    if (item < G * (DV / 64)) {
      const int g = item / (DV / 64), cb = item % (DV / 64);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int c = cb * 64 + 8 * j + 2 * qc;
        if (quad_row < per)
          *reinterpret_cast<float2*>(part_o + ((t * H + g * per + quad_row) * gridDim.x + blockIdx.x) * DV + c) = make_float2(o[i][j][0], o[i][j][1]);
        if (quad_row + 8 < per)
          *reinterpret_cast<float2*>(part_o + ((t * H + g * per + quad_row + 8) * gridDim.x + blockIdx.x) * DV + c) = make_float2(o[i][j][2], o[i][j][3]);
      }
    }
  }
}

// keys per chunk (32 or 16) of the decode kernel, 0 when it does not take these sizes
static int mix_attn_decode_plan(int H, int G, int dk, int dv, int dtype) {
  if ((dtype != B200P_F16 && dtype != B200P_BF16) || (dk != 64 && dk != 128) || (dv != 64 && dv != 128) || H > 32 || H / G > 16) return 0;
  if ((G * (dv / 64) + MD_WARPS - 1) / MD_WARPS > 4) return 0;
  for (int kt = 32; kt >= 16; kt /= 2)
    if (md_smem(H, G, dk, dv, kt) <= (size_t)MX_SMEM_MAX) return kt;
  return 0;
}

template <typename T, int DK, int DV, int MB, int KT, int ITEMS>
static int mix_attn_decode_launch(const float* q, const void* kc, const void* vc, int64_t Tcap, const int32_t* t_row, const int32_t* t_pos,
                                  const float* talk, const float* sink, int64_t window, void* out, int64_t ld_out, int64_t M, int H, int G,
                                  float* ws, size_t ws_bytes, cudaStream_t st) {
  auto kern = mix_attn_decode_kernel<T, DK, DV, MB, KT, ITEMS>;
  static bool attr = false;
  if (!attr) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, MX_SMEM_MAX);
    if (e != cudaSuccess) return cuda_fail(e, "cudaFuncSetAttribute(mix_attn_decode_kernel)");
    attr = true;
  }
  const size_t smem = md_smem(H, G, DK, DV, KT);
  // as many shares as fill the SMs once
  int per_sm = 1;
  if (cudaOccupancyMaxActiveBlocksPerMultiprocessor(&per_sm, kern, MD_THREADS, smem) != cudaSuccess || per_sm < 1) per_sm = 1;
  int splits = (int)(148 * (int64_t)per_sm / M);
  splits = splits < 1 ? 1 : splits > MX_MAX_SPLITS ? MX_MAX_SPLITS : splits;
  const size_t per_split = (size_t)M * H * (DV + 2) * sizeof(float);
  if ((size_t)splits * per_split > ws_bytes) splits = (int)(ws_bytes / per_split);
  if (splits < 1) return 1;                                          // no room for partial sums: the caller takes the per-token kernel
  float* part_o = ws;
  float* part_ms = ws + (size_t)M * H * splits * DV;
  kern<<<dim3((unsigned)splits, (unsigned)M), MD_THREADS, smem, st>>>(q, (const T*)kc, (const T*)vc, Tcap, t_row, t_pos, talk, window, H, G, part_o,
                                                                       part_ms);
  B200P_LAUNCH_CHECK("mix_attn_decode_kernel");
  attn_merge_kernel<T><<<dim3((unsigned)M, (unsigned)H), DV >= 128 ? 128 : 64, 0, st>>>(part_o, part_ms, nullptr, sink, (T*)out, ld_out, 1.f, H,
                                                                                         DV, splits, nullptr, 0);
  B200P_LAUNCH_CHECK("attn_merge_kernel");
  return B200P_OK;
}

template <typename T>
static int mix_attn_decode(const float* q, const void* kc, const void* vc, int64_t Tcap, const int32_t* t_row, const int32_t* t_pos,
                           const float* talk, const float* sink, int64_t window, void* out, int64_t ld_out, int64_t M, int H, int G, int dk,
                           int dv, int kt, float* ws, size_t ws_bytes, cudaStream_t st) {
  const int items = (G * (dv / 64) + MD_WARPS - 1) / MD_WARPS, mb = (H + 15) / 16;
#define MD_CASE(DK_, DV_, MB_, KT_, I_)                                                                                         \
  if (dk == DK_ && dv == DV_ && mb == MB_ && kt == KT_ && items <= I_)                                                          \
    return mix_attn_decode_launch<T, DK_, DV_, MB_, KT_, I_>(q, kc, vc, Tcap, t_row, t_pos, talk, sink, window, out, ld_out, M, H, G, ws, ws_bytes, st)
#define MD_ITEMS(DK_, DV_, MB_, KT_) MD_CASE(DK_, DV_, MB_, KT_, 1); MD_CASE(DK_, DV_, MB_, KT_, 2); MD_CASE(DK_, DV_, MB_, KT_, 4)
#define MD_SIZES(DK_, DV_) MD_ITEMS(DK_, DV_, 1, 32); MD_ITEMS(DK_, DV_, 1, 16); MD_ITEMS(DK_, DV_, 2, 32); MD_ITEMS(DK_, DV_, 2, 16)
  MD_SIZES(64, 64);
  MD_SIZES(64, 128);
  MD_SIZES(128, 64);
  MD_SIZES(128, 128);
#undef MD_SIZES
#undef MD_ITEMS
#undef MD_CASE
  set_error("mixed-score decode attention: unsupported sizes");
  return B200P_ERR_ARG;
}

template <typename T, int DK, int DV, int HB, int KT>
static int mix_attn_tile_launch(const float* q, const void* kc, const void* vc, int64_t Tcap, const int32_t* cu, const int32_t* rows,
                                const int32_t* t_pos, const float* talk, const float* sink, int window, void* out, int64_t ld_out, int nb,
                                int max_n, int H, int G, size_t smem, cudaStream_t st) {
  auto kern = mix_attn_tile_kernel<T, DK, DV, HB, KT>;
  static bool attr = false;
  if (!attr) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, MX_SMEM_MAX);
    if (e != cudaSuccess) return cuda_fail(e, "cudaFuncSetAttribute(mix_attn_tile_kernel)");
    attr = true;
  }
  constexpr int QB = 16 / HB;
  dim3 grid((unsigned)((max_n + QB - 1) / QB), (unsigned)nb);
  kern<<<grid, (unsigned)((H + HB - 1) / HB * 32), smem, st>>>(q, (const T*)kc, (const T*)vc, Tcap, cu, rows, t_pos, talk, sink, window,
                                                                (T*)out, ld_out, H, G);
  B200P_LAUNCH_CHECK("mix_attn_tile_kernel");
  return B200P_OK;
}

// heads per warp (1 or 2) and keys per chunk (32 or 16) of the tile kernel; false when it does not take these sizes
static bool mix_attn_tile_plan(int H, int G, int dk, int dv, int dtype, int* hb, int* kt) {
  if ((dtype != B200P_F16 && dtype != B200P_BF16) || (dk != 64 && dk != 128) || (dv != 64 && dv != 128)) return false;
  if (H <= MT_MAX_WARPS) *hb = 1;
  else if (H <= 2 * MT_MAX_WARPS && (H / G) % 2 == 0) *hb = 2;
  else return false;
  for (*kt = 32; *kt >= 16; *kt /= 2)
    if (mt_smem(H, G, dk, dv, *hb, *kt) <= (size_t)MX_SMEM_MAX) return true;
  return false;
}

template <typename T>
static int mix_attn_tiles(const float* q, const void* kc, const void* vc, int64_t Tcap, const int32_t* cu, const int32_t* rows,
                          const int32_t* t_pos, const float* talk, const float* sink, int window, void* out, int64_t ld_out, int nb,
                          int max_n, int H, int G, int dk, int dv, int hb, int kt, cudaStream_t st) {
  const size_t smem = mt_smem(H, G, dk, dv, hb, kt);
#define MT_CASE(DK_, DV_, HB_, KT_)                                                                                               \
  if (dk == DK_ && dv == DV_ && hb == HB_ && kt == KT_)                                                                           \
    return mix_attn_tile_launch<T, DK_, DV_, HB_, KT_>(q, kc, vc, Tcap, cu, rows, t_pos, talk, sink, window, out, ld_out, nb, max_n, H, G, smem, st)
#define MT_SIZES(DK_, DV_) MT_CASE(DK_, DV_, 1, 32); MT_CASE(DK_, DV_, 1, 16); MT_CASE(DK_, DV_, 2, 32); MT_CASE(DK_, DV_, 2, 16)
  MT_SIZES(64, 64);
  MT_SIZES(64, 128);
  MT_SIZES(128, 64);
  MT_SIZES(128, 128);
#undef MT_SIZES
#undef MT_CASE
  set_error("mixed-score tile attention: unsupported sizes");
  return B200P_ERR_ARG;
}

constexpr int MIX_ATTN_TILES_MIN_TOKENS = 4;   // shorter portions (and decode steps) take the per-token kernel

template <typename T, int VEC>
static int mix_attn_token(const float* q, const void* kc, const void* vc, int64_t Tcap, const int32_t* t_row, const int32_t* t_pos,
                          const float* talk, const float* sink, int64_t window, void* out, int64_t ld_out, int64_t M, int H, int G, int dk,
                          int dv, bool split, float* ws, size_t ws_bytes, cudaStream_t st) {
  const int KP = VEC > 1 ? dk + VEC : dk + 1;
  const size_t per_kv = (size_t)MX_KEYS * KP * sizeof(T), rest = ((size_t)H * (dk + dv + H + 2 * MX_KEYS + 3)) * sizeof(float) + 16;
  B200P_REQUIRE(rest + per_kv <= (size_t)MX_SMEM_MAX, B200P_ERR_ARG, "%d heads of %d / %d values do not fit the per-token kernel", H, dk, dv);
  size_t room = MX_SMEM_MAX - rest;
  if (room > 48 * 1024) room = per_kv > 48 * 1024 ? per_kv : 48 * 1024;          // leave room for several CTAs per SM
  int kv_block = (int)(room / per_kv);
  if (kv_block > G) kv_block = G;
  const size_t smem = rest + kv_block * per_kv;
  auto kern = mix_attn_kernel<T, VEC>;
  static size_t attr_smem = 48 * 1024;
  if (smem > attr_smem) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return cuda_fail(e, "cudaFuncSetAttribute(mix_attn_kernel)");
    attr_smem = smem;
  }
  int splits = 1;
  const size_t per_split = (size_t)M * H * (dv + 2) * sizeof(float);
  if (split) {
    splits = (int)((4 * 148 + M - 1) / M);
    splits = splits < 1 ? 1 : splits > MX_MAX_SPLITS ? MX_MAX_SPLITS : splits;
    if ((size_t)splits * per_split > ws_bytes) splits = (int)(ws_bytes / per_split);
  }
  B200P_REQUIRE(M < 65536, B200P_ERR_ARG, "at most 65535 tokens per call");
  if (splits <= 1) {
    kern<<<dim3(1, (unsigned)M), MX_THREADS, smem, st>>>(q, (const T*)kc, (const T*)vc, Tcap, t_row, t_pos, talk, sink, window, (T*)out, ld_out,
                                                          H, G, dk, dv, nullptr, nullptr, kv_block);
    B200P_LAUNCH_CHECK("mix_attn_kernel");
    return B200P_OK;
  }
  float* part_o = ws;
  float* part_ms = ws + (size_t)M * H * splits * dv;
  kern<<<dim3((unsigned)splits, (unsigned)M), MX_THREADS, smem, st>>>(q, (const T*)kc, (const T*)vc, Tcap, t_row, t_pos, talk, sink, window,
                                                                       (T*)out, ld_out, H, G, dk, dv, part_o, part_ms, kv_block);
  B200P_LAUNCH_CHECK("mix_attn_kernel");
  attn_merge_kernel<T><<<dim3((unsigned)M, (unsigned)H), dv >= 128 ? 128 : 64, 0, st>>>(part_o, part_ms, nullptr, sink, (T*)out, ld_out, 1.f, H,
                                                                                         dv, splits, nullptr, 0);
  B200P_LAUNCH_CHECK("attn_merge_kernel");
  return B200P_OK;
}

}  // namespace b200p

using namespace b200p;

extern "C" size_t b200p_mix_attn_workspace_bytes(int64_t nb, int H, int dv) {
  return (size_t)nb * H * MX_MAX_SPLITS * (dv + 2) * sizeof(float);
}

extern "C" int b200p_mix_attn_tiles_supported(int H, int G, int dk, int dv, int dtype) {
  int hb, kt;
  return H > 0 && G > 0 && H % G == 0 && mix_attn_tile_plan(H, G, dk, dv, dtype, &hb, &kt) ? hb * 100 + kt : 0;
}

extern "C" int b200p_mix_attn(const float* q, const void* kcache, const void* vcache, int64_t Tcap, const int32_t* t_row,
                              const int32_t* t_pos, const int32_t* cu, const int32_t* rows, int nb, int max_n, const float* talk,
                              const float* sink, int64_t window, void* out, int64_t ld_out, int64_t M, int H, int G, int dk, int dv,
                              int dtype, void* workspace, size_t workspace_bytes, void* stream) {
  B200P_REQUIRE(q && kcache && vcache && t_row && t_pos && talk && out, B200P_ERR_ARG, "null pointer");
  B200P_REQUIRE(H > 0 && G > 0 && H % G == 0 && dk > 0 && dv > 0, B200P_ERR_ARG, "bad head geometry");
  B200P_REQUIRE(window >= 0 && window < 0x7fffffff, B200P_ERR_ARG, "bad window");
  B200P_REQUIRE(ld_out >= (int64_t)H * dv, B200P_ERR_ARG, "output rows are shorter than the heads");
  if (M == 0) return B200P_OK;
  cudaStream_t st = (cudaStream_t)stream;
  int hb = 0, kt = 0;
  if (cu && rows && nb > 0 && nb < 65536 && max_n >= MIX_ATTN_TILES_MIN_TOKENS && ld_out % 2 == 0 &&
      (int64_t)G * Tcap * (dk > dv ? dk : dv) < 0xffffffffll && aligned(kcache, 16) &&
      aligned(vcache, 16) && aligned(out, 4) && aligned(q, 8) && mix_attn_tile_plan(H, G, dk, dv, dtype, &hb, &kt)) {
    return dtype == B200P_F16
        ? mix_attn_tiles<__half>(q, kcache, vcache, Tcap, cu, rows, t_pos, talk, sink, (int)window, out, ld_out, nb, max_n, H, G, dk, dv, hb, kt, st)
        : mix_attn_tiles<__nv_bfloat16>(q, kcache, vcache, Tcap, cu, rows, t_pos, talk, sink, (int)window, out, ld_out, nb, max_n, H, G, dk, dv, hb,
                                        kt, st);
  }
  // 16-bit decode steps (one token per entry) split their keys over CTAs, given room for the partial sums
  const bool split = max_n == 1 && dtype != B200P_F32 && workspace && aligned(workspace, 16);
  kt = split && M < 65536 && (int64_t)G * Tcap * (dk > dv ? dk : dv) < 0xffffffffll && aligned(kcache, 16) && aligned(vcache, 16) && aligned(q, 8)
           ? mix_attn_decode_plan(H, G, dk, dv, dtype) : 0;
  if (kt) {
    const int rc = dtype == B200P_F16
        ? mix_attn_decode<__half>(q, kcache, vcache, Tcap, t_row, t_pos, talk, sink, window, out, ld_out, M, H, G, dk, dv, kt, (float*)workspace,
                                  workspace_bytes, st)
        : mix_attn_decode<__nv_bfloat16>(q, kcache, vcache, Tcap, t_row, t_pos, talk, sink, window, out, ld_out, M, H, G, dk, dv, kt,
                                         (float*)workspace, workspace_bytes, st);
    if (rc != 1) return rc;
  }
  const int vec = dtype == B200P_F32 ? 4 : 8;
  const bool whole = dk % vec == 0 && dv % vec == 0 && aligned(kcache, 16) && aligned(vcache, 16);
#define MX_CASE(T, V_) \
  mix_attn_token<T, V_>(q, kcache, vcache, Tcap, t_row, t_pos, talk, sink, window, out, ld_out, M, H, G, dk, dv, split, (float*)workspace, workspace_bytes, st)
  switch (dtype) {
    case B200P_F32: return whole ? MX_CASE(float, 4) : MX_CASE(float, 1);
    case B200P_F16: return whole ? MX_CASE(__half, 8) : MX_CASE(__half, 1);
    case B200P_BF16: return whole ? MX_CASE(__nv_bfloat16, 8) : MX_CASE(__nv_bfloat16, 1);
    default: set_error("bad dtype %d", dtype); return B200P_ERR_ARG;
  }
#undef MX_CASE
}
