// Hyper-connections: the residual stream of a token is S copies x_1 .. x_S (fp32 rows [T][S][W]) that are mixed around every
// sublayer.  A sublayer reads u = sum_s r_s x_s through an RMS norm, and its output y goes back as
//     x_t <- sum_s M[s][t] x_s + o_t y          (M[s][t]: how much of the previous copy s goes into the next copy t).
//   * hyper_embed: every copy = the token's embedding row, and the first sublayer's normed input;
//   * hyper_residual: one pass over the copies per sublayer: gathers y (a branch row plus the weighted sum of expert rows), mixes,
//     stores, reads the next sublayer's u from the new copies and norms it into the next GEMM's operand.
// One CTA per token; u stays in shared memory between the two passes over the row.  All sums are fp32 in a fixed order, so a row
// does not depend on what else is in the batch.
#include "hybrid_common.cuh"

namespace b200 {

constexpr int HC_MAX = 32;  // most copies

template <int V>
struct HcVec {
  float v[V];
};
template <int V>
__device__ __forceinline__ HcVec<V> hc_ld(const float* p) {
  HcVec<V> a;
  if constexpr (V == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    a.v[0] = f.x, a.v[1] = f.y, a.v[2] = f.z, a.v[3] = f.w;
  } else {
    a.v[0] = *p;
  }
  return a;
}
template <int V>
__device__ __forceinline__ void hc_st(float* p, const HcVec<V>& a) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(a.v[0], a.v[1], a.v[2], a.v[3]);
  else *p = a.v[0];
}
template <typename OT, int V>
__device__ __forceinline__ void hc_out(OT* p, const HcVec<V>& a) {
  if constexpr (V == 4 && sizeof(OT) == 2) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(a.v[0], a.v[1]), pack_bf16(a.v[2], a.v[3]));
  } else {
#pragma unroll
    for (int k = 0; k < V; ++k) stf(p, k, a.v[k]);
  }
}

// out[t] = row / sqrt(mean(row^2) + eps) * w, the row in shared memory, ss = this thread's share of the sum of squares
template <typename OT, int V>
__device__ __forceinline__ void hc_norm_row(const float* row, float ss, const float* __restrict__ w, float eps, OT* __restrict__ out, int W) {
  __shared__ float red[33];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  if (warp == 0) {
    const float s = warp_sum(lane < (int)((blockDim.x + 31) >> 5) ? red[lane] : 0.f);
    if (lane == 0) red[32] = s;
  }
  __syncthreads();
  const float inv = 1.0f / sqrtf(red[32] / (float)W + eps);
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
    HcVec<V> u = hc_ld<V>(row + i);
    const HcVec<V> g = hc_ld<V>(w + i);
#pragma unroll
    for (int k = 0; k < V; ++k) u.v[k] = u.v[k] * inv * g.v[k];
    hc_out<OT, V>(out + i, u);
  }
}

template <typename ET, int V>
__global__ void hyper_embed_kernel(const int32_t* __restrict__ tokens, const ET* __restrict__ table, float* __restrict__ x, int S,
                                   const float* __restrict__ read, const float* __restrict__ w, float eps, ET* __restrict__ out,
                                   int W, int vocab) {
  griddep_launch();
  griddep_wait();
  extern __shared__ __align__(16) float row[];
  const int64_t t = blockIdx.x;
  int tok = tokens[t];
  tok = tok < 0 ? 0 : (tok >= vocab ? vocab - 1 : tok);
  float r = 0.f, ss = 0.f;
  for (int s = 0; s < S; ++s) r += read[s];
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
    HcVec<V> e;
#pragma unroll
    for (int k = 0; k < V; ++k) e.v[k] = ldf(table, (int64_t)tok * W + i + k);
    for (int s = 0; s < S; ++s) hc_st<V>(x + (t * S + s) * W + i, e);
#pragma unroll
    for (int k = 0; k < V; ++k) {
      e.v[k] *= r;
      ss += e.v[k] * e.v[k];
    }
    hc_st<V>(row + i, e);
  }
  hc_norm_row<ET, V>(row, ss, w, eps, out + t * W, W);
}

// NS: the number of copies when it is known at compile time (coefficients and copies in registers), 0: S copies, S <= HC_MAX
template <typename OT, int NS, int V>
__global__ void hyper_residual_kernel(float* __restrict__ x, int S, const float* __restrict__ y1, int ld1, const float* __restrict__ y2,
                                      int nsum, const float* __restrict__ y2_weight, const float* __restrict__ mix,
                                      const float* __restrict__ write, const float* __restrict__ read, const float* __restrict__ w,
                                      float eps, int store, OT* __restrict__ out, int W) {
  griddep_launch();
  griddep_wait();
  extern __shared__ __align__(16) float row[];
  constexpr int N = NS > 0 ? NS : HC_MAX, UN = NS > 0 ? NS : 1;
  const int n = NS > 0 ? NS : S;
  const int64_t t = blockIdx.x;
  float* xr = x + t * n * W;
  float M[NS > 0 ? NS * NS : 1], O[NS > 0 ? NS : 1], R[NS > 0 ? NS : 1];
  if constexpr (NS > 0) {
#pragma unroll
    for (int i = 0; i < NS * NS; ++i) M[i] = __ldg(mix + i);
#pragma unroll
    for (int i = 0; i < NS; ++i) O[i] = __ldg(write + i), R[i] = __ldg(read + i);
  }
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
    HcVec<V> xs[N], y, u;
#pragma unroll UN
    for (int s = 0; s < N; ++s)
      if (NS > 0 || s < n) xs[s] = hc_ld<V>(xr + (int64_t)s * W + i);
#pragma unroll
    for (int k = 0; k < V; ++k) y.v[k] = u.v[k] = 0.f;
    if (y1) y = hc_ld<V>(y1 + t * ld1 + i);
    if (y2) {
#pragma unroll 4
      for (int c = 0; c < nsum; ++c) {
        const HcVec<V> b = hc_ld<V>(y2 + (t * nsum + c) * W + i);
        const float f = y2_weight ? y2_weight[t * nsum + c] : 1.0f;
#pragma unroll
        for (int k = 0; k < V; ++k) y.v[k] += f * b.v[k];
      }
    }
#pragma unroll UN
    for (int d = 0; d < N; ++d) {
      if (NS == 0 && d >= n) continue;
      const float o = NS > 0 ? O[NS > 0 ? d : 0] : write[d], r = NS > 0 ? R[NS > 0 ? d : 0] : read[d];
      HcVec<V> a;
#pragma unroll
      for (int k = 0; k < V; ++k) a.v[k] = o * y.v[k];
#pragma unroll UN
      for (int s = 0; s < N; ++s) {
        if (NS == 0 && s >= n) continue;
        const float m = NS > 0 ? M[NS > 0 ? s * NS + d : 0] : mix[s * n + d];
#pragma unroll
        for (int k = 0; k < V; ++k) a.v[k] += m * xs[s].v[k];
      }
      if (store) hc_st<V>(xr + (int64_t)d * W + i, a);
#pragma unroll
      for (int k = 0; k < V; ++k) u.v[k] += r * a.v[k];
    }
#pragma unroll
    for (int k = 0; k < V; ++k) ss += u.v[k] * u.v[k];
    hc_st<V>(row + i, u);
  }
  hc_norm_row<OT, V>(row, ss, w, eps, out + t * W, W);
}

// many tokens: small CTAs, so that several rows per SM are in different phases; few tokens: more threads on each row
static int hc_threads(int T, int W, bool v4) {
  const int per = v4 ? W / 4 : W;
  return T >= 512 || per <= 128 ? 128 : 256;
}

}  // namespace b200

using namespace b200;

extern "C" {

int b200_hyper_embed(const int32_t* tokens, const void* table, int dtype, float* x, int S, const float* read, const float* w, float eps,
                     void* out, int T, int W, int vocab, void* stream) {
  B200_REQUIRE(tokens && table && x && read && w && out, "hyper_embed: null pointer");
  B200_REQUIRE(S >= 1 && S <= HC_MAX && W >= 1 && vocab >= 1, "hyper_embed: %d copies of rows of %d", S, W);
  B200_REQUIRE((size_t)W * 4 <= 200 * 1024, "hyper_embed: rows of %d do not fit shared memory", W);
  if (T <= 0) return B200_OK;
  const size_t smem = (size_t)W * 4;
  auto a16 = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  const bool v4 = W % 4 == 0 && a16(x) && a16(w) && a16(out);
#define HC_EMBED(V)                                                                                                              \
  B200_DISPATCH_ELEM(dtype, ET, {                                                                                                \
    if (smem > 48 * 1024)                                                                                                        \
      B200_CUDA_OK(cudaFuncSetAttribute(hyper_embed_kernel<ET, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));     \
    B200_CUDA_OK(launch_kernel(hyper_embed_kernel<ET, V>, dim3(T), dim3(hc_threads(T, W, V == 4)), smem, (cudaStream_t)stream, tokens, \
                               (const ET*)table, x, S, read, w, eps, (ET*)out, W, vocab));                                       \
  })
  if (v4) HC_EMBED(4);
  else HC_EMBED(1);
#undef HC_EMBED
  return B200_OK;
}

int b200_hyper_residual(float* x, int S, const float* y1, int ld1, const float* y2, int nsum, const float* y2_weight, const float* mix,
                        const float* write, const float* read, const float* w, float eps, int store, void* out, int out_dtype, int T,
                        int W, void* stream) {
  B200_REQUIRE(x && mix && write && read && w && out && (!y2 || nsum >= 1), "hyper_residual: null pointer");
  B200_REQUIRE(S >= 1 && S <= HC_MAX && W >= 1, "hyper_residual: %d copies of rows of %d", S, W);
  B200_REQUIRE((size_t)W * 4 <= 200 * 1024, "hyper_residual: rows of %d do not fit shared memory", W);
  if (T <= 0) return B200_OK;
  const size_t smem = (size_t)W * 4;
  auto a16 = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  const bool v4 = W % 4 == 0 && ld1 % 4 == 0 && a16(x) && a16(y1) && a16(y2) && a16(w) && a16(out);
#define HC_LAUNCH(NS, V)                                                                                                            \
  B200_DISPATCH_ELEM(out_dtype, OT, {                                                                                               \
    if (smem > 48 * 1024)                                                                                                           \
      B200_CUDA_OK(cudaFuncSetAttribute(hyper_residual_kernel<OT, NS, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
    B200_CUDA_OK(launch_kernel(hyper_residual_kernel<OT, NS, V>, dim3(T), dim3(hc_threads(T, W, V == 4)), smem, (cudaStream_t)stream, x, \
                               S, y1, ld1, y2, nsum, y2_weight, mix, write, read, w, eps, store, (OT*)out, W));                     \
  })
#define HC_PICK(NS)                \
  do {                             \
    if (v4) HC_LAUNCH(NS, 4);      \
    else HC_LAUNCH(NS, 1);         \
  } while (0)
  if (S == 1) HC_PICK(1);
  else if (S == 2) HC_PICK(2);
  else if (S == 3) HC_PICK(3);
  else if (S == 4) HC_PICK(4);
  else HC_LAUNCH(0, 1);
#undef HC_PICK
#undef HC_LAUNCH
  return B200_OK;
}

}  // extern "C"
