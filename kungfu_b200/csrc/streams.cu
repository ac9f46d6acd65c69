// A residual of several streams ("hyper-connections"): n copies x_1 .. x_n of the row instead of one, [rows, n, W] in 32-bit.
//   what a sublayer reads    u = sum_s in[s] x_s, then an RMS norm of u
//   what becomes of it       x_t <- sum_s mix[s, t] x_s + out[t] y     (all streams at once from the old ones)
// kf_streams_step does the second and, in the same pass over the streams, the first of the sublayer that comes next; without
// a result y it only reads (the first sublayer of a model, the output head on some rows).  The learned numbers are 32-bit.
// One block per row; the combination u stays in shared memory between the sum of squares and the scaling, and a thread reads
// back only elements it wrote itself.
#include "common.cuh"

namespace {

constexpr int ST_MAX = 16;

template <int V> __device__ __forceinline__ void st_load(const float* p, float* v) {
  if constexpr (V == 4) { const float4 a = *reinterpret_cast<const float4*>(p); v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w; }
  else v[0] = *p;
}
template <int V> __device__ __forceinline__ void st_store(float* p, const float* v) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}
template <int V> __device__ __forceinline__ void st_store(__nv_bfloat16* p, const float* v) {
  if constexpr (V == 4) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  } else {
    *p = __float2bfloat16_rn(v[0]);
  }
}

// S: the number of streams, or (16) its bound; n: the number itself.
template <typename TW, typename TO, int S, int V>
__global__ void __launch_bounds__(512)
streams_step_kernel(float* x, const float* y, const float* __restrict__ mix, const float* __restrict__ outw, const int* rows,
                    const float* __restrict__ in, const TW* __restrict__ w, float eps, TO* __restrict__ next, int n, int W) {
  kf_pdl_trigger();
  const int N = S == ST_MAX ? n : S;
  extern __shared__ __align__(16) float st_u[];
  __shared__ float m[S * S], ow[S], iw[S], red[33];
  const bool update = y != nullptr;
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) {
    const int s = i / S, t = i - s * S;
    m[i] = (update && s < N && t < N) ? mix[s * N + t] : 0.f;
    if (s == 0) {
      ow[t] = (update && t < N) ? outw[t] : 0.f;
      iw[t] = (next && t < N) ? in[t] : 0.f;
    }
  }
  kf_pdl_wait();
  x = kf_produced(x), y = kf_produced(y), rows = kf_produced(rows);
  __syncthreads();
  const int r = blockIdx.x;
  float* xr = x + (size_t)(rows ? rows[r] : r) * N * W;
  float ss = 0.f;
#pragma unroll 2
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
    float v[S][V], u[V];
#pragma unroll
    for (int s = 0; s < S; ++s)
      if (s < N) st_load<V>(xr + (size_t)s * W + i, v[s]);
#pragma unroll
    for (int e = 0; e < V; ++e) u[e] = 0.f;
    if (update) {
      float b[V];
      st_load<V>(y + (size_t)r * W + i, b);
#pragma unroll
      for (int t = 0; t < S; ++t) {
        if (t >= N) continue;
        float a[V];
#pragma unroll
        for (int e = 0; e < V; ++e) a[e] = ow[t] * b[e];
#pragma unroll
        for (int s = 0; s < S; ++s)
          if (s < N) {
#pragma unroll
            for (int e = 0; e < V; ++e) a[e] = fmaf(m[s * S + t], v[s][e], a[e]);
          }
        st_store<V>(xr + (size_t)t * W + i, a);
#pragma unroll
        for (int e = 0; e < V; ++e) u[e] = fmaf(iw[t], a[e], u[e]);
      }
    } else {
#pragma unroll
      for (int s = 0; s < S; ++s)
        if (s < N) {
#pragma unroll
          for (int e = 0; e < V; ++e) u[e] = fmaf(iw[s], v[s][e], u[e]);
        }
    }
    if (next) {
      st_store<V>(st_u + i, u);
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(u[e], u[e], ss);
    }
  }
  if (!next) return;
  ss = kf_block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / (float)W + eps);
  TO* o = next + (size_t)r * W;
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
    float u[V];
    st_load<V>(st_u + i, u);
#pragma unroll
    for (int e = 0; e < V; ++e) u[e] = u[e] * inv * kf_load(w, i + e);
    st_store<V>(o + i, u);
  }
}

template <typename TW, typename TO, int V>
int streams_go(float* x, const float* y, const float* mix, const float* outw, const int* rows, const float* in, const void* w,
               float eps, void* next, int T, int n, int W, cudaStream_t stream) {
  const int groups = kf_ceil_div(W, V), most = T >= 148 ? 256 : 512;
  const int threads = groups >= most ? most : kf_ceil_div(groups, 32) * 32;
  const size_t smem = next ? (size_t)W * sizeof(float) : 0;
#define KF_GO(S)                                                                                                         \
  case S:                                                                                                                \
    kf_launch(streams_step_kernel<TW, TO, S, V>, dim3(T), dim3(threads), smem, stream, x, y, mix, outw, rows, in, (const TW*)w, \
              eps, (TO*)next, n, W);                                                                                     \
    break
  switch (n <= 8 ? n : ST_MAX) {
    KF_GO(1); KF_GO(2); KF_GO(3); KF_GO(4); KF_GO(5); KF_GO(6); KF_GO(7); KF_GO(8); KF_GO(16);
  }
#undef KF_GO
  KF_CHECK_LAUNCH();
  return KF_OK;
}

}  // namespace

// x [rows, n, W]; y [T, W], mix [n, n] (from, to) and outw [n], or all null; next [T, W] with in [n] and w [W], or all null.
// rows (only without y): row r of `next` comes from row rows[r] of x.
KF_API int kf_streams_step(float* x, const float* y, const float* mix, const float* outw, const int* rows, const float* in,
                           const void* w, int w_dtype, float eps, void* next, int next_dtype, int T, int n, int W,
                           cudaStream_t stream) {
  if (T <= 0) return KF_OK;
  if (n < 1 || n > ST_MAX || W < 1 || W > 10240 || (y && (rows || !mix || !outw)) || (next && (!in || !w)) || (!y && !next))
    return KF_ERR_SIZE;                                    // W: the combination stands in 40 KB of shared memory
  const bool by4 = W % 4 == 0 && (((uintptr_t)x | (uintptr_t)y | (uintptr_t)next) & 15) == 0;
#define KF_DT(TW, TO)                                                                                                   \
  return by4 ? streams_go<TW, TO, 4>(x, y, mix, outw, rows, in, w, eps, next, T, n, W, stream)                           \
             : streams_go<TW, TO, 1>(x, y, mix, outw, rows, in, w, eps, next, T, n, W, stream)
  if (!next || (w_dtype == KF_F32 && next_dtype == KF_F32)) KF_DT(float, float);
  if (w_dtype == KF_BF16 && next_dtype == KF_BF16) KF_DT(__nv_bfloat16, __nv_bfloat16);
#undef KF_DT
  return KF_ERR_DTYPE;
}
