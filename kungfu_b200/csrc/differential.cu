// Differential attention's last step: every head has two attention results a_1, a_2 over the same values (two maps with
// queries and keys of their own), of which the second is taken from the first:
//   d = a_1 - lambda a_2;   out_h = d / sqrt(mean(d^2) + eps) * factor * sigmoid(g_h)
// The attention kernels leave the maps as neighbouring result heads 2h and 2h + 1 of D elements, of which the first dv
// count; `out` is packed, dv per head.  Sums and factors are 32-bit.
#include "common.cuh"

namespace {

constexpr int DF_THREADS = 128;

template <int V> __device__ __forceinline__ void df_load(const float* p, float* v) {
  if constexpr (V == 4) { const float4 a = *reinterpret_cast<const float4*>(p); v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w; }
  else v[0] = *p;
}
template <int V> __device__ __forceinline__ void df_load(const __nv_bfloat16* p, float* v) {
  if constexpr (V == 8) {
    const uint4 r = *reinterpret_cast<const uint4*>(p);
    const uint32_t u[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u[k]));
      v[2 * k] = f.x, v[2 * k + 1] = f.y;
    }
  } else if constexpr (V == 4) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
    v[0] = a.x, v[1] = a.y, v[2] = b.x, v[3] = b.y;
  } else {
    v[0] = __bfloat162float(*p);
  }
}
template <int V> __device__ __forceinline__ void df_store(float* p, const float* v) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}
template <int V> __device__ __forceinline__ void df_store(__nv_bfloat16* p, const float* v) {
  if constexpr (V == 8) {
    uint32_t u[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const __nv_bfloat162 h = __floats2bfloat162_rn(v[2 * k], v[2 * k + 1]);
      u[k] = *reinterpret_cast<const uint32_t*>(&h);
    }
    *reinterpret_cast<uint4*>(p) = make_uint4(u[0], u[1], u[2], u[3]);
  } else if constexpr (V == 4) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  } else {
    *p = __float2bfloat16_rn(v[0]);
  }
}

// L lanes per (row, head), V neighbouring elements per lane and round.  A head above L * V elements is read twice (its second
// reading comes from the first-level cache).
template <typename T, int V, int L>
__global__ void __launch_bounds__(DF_THREADS)
diff_combine_kernel(const T* __restrict__ o, float lambda, float factor, float eps, const float* __restrict__ g, int ld, int gcol0,
                    int nh, int dv, int D, T* __restrict__ out, const int* __restrict__ row_req, int rows) {
  kf_pdl_trigger();
  kf_pdl_wait();
  const int lane = threadIdx.x % L;
  const long item = (long)blockIdx.x * (DF_THREADS / L) + threadIdx.x / L;
  const bool live = item < (long)rows * nh;             // every lane of a warp reaches the shuffles
  const int t = live ? (int)(item / nh) : 0, h = live ? (int)(item - (long)t * nh) : 0;
  const bool pad = !live || row_req[t] < 0;
  const T* a1 = o + ((size_t)t * nh + h) * 2 * D;
  const T* a2 = a1 + D;
  float first[V], ss = 0.f;
#pragma unroll
  for (int e = 0; e < V; ++e) first[e] = 0.f;
  auto diff = [&](int i, float* d) {
    float b[V];
    df_load<V>(a1 + i, d);
    df_load<V>(a2 + i, b);
#pragma unroll
    for (int e = 0; e < V; ++e) d[e] = fmaf(-lambda, b[e], d[e]);
  };
  if (!pad)
    for (int i = lane * V; i < dv; i += L * V) {
      float d[V];
      diff(i, d);
#pragma unroll
      for (int e = 0; e < V; ++e) {
        ss = fmaf(d[e], d[e], ss);
        if (i < L * V) first[e] = d[e];
      }
    }
#pragma unroll
  for (int k = L / 2; k > 0; k >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, k);
  if (!live) return;
  float s = 0.f;
  if (!pad) {
    s = factor / sqrtf(ss / (float)dv + eps);
    if (g) s *= 1.f / (1.f + expf(-g[(size_t)t * ld + gcol0 + h]));
  }
  for (int i = lane * V; i < dv; i += L * V) {
    float d[V];
    if (i < L * V || pad) {
#pragma unroll
      for (int e = 0; e < V; ++e) d[e] = first[e];      // zeros in a row of padding
    } else {
      diff(i, d);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) d[e] *= s;
    df_store<V>(out + ((size_t)t * nh + h) * dv + i, d);
  }
}

template <typename T>
int diff_go(const void* o, float lambda, float factor, float eps, const float* g, int ld, int gcol0, int nh, int dv, int D, void* out,
            const int* row_req, int rows, cudaStream_t stream) {
  const bool by4 = dv % 4 == 0 && D % 4 == 0 && (((uintptr_t)o | (uintptr_t)out) & 15) == 0;
#define KF_GO(V, L)                                                                                                        \
  kf_launch(diff_combine_kernel<T, V, L>, dim3((unsigned)kf_ceil_div((long)rows * nh, DF_THREADS / L)), dim3(DF_THREADS), 0, stream, \
            (const T*)o, lambda, factor, eps, g, ld, gcol0, nh, dv, D, (T*)out, row_req, rows)
  if constexpr (sizeof(T) == 2) {
    if (by4 && dv % 8 == 0 && D % 8 == 0) {                // 16 bytes per lane and load
      if (dv <= 64) KF_GO(8, 8); else if (dv <= 128) KF_GO(8, 16); else KF_GO(8, 32);
      KF_CHECK_LAUNCH();
      return KF_OK;
    }
  }
  if (!by4) KF_GO(1, 32);
  else if (dv <= 32) KF_GO(4, 8);
  else if (dv <= 64) KF_GO(4, 16);
  else KF_GO(4, 32);
#undef KF_GO
  KF_CHECK_LAUNCH();
  return KF_OK;
}

}  // namespace

// o [rows, 2 nh, D]; out [rows, nh dv]; g: a 32-bit matrix with ld columns, head h's gate in column gcol0 + h (null: no gate).
KF_API int kf_diff_combine(const void* o, float lambda, float factor, float eps, const float* g, int ld, int gcol0, int nh, int dv,
                           int D, void* out, int dtype, const int* row_req, int rows, cudaStream_t stream) {
  if (rows <= 0) return KF_OK;
  if (nh < 1 || dv < 1 || dv > D) return KF_ERR_SIZE;
  if (dtype == KF_F32) return diff_go<float>(o, lambda, factor, eps, g, ld, gcol0, nh, dv, D, out, row_req, rows, stream);
  if (dtype == KF_BF16) return diff_go<__nv_bfloat16>(o, lambda, factor, eps, g, ld, gcol0, nh, dv, D, out, row_req, rows, stream);
  return KF_ERR_DTYPE;
}
