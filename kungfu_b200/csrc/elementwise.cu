// Embedding gather, rotary tables, gated activation, residual add.
#include "common.cuh"

// x[t, :] = table[token[t], :] * scale, `copies` times over (x [rows, copies, H]).  A token id outside [0, V) writes zeros and sets *bad.
// Reference: gather then scale, crates/kf-layers/src/basic.rs:35-36.
template <typename TW>
__global__ void embed_kernel(const int* __restrict__ tokens, const TW* __restrict__ table, float scale,
                             float* __restrict__ out, int H, int V, int copies, int* __restrict__ bad) {
  kf_pdl_trigger();
  kf_pdl_wait();
  const int t = blockIdx.x;
  const int tok = tokens[t];
  const bool ok = tok >= 0 && tok < V;
  if (!ok && threadIdx.x == 0 && bad) atomicExch(bad, 1);
  const TW* row = table + (size_t)(ok ? tok : 0) * H;
  float* o = out + (size_t)t * copies * H;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    const float v = ok ? kf_load(row, i) * scale : 0.f;
    for (int c = 0; c < copies; ++c) o[(size_t)c * H + i] = v;
  }
}

KF_API int kf_embed(const int* tokens, const void* table, int table_dtype, float scale, float* out,
                    int T, int H, int V, int copies, int* bad_flag, cudaStream_t stream) {
  if (T <= 0) return KF_OK;
  if (copies < 1) return KF_ERR_SIZE;
  const int threads = H >= 1024 ? 256 : 128;
  if (table_dtype == KF_F32)
    kf_launch(embed_kernel<float>, dim3(T), dim3(threads), 0, stream, tokens, (const float*)table, scale, out, H, V, copies, bad_flag);
  else if (table_dtype == KF_BF16)
    kf_launch(embed_kernel<__nv_bfloat16>, dim3(T), dim3(threads), 0, stream, tokens, (const __nv_bfloat16*)table, scale, out, H, V, copies, bad_flag);
  else
    return KF_ERR_DTYPE;
  KF_CHECK_LAUNCH();
  return KF_OK;
}

__device__ __forceinline__ float4 kf_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 kf_load4(const __nv_bfloat16* p) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
  return make_float4(a.x, a.y, b.x, b.y);
}

// x[t, :] = table[token[t], :] * scale + pair[row(t), :], a second table read by the token and the one before it:
// row(t) = (previous * mul_prev + token * mul_cur) mod buckets in 64-bit integers, the table's last row (number `buckets`)
// for a request's first token.  The previous token of a step's first row of a request is its state, prev[slot] (written
// here too: the block of that row is the only one that reads or writes it).  Padding rows (request -1) give zeros.
template <typename TW>
__global__ void embed_pair_kernel(const int* __restrict__ tokens, const TW* __restrict__ table, const TW* __restrict__ pair,
                                  float scale, long long mul_prev, long long mul_cur, long long buckets, int* prev,
                                  float* __restrict__ out, int H, int V, const int* __restrict__ positions,
                                  const int* __restrict__ row_req, const int* __restrict__ req_row_start,
                                  const int* __restrict__ req_n_rows, const int* __restrict__ req_state_slot, int writes) {
  kf_pdl_trigger();
  kf_pdl_wait();
  __shared__ long long s_row;
  const int t = blockIdx.x, req = row_req[t];
  float* o = out + (size_t)t * H;
  if (req < 0) {
    for (int i = threadIdx.x; i < H; i += blockDim.x) o[i] = 0.f;
    return;
  }
  const int tok = tokens[t];
  if (threadIdx.x == 0) {
    const int row0 = req_row_start[req], slot = req_state_slot[req];
    long long r = buckets;
    if (positions[t] > 0) {
      const long long before = t > row0 ? tokens[t - 1] : prev[slot];
      r = (before * mul_prev + (long long)tok * mul_cur) % buckets;
      if (r < 0) r += buckets;
    }
    s_row = r;
    if (t == row0 && writes) prev[slot] = tokens[row0 + req_n_rows[req] - 1];
  }
  __syncthreads();
  const bool ok = tok >= 0 && tok < V;
  const TW* a = table + (size_t)(ok ? tok : 0) * H;
  const TW* b = pair + (size_t)s_row * H;
  if ((H & 3) == 0) {                                   // rows start on four elements
    for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (ok) {
        const float4 x = kf_load4(a + i), y = kf_load4(b + i);
        v = make_float4(x.x * scale + y.x, x.y * scale + y.y, x.z * scale + y.z, x.w * scale + y.w);
      }
      *reinterpret_cast<float4*>(o + i) = v;
    }
    return;
  }
  for (int i = threadIdx.x; i < H; i += blockDim.x) o[i] = ok ? kf_load(a, i) * scale + kf_load(b, i) : 0.f;
}

KF_API int kf_embed_pair(const int* tokens, const void* table, const void* pair, int dtype, float scale, long long mul_prev,
                         long long mul_cur, long long buckets, int* prev, float* out, int T, int H, int V, const int* positions,
                         const int* row_req, const int* req_row_start, const int* req_n_rows, const int* req_state_slot,
                         int writes, cudaStream_t stream) {
  if (T <= 0) return KF_OK;
  if (buckets < 1 || !prev) return KF_ERR_SIZE;
  if (H % 4 == 0 && (((uintptr_t)table | (uintptr_t)pair | (uintptr_t)out) & 15)) return KF_ERR_ALIGN;
  const int threads = H >= 1024 ? 256 : 128;
#define KF_GO(TW)                                                                                                          \
  kf_launch(embed_pair_kernel<TW>, dim3(T), dim3(threads), 0, stream, tokens, (const TW*)table, (const TW*)pair, scale, mul_prev, \
            mul_cur, buckets, prev, out, H, V, positions, row_req, req_row_start, req_n_rows, req_state_slot, writes)
  if (dtype == KF_F32) KF_GO(float);
  else if (dtype == KF_BF16) KF_GO(__nv_bfloat16);
  else return KF_ERR_DTYPE;
#undef KF_GO
  KF_CHECK_LAUNCH();
  return KF_OK;
}

// out[t, i] = x[t, i] * sigmoid(gate[t, col0 + i]), gate a wider 32-bit matrix: one gate per element.  VEC = 4 where rows and
// columns start on four elements.
template <typename T, int VEC>
__global__ void element_gate_kernel(const T* __restrict__ x, const float* __restrict__ gate, int ld, int col0, T* __restrict__ out,
                                    int n_rows, int n) {
  kf_pdl_trigger();
  kf_pdl_wait();
  const long i = ((long)blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (i >= (long)n_rows * n) return;
  const int t = (int)(i / n), c = (int)(i - (long)t * n);
  const float* g = gate + (size_t)t * ld + col0 + c;
  float z[VEC], v[VEC];
  if constexpr (VEC == 4) {
    const float4 q = *reinterpret_cast<const float4*>(g);
    z[0] = q.x, z[1] = q.y, z[2] = q.z, z[3] = q.w;
  } else z[0] = g[0];
#pragma unroll
  for (int k = 0; k < VEC; ++k) v[k] = kf_load(x, (size_t)i + k) / (1.f + expf(-z[k]));
#pragma unroll
  for (int k = 0; k < VEC; ++k) kf_store(out, (size_t)i + k, v[k]);
}

KF_API int kf_element_gate(const void* x, const float* gate, int ld, int col0, void* out, int dtype, int n_rows, int n,
                           cudaStream_t stream) {
  if (n_rows <= 0 || n <= 0) return KF_OK;
  if (col0 < 0 || col0 + n > ld) return KF_ERR_SIZE;
  const bool vec = n % 4 == 0 && ld % 4 == 0 && col0 % 4 == 0 && (((uintptr_t)x | (uintptr_t)gate | (uintptr_t)out) & 15) == 0;
  const int grid = kf_ceil_div((long)n_rows * n, 256 * (vec ? 4 : 1));
#define KF_GO(T, VEC) kf_launch(element_gate_kernel<T, VEC>, dim3(grid), dim3(256), 0, stream, (const T*)x, gate, ld, col0, (T*)out, n_rows, n)
  if (dtype == KF_F32) { if (vec) KF_GO(float, 4); else KF_GO(float, 1); }
  else if (dtype == KF_BF16) { if (vec) KF_GO(__nv_bfloat16, 4); else KF_GO(__nv_bfloat16, 1); }
  else return KF_ERR_DTYPE;
#undef KF_GO
  KF_CHECK_LAUNCH();
  return KF_OK;
}

// cos/sin of position * inv_freq[i], all in 32-bit (accurate sincosf: no fast-math in this library).
// The product of a position and a 32-bit frequency has up to 48 significant bits; rounded to 32-bit it is off by up to
// 2.4e-4 rad at position 4,000, which a 32-bit engine with scores of 40 shows in its logits.  So the product is kept as
// an unevaluated sum hi + lo (lo = fma(p, f, -hi) is its exact rounding error) and the tables are
// cos(hi) (1 - lo^2/2) - lo sin(hi) and sin(hi) (1 - lo^2/2) + lo cos(hi): exact to second order in lo, which is below
// 2^-11 up to position 8,192 and below 2^-8 up to 131,072 (error below 1e-7 there).
// Reference: crates/kf-backend-cuda/src/kernels/rope.cu:4-14 (angle as one 32-bit product).
__global__ void rope_table_kernel(const int* __restrict__ positions, const float* __restrict__ inv_freq,
                                  float* __restrict__ cos_out, float* __restrict__ sin_out, int T, int half) {
  kf_pdl_trigger();
  kf_pdl_wait();
  const int idx = blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= T * half) return;
  const int t = idx / half, i = idx - t * half;
  const float p = (float)positions[t], f = inv_freq[i];
  const float hi = __fmul_rn(p, f);
  const float lo = __fmaf_rn(p, f, -hi);
  float s, c;
  sincosf(hi, &s, &c);
  const float h = 1.f - 0.5f * lo * lo;
  cos_out[idx] = __fmaf_rn(-lo, s, c * h);
  sin_out[idx] = __fmaf_rn(lo, c, s * h);
}

KF_API int kf_rope_table(const int* positions, const float* inv_freq, float* cos_out, float* sin_out,
                         int T, int half, cudaStream_t stream) {
  if (T <= 0 || half <= 0) return KF_OK;
  const int n = T * half;
  kf_launch(rope_table_kernel, dim3(kf_ceil_div(n, 256)), dim3(256), 0, stream, positions, inv_freq, cos_out, sin_out, T, half);
  KF_CHECK_LAUNCH();
  return KF_OK;
}

// out[t, j] = act(gu[t, j]) * gu[t, I + j]: gate columns first, up columns second.
// Reference: crates/kf-backend-cuda/src/kernels/elementwise.cu:42-44.
template <typename TI, typename TO>
__global__ void gated_act_kernel(const TI* __restrict__ gu, TO* __restrict__ out, int T, int I, int act, float limit) {
  kf_pdl_trigger();
  kf_pdl_wait();
  const size_t n = (size_t)T * I;
  for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < n; idx += (size_t)gridDim.x * blockDim.x) {
    const size_t t = idx / I, j = idx - t * I;
    const float g = kf_load(gu, t * 2 * I + j), u = kf_load(gu, t * 2 * I + I + j);
    kf_store(out, idx, act == KF_ACT_CLAMPED_SWISH ? kf_clamped_swish(g, u, limit) : kf_act(g, act) * u);
  }
}

// act 3 (the clamped form, see kf_clamped_swish) reads `limit`.
KF_API int kf_gated_act(const void* gu, int in_dtype, void* out, int out_dtype, int T, int I, int act, float limit,
                        cudaStream_t stream) {
  if (T <= 0) return KF_OK;
  const size_t n = (size_t)T * I;
  const int blocks = (int)((n + 255) / 256 > kf_sm_count() * 16 ? kf_sm_count() * 16 : (n + 255) / 256);
  if (in_dtype == KF_F32 && out_dtype == KF_F32)
    kf_launch(gated_act_kernel<float, float>, dim3(blocks), dim3(256), 0, stream, (const float*)gu, (float*)out, T, I, act, limit);
  else if (in_dtype == KF_F32 && out_dtype == KF_BF16)
    kf_launch(gated_act_kernel<float, __nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, (const float*)gu, (__nv_bfloat16*)out, T, I, act, limit);
  else if (in_dtype == KF_BF16 && out_dtype == KF_BF16)
    kf_launch(gated_act_kernel<__nv_bfloat16, __nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, (const __nv_bfloat16*)gu, (__nv_bfloat16*)out, T, I, act, limit);
  else
    return KF_ERR_DTYPE;
  KF_CHECK_LAUNCH();
  return KF_OK;
}

__global__ void add_kernel(const float* __restrict__ a, float* __restrict__ x, size_t n) {
  kf_pdl_trigger();
  kf_pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) x[i] += a[i];
}

KF_API int kf_add(const float* a, float* x, long n, cudaStream_t stream) {
  if (n <= 0) return KF_OK;
  const long b = (n + 255) / 256;
  kf_launch(add_kernel, dim3((int)(b > kf_sm_count() * 16 ? kf_sm_count() * 16 : b)), dim3(256), 0, stream, a, x, (size_t)n);
  KF_CHECK_LAUNCH();
  return KF_OK;
}

// out = sa * a + sb * b, 32-bit (the results of two mixers that run side by side on one input).
__global__ void weighted_sum2_kernel(const float* __restrict__ a, float sa, const float* __restrict__ b, float sb,
                                     float* __restrict__ out, size_t n) {
  kf_pdl_trigger();
  kf_pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
    out[i] = fmaf(sb, b[i], sa * a[i]);
}

KF_API int kf_weighted_sum2(const float* a, float sa, const float* b, float sb, float* out, long n, cudaStream_t stream) {
  if (n <= 0) return KF_OK;
  const long nb = (n + 255) / 256;
  kf_launch(weighted_sum2_kernel, dim3((int)(nb > kf_sm_count() * 16 ? kf_sm_count() * 16 : nb)), dim3(256), 0, stream, a, sa,
            b, sb, out, (size_t)n);
  KF_CHECK_LAUNCH();
  return KF_OK;
}

// dst = (bf16 or f32) copy of src with conversion; used where a 32-bit weight meets bf16 activations.
template <typename TI, typename TO>
__global__ void convert_kernel(const TI* __restrict__ src, TO* __restrict__ dst, size_t n) {
  kf_pdl_trigger();
  kf_pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
    kf_store(dst, i, kf_load(src, i));
}

KF_API int kf_convert(const void* src, int src_dtype, void* dst, int dst_dtype, long n, cudaStream_t stream) {
  if (n <= 0) return KF_OK;
  const long b = (n + 255) / 256;
  const int blocks = (int)(b > kf_sm_count() * 16 ? kf_sm_count() * 16 : b);
  if (src_dtype == KF_BF16 && dst_dtype == KF_F32)
    kf_launch(convert_kernel<__nv_bfloat16, float>, dim3(blocks), dim3(256), 0, stream, (const __nv_bfloat16*)src, (float*)dst, (size_t)n);
  else if (src_dtype == KF_F32 && dst_dtype == KF_BF16)
    kf_launch(convert_kernel<float, __nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, (const float*)src, (__nv_bfloat16*)dst, (size_t)n);
  else
    return KF_ERR_DTYPE;
  KF_CHECK_LAUNCH();
  return KF_OK;
}

// ---- random weights: a counter-based generator that the host restates bit for bit ---------------------------------
// Element i of a tensor with 64-bit key k: three 64-bit words w_j = mix(k + (3 i + j) * 0x9E3779B97F4A7C15), j = 0..2
// (the splitmix64 finaliser), cut into twelve 16-bit numbers whose sum s has mean 393210 and standard deviation 65536
// (to 1e-10); value = float(s - 393210) * (std / 65536).  Integer arithmetic, one exact conversion and one 32-bit
// multiplication: the same bits on any machine (kungfu_b200/weights/store.py restates it with numpy).  The sum of
// twelve uniforms is bell-shaped within +-6 standard deviations, which is all random test weights need.
// The reference's tests draw their tensors from a small generator of their own the same way
// (crates/kf-backend-cuda/tests/common/mod.rs:71-97).
__host__ __device__ __forceinline__ unsigned long long kf_mix64(unsigned long long z) {
  z = (z ^ (z >> 30)) * 0xBF58476D1CE4E5B9ull;
  z = (z ^ (z >> 27)) * 0x94D049BB133111EBull;
  return z ^ (z >> 31);
}

template <typename TO>
__global__ void random_normal_kernel(TO* __restrict__ out, size_t n, unsigned long long key, float step) {
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
    int s = 0;
#pragma unroll
    for (int j = 0; j < 3; ++j) {
      const unsigned long long w = kf_mix64(key + (3ull * i + j) * 0x9E3779B97F4A7C15ull);
      s += (int)(w & 0xFFFF) + (int)((w >> 16) & 0xFFFF) + (int)((w >> 32) & 0xFFFF) + (int)(w >> 48);
    }
    kf_store(out, i, __fmul_rn((float)(s - 393210), step));
  }
}

__global__ void random_table_kernel(int* __restrict__ out, size_t n, unsigned long long key) {
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
    out[i] = (int)(kf_mix64(key + (3ull * i) * 0x9E3779B97F4A7C15ull) & 0x7FFF);
}

// out[i] = the i-th value of stream `key` times std (32-bit or bfloat16, rounded to nearest even), or, for
// dtype -1, a 15-bit integer.
KF_API int kf_random_fill(void* out, int dtype, long n, unsigned long long key, float std, cudaStream_t stream) {
  if (n <= 0) return KF_OK;
  const long b = (n + 255) / 256;
  const int blocks = (int)(b > kf_sm_count() * 32 ? kf_sm_count() * 32 : b);
  const float step = std / 65536.0f;
  if (dtype == KF_F32) random_normal_kernel<float><<<blocks, 256, 0, stream>>>((float*)out, (size_t)n, key, step);
  else if (dtype == KF_BF16) random_normal_kernel<__nv_bfloat16><<<blocks, 256, 0, stream>>>((__nv_bfloat16*)out, (size_t)n, key, step);
  else if (dtype == -1) random_table_kernel<<<blocks, 256, 0, stream>>>((int*)out, (size_t)n, key);
  else return KF_ERR_DTYPE;
  KF_CHECK_LAUNCH();
  return KF_OK;
}
