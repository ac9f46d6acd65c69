// From a 32-bit stacked projection to the attention's operands, for mixers that norm q and k over the WHOLE projection
// (all heads of a row at once) instead of head by head.
//
// kf_rownorm_rope_append, one block per row of the step:
//   q = in[t, col0 ..] + bias_q,  k = ... + bias_k,  v = ... + bias_v                    (bias optional)
//   q <- q / sqrt(mean over all nh * dk elements of q^2 + eps) * wq[i]   (wq: nh * dk weights; null: no norm), k likewise
//   the first `rot` elements of every head of q and k are turned by the row's angles, pairs (2i, 2i + 1) when
//   `interleaved`, else (i, i + rot/2); cos and sin are multiplied by `mag`
//   value mixing: vmode 1 writes the biased v of the row to v_shared [T, nkv * dv] (32-bit); vmode 2 replaces v by
//   (1 - lambda) v + lambda v_shared[t] (lambda: one number on the device); what was mixed is what is filed
//   v_at: the column (from col0) v starts at, nq + nk for a v of its own, nq where the keys as projected (biased, before norm and
//   rotation) are the values too; its bias stands at the same place
//   q goes to q_out [T, nh * D], k and v to the token's place in the request's pages; heads use D elements, tails zero.
// kf_cols_rmsnorm: out[t, i] = in[t, c0 + i] / sqrt(mean_i(in[t, c0 + i]^2) + eps) * w[i] for a column range of a 32-bit
//   matrix (the normed latent a second projection reads).
// Everything is computed in 32-bit; only the stores round.
#include "common.cuh"

template <typename TW, typename TQ, typename TKV>
__global__ void __launch_bounds__(256)
rownorm_rope_append_kernel(const float* __restrict__ in, int ld, int col0, const TW* __restrict__ bias,
                           const TW* __restrict__ wq, const TW* __restrict__ wk, float eps, const float* __restrict__ cos_t,
                           const float* __restrict__ sin_t, int rot, int interleaved, float mag, int nh, int nkv, int dk,
                           int dv, int D, int v_at, const TW* __restrict__ lambda, float* __restrict__ v_shared, int vmode,
                           const int* __restrict__ positions, const int* __restrict__ row_req,
                           const int* __restrict__ block_table, int table_stride, int page_size, TKV* __restrict__ pages,
                           TQ* __restrict__ q_out, int write_kv, int T) {
  kf_pdl_trigger();
  kf_pdl_wait();
  extern __shared__ float row[];                            // q (nh * dk) then k (nkv * dk), biased
  __shared__ float red[33];
  const int t = blockIdx.x;
  const int req = row_req[t];
  const int nq = nh * dk, nk = nkv * dk, nv = nkv * dv;
  if (req < 0) {                                            // padding row: zero queries, nothing filed
    for (int i = threadIdx.x; i < nh * D; i += blockDim.x) kf_store(q_out, (size_t)t * nh * D + i, 0.f);
    return;
  }
  const float* src = in + (size_t)t * ld + col0;
  float sq = 0.f, sk = 0.f;
  for (int i = threadIdx.x; i < nq + nk; i += blockDim.x) {
    const float x = src[i] + (bias ? kf_load(bias, i) : 0.f);
    row[i] = x;
    if (i < nq) sq = fmaf(x, x, sq); else sk = fmaf(x, x, sk);
  }
  sq = kf_block_sum(sq, red);
  sk = kf_block_sum(sk, red);
  const float inv_q = wq ? 1.f / sqrtf(sq / (float)nq + eps) : 1.f;
  const float inv_k = wk ? 1.f / sqrtf(sk / (float)nk + eps) : 1.f;
  const int half = rot >> 1;
  const float* c = cos_t + (size_t)t * half;
  const float* s = sin_t + (size_t)t * half;
  const int pos = positions[t];
  const int page = block_table[(size_t)req * table_stride + pos / page_size];
  const int in_page = pos % page_size;
  const bool file = write_kv && page >= 0;
  const int n_heads_qk = nh + (file ? nkv : 0);
  for (int i = threadIdx.x; i < n_heads_qk * D; i += blockDim.x) {
    const int hs = i / D, e = i - hs * D;
    const bool is_q = hs < nh;
    const int head = is_q ? hs : hs - nh;
    float y = 0.f;
    if (e < dk) {
      const int base = (is_q ? 0 : nq) + head * dk;
      const TW* w = is_q ? wq : wk;
      const float inv = is_q ? inv_q : inv_k;
      const int wbase = head * dk;
      auto normed = [&](int j) { return row[base + j] * inv * (w ? kf_load(w, wbase + j) : 1.f); };
      y = normed(e);
      if (e < rot) {
        int pair, partner;
        bool first;
        if (interleaved) { pair = e >> 1; first = !(e & 1); partner = e ^ 1; }
        else { first = e < half; pair = first ? e : e - half; partner = first ? e + half : e - half; }
        const float cs = c[pair] * mag, sn = s[pair] * mag, o = normed(partner);
        y = first ? y * cs - o * sn : y * cs + o * sn;
      }
    }
    if (is_q) kf_store(q_out, ((size_t)t * nh + head) * D + e, y);
    else kf_store(pages, ((((size_t)page * 2 + 0) * nkv + head) * page_size + in_page) * D + e, y);
  }
  if (!write_kv) return;
  const float lam = (vmode == 2 && lambda) ? kf_load(lambda, 0) : 0.f;
  for (int i = threadIdx.x; i < nkv * D; i += blockDim.x) {
    const int head = i / D, e = i - head * D;
    float y = 0.f;
    if (e < dv) {
      const int j = head * dv + e;
      y = src[v_at + j] + (bias ? kf_load(bias, v_at + j) : 0.f);
      if (vmode == 1) v_shared[(size_t)t * nv + j] = y;
      else if (vmode == 2) y = (1.f - lam) * y + lam * v_shared[(size_t)t * nv + j];
    }
    if (page >= 0) kf_store(pages, ((((size_t)page * 2 + 1) * nkv + head) * page_size + in_page) * D + e, y);
  }
}

// The same with 16-byte loads and 8- or 16-byte stores, four neighbouring elements of a head per thread and turn: sizes and
// offsets are multiples of four elements, and a group of four lies in one half of the rotated part (halves of a multiple
// of four) or holds two whole pairs (interleaved).  The step's integers are read before the grid dependency is waited for.
__device__ __forceinline__ float4 rq_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 rq_load4(const __nv_bfloat16* p) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void rq_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void rq_store4(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

template <typename TW, typename TQ, typename TKV>
__global__ void __launch_bounds__(512)
rownorm_rope_append4_kernel(const float* in, int ld, int col0, const TW* __restrict__ bias,
                            const TW* __restrict__ wq, const TW* __restrict__ wk, float eps, const float* cos_t,
                            const float* sin_t, int rot, int interleaved, float mag, int nh, int nkv, int dk,
                            int dv, int D, int v_at, const TW* __restrict__ lambda, float* v_shared, int vmode,
                            const int* __restrict__ positions, const int* __restrict__ row_req,
                            const int* __restrict__ block_table, int table_stride, int page_size, TKV* __restrict__ pages,
                            TQ* __restrict__ q_out, int write_kv) {
  kf_pdl_trigger();
  extern __shared__ __align__(16) float row[];              // q (nh * dk) then k (nkv * dk), biased
  __shared__ float red[33];
  const int t = blockIdx.x, tid = threadIdx.x, nt = blockDim.x;
  const int req = row_req[t], pos = positions[t];
  const int page = req >= 0 ? block_table[(size_t)req * table_stride + pos / page_size] : -1;
  const int in_page = pos % page_size;
  const int nq = nh * dk, nk = nkv * dk, nv = nkv * dv;
  kf_pdl_wait();
  in = kf_produced(in), cos_t = kf_produced(cos_t), sin_t = kf_produced(sin_t), v_shared = kf_produced(v_shared);
  if (req < 0) {                                            // padding row: zero queries, nothing filed
    for (int i = tid * 4; i < nh * D; i += nt * 4) rq_store4(q_out + (size_t)t * nh * D + i, make_float4(0.f, 0.f, 0.f, 0.f));
    return;
  }
  const float* src = in + (size_t)t * ld + col0;
  float sq = 0.f, sk = 0.f;
  for (int i = tid * 4; i < nq + nk; i += nt * 4) {
    float4 x = rq_load4(src + i);
    if (bias) { const float4 b = rq_load4(bias + i); x.x += b.x; x.y += b.y; x.z += b.z; x.w += b.w; }
    *reinterpret_cast<float4*>(row + i) = x;
    const float s = fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, x.w * x.w)));
    if (i < nq) sq += s; else sk += s;
  }
  sq = kf_block_sum(sq, red);
  sk = kf_block_sum(sk, red);
  const float inv_q = wq ? 1.f / sqrtf(sq / (float)nq + eps) : 1.f;
  const float inv_k = wk ? 1.f / sqrtf(sk / (float)nk + eps) : 1.f;
  const int half = rot >> 1, per = D >> 2;
  const float* c = cos_t + (size_t)t * half;
  const float* s = sin_t + (size_t)t * half;
  const bool file = write_kv && page >= 0;
  const int groups = (nh + (file ? nkv : 0)) * per;
  for (int i = tid; i < groups; i += nt) {
    const int hs = i / per, e = (i - hs * per) * 4;
    const bool is_q = hs < nh;
    const int head = is_q ? hs : hs - nh;
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
    if (e < dk) {
      const float* base = row + (is_q ? 0 : nq) + head * dk;
      const TW* w = is_q ? wq : wk;
      const float inv = is_q ? inv_q : inv_k;
      auto normed4 = [&](int j) {
        const float4 x = *reinterpret_cast<const float4*>(base + j);
        const float4 g = w ? rq_load4(w + head * dk + j) : make_float4(1.f, 1.f, 1.f, 1.f);
        return make_float4(x.x * inv * g.x, x.y * inv * g.y, x.z * inv * g.z, x.w * inv * g.w);
      };
      y = normed4(e);
      if (e < rot) {
        if (interleaved) {
          const int p = e >> 1;
          const float c0 = c[p] * mag, s0 = s[p] * mag, c1 = c[p + 1] * mag, s1 = s[p + 1] * mag;
          y = make_float4(y.x * c0 - y.y * s0, y.y * c0 + y.x * s0, y.z * c1 - y.w * s1, y.w * c1 + y.z * s1);
        } else {
          const bool first = e < half;
          const int p = first ? e : e - half;
          const float4 o = normed4(first ? e + half : e - half);
          const float4 cs = rq_load4(c + p), sn = rq_load4(s + p);
          const float sg = first ? -mag : mag;
          y = make_float4(y.x * (cs.x * mag) + o.x * (sn.x * sg), y.y * (cs.y * mag) + o.y * (sn.y * sg),
                          y.z * (cs.z * mag) + o.z * (sn.z * sg), y.w * (cs.w * mag) + o.w * (sn.w * sg));
        }
      }
    }
    if (is_q) rq_store4(q_out + ((size_t)t * nh + head) * D + e, y);
    else rq_store4(pages + ((((size_t)page * 2 + 0) * nkv + head) * page_size + in_page) * D + e, y);
  }
  if (!write_kv) return;
  const float lam = (vmode == 2 && lambda) ? kf_load(lambda, 0) : 0.f;
  for (int i = tid; i < nkv * per; i += nt) {
    const int head = i / per, e = (i - head * per) * 4;
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
    if (e < dv) {
      const int j = head * dv + e;
      y = rq_load4(src + v_at + j);
      if (bias) { const float4 b = rq_load4(bias + v_at + j); y.x += b.x; y.y += b.y; y.z += b.z; y.w += b.w; }
      if (vmode == 1) *reinterpret_cast<float4*>(v_shared + (size_t)t * nv + j) = y;
      else if (vmode == 2) {
        const float4 f = rq_load4(v_shared + (size_t)t * nv + j);
        y = make_float4((1.f - lam) * y.x + lam * f.x, (1.f - lam) * y.y + lam * f.y, (1.f - lam) * y.z + lam * f.z,
                        (1.f - lam) * y.w + lam * f.w);
      }
    }
    if (page >= 0) rq_store4(pages + ((((size_t)page * 2 + 1) * nkv + head) * page_size + in_page) * D + e, y);
  }
}

KF_API int kf_rownorm_rope_append(const float* in, int ld, int col0, const void* bias, const void* wq, const void* wk,
                                  int w_dtype, float eps, const float* cos_t, const float* sin_t, int rot, int interleaved,
                                  float mag, int nh, int nkv, int dk, int dv, int D, int v_at, const void* lambda, float* v_shared,
                                  int vmode, const int* positions, const int* row_req, const int* block_table,
                                  int table_stride, int page_size, void* pages, int kv_dtype, void* q_out, int q_dtype,
                                  int write_kv, int T, cudaStream_t stream) {
  if (T <= 0) return KF_OK;
  if (dk > D || dv > D || dk < 1 || dv < 1 || rot > dk || (rot & 1) || nkv < 1 || nh % nkv) return KF_ERR_SIZE;
  if (rot > 0 && (!cos_t || !sin_t)) return KF_ERR_SIZE;
  if (vmode != 0 && !v_shared) return KF_ERR_SIZE;
  if (v_at < 0 || col0 + v_at + nkv * dv > ld) return KF_ERR_SIZE;
  const size_t smem = (size_t)(nh + nkv) * dk * sizeof(float);
  if (smem > 200 * 1024) return KF_ERR_SIZE;
  const bool by4 = dk % 4 == 0 && dv % 4 == 0 && D % 4 == 0 && v_at % 4 == 0 && ld % 4 == 0 && col0 % 4 == 0 &&
                   rot % (interleaved ? 4 : 8) == 0 &&
                   (((uintptr_t)in | (uintptr_t)bias | (uintptr_t)wq | (uintptr_t)wk | (uintptr_t)cos_t | (uintptr_t)sin_t |
                     (uintptr_t)v_shared | (uintptr_t)pages | (uintptr_t)q_out) & 15) == 0;
  const int threads = (nh + nkv) * D >= 2048 ? 512 : ((nh + nkv) * D >= 1024 ? 256 : 128);
#define KF_GO(TW, TQ, TKV)                                                                                              \
  do {                                                                                                                  \
    if (by4) {                                                                                                          \
      if (smem > 48 * 1024)                                                                                             \
        cudaFuncSetAttribute(rownorm_rope_append4_kernel<TW, TQ, TKV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
      kf_launch(rownorm_rope_append4_kernel<TW, TQ, TKV>, dim3(T), dim3(threads), smem, stream, in, ld, col0, (const TW*)bias, \
                (const TW*)wq, (const TW*)wk, eps, cos_t, sin_t, rot, interleaved, mag, nh, nkv, dk, dv, D, v_at,      \
                (const TW*)lambda, v_shared, vmode, positions, row_req, block_table, table_stride, page_size,          \
                (TKV*)pages, (TQ*)q_out, write_kv);                                                                     \
      break;                                                                                                            \
    }                                                                                                                   \
    if (smem > 48 * 1024)                                                                                               \
      cudaFuncSetAttribute(rownorm_rope_append_kernel<TW, TQ, TKV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    kf_launch(rownorm_rope_append_kernel<TW, TQ, TKV>, dim3(T), dim3(256), smem, stream, in, ld, col0, (const TW*)bias,  \
              (const TW*)wq, (const TW*)wk, eps, cos_t, sin_t, rot, interleaved, mag, nh, nkv, dk, dv, D, v_at,        \
              (const TW*)lambda, v_shared, vmode, positions, row_req, block_table, table_stride, page_size,            \
              (TKV*)pages, (TQ*)q_out, write_kv, T);                                                                    \
  } while (0)
  if (w_dtype == KF_F32 && q_dtype == KF_F32 && kv_dtype == KF_F32) KF_GO(float, float, float);
  else if (w_dtype == KF_BF16 && q_dtype == KF_BF16 && kv_dtype == KF_BF16) KF_GO(__nv_bfloat16, __nv_bfloat16, __nv_bfloat16);
  else if (w_dtype == KF_BF16 && q_dtype == KF_F32 && kv_dtype == KF_F32) KF_GO(__nv_bfloat16, float, float);
  else if (w_dtype == KF_F32 && q_dtype == KF_BF16 && kv_dtype == KF_BF16) KF_GO(float, __nv_bfloat16, __nv_bfloat16);
  else return KF_ERR_DTYPE;
#undef KF_GO
  KF_CHECK_LAUNCH();
  return KF_OK;
}

template <typename TW, typename TO>
__global__ void __launch_bounds__(128) cols_rmsnorm_kernel(const float* __restrict__ in, int ld, int c0, int n,
                                                           const TW* __restrict__ w, float eps, TO* __restrict__ out) {
  kf_pdl_trigger();
  kf_pdl_wait();
  __shared__ float red[33];
  const int t = blockIdx.x;
  const float* src = in + (size_t)t * ld + c0;
  float ss = 0.f;
  for (int i = threadIdx.x; i < n; i += blockDim.x) ss = fmaf(src[i], src[i], ss);
  ss = kf_block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / (float)n + eps);
  for (int i = threadIdx.x; i < n; i += blockDim.x) kf_store(out, (size_t)t * n + i, src[i] * inv * kf_load(w, i));
}

KF_API int kf_cols_rmsnorm(const float* in, int ld, int c0, int n, const void* w, int w_dtype, float eps, void* out,
                           int out_dtype, int T, cudaStream_t stream) {
  if (T <= 0) return KF_OK;
  if (n < 1 || c0 < 0 || c0 + n > ld) return KF_ERR_SIZE;
#define KF_GO(TW, TO) kf_launch(cols_rmsnorm_kernel<TW, TO>, dim3(T), dim3(128), 0, stream, in, ld, c0, n, (const TW*)w, eps, (TO*)out)
  if (w_dtype == KF_F32 && out_dtype == KF_F32) KF_GO(float, float);
  else if (w_dtype == KF_BF16 && out_dtype == KF_BF16) KF_GO(__nv_bfloat16, __nv_bfloat16);
  else if (w_dtype == KF_BF16 && out_dtype == KF_F32) KF_GO(__nv_bfloat16, float);
  else if (w_dtype == KF_F32 && out_dtype == KF_BF16) KF_GO(float, __nv_bfloat16);
  else return KF_ERR_DTYPE;
#undef KF_GO
  KF_CHECK_LAUNCH();
  return KF_OK;
}
