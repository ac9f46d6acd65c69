// The convolution in front of a sublayer that reads the residual stream itself:
//   out_t[c] = h_t[c] + sum_j w[c][j] h_(t - taps + 1 + j)[c],  j = 0..taps-1,  zeros before the sequence's first token
// (a short causal convolution over time, one filter per channel, added to its own input).  h is 32-bit, the result goes
// to the element type the sublayer's products take.
//
// A step brings only some rows of a request, so its last taps-1 inputs are kept: state[slot][s][c] is the input at
// sequence index length - (taps-1) + s (zeros at admission).  The state of a request is read and moved on by ONE thread per
// channel group: the owner of the request's first row of the step also computes the rows that still reach into the
// state (the first taps-1 of them), and writes the new tail when it has read the old one.  So no second launch is needed.
//
// kf_input_conv:         the above for every row of a step.
// kf_add_rmsnorm_conv:   steps in which no request has more than one row: x += rmsnorm(a) * w1 and the convolution of the
//                        new x, in one launch (a block per row).
#include "common.cuh"

namespace {

constexpr int IC_MAX_TAPS = 8;
constexpr int IC_FAST_ROWS = 8;              // rows per block of a long prompt

template <int VEC>
__device__ __forceinline__ void ic_load(const float* p, float* v) {
  if constexpr (VEC == 4) {
    const float4 q = *reinterpret_cast<const float4*>(p);
    v[0] = q.x, v[1] = q.y, v[2] = q.z, v[3] = q.w;
  } else v[0] = p[0];
}
template <int VEC>
__device__ __forceinline__ void ic_store(float* p, const float* v) {
  if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else p[0] = v[0];
}
template <int VEC>
__device__ __forceinline__ void ic_store(__nv_bfloat16* p, const float* v) {
  if constexpr (VEC == 4) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  } else p[0] = __float2bfloat16_rn(v[0]);
}

__device__ __forceinline__ void ic_load4(const float* p, float* v) {
  const float4 q = *reinterpret_cast<const float4*>(p);
  v[0] = q.x, v[1] = q.y, v[2] = q.z, v[3] = q.w;
}
__device__ __forceinline__ void ic_load4(const __nv_bfloat16* p, float* v) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
  v[0] = a.x, v[1] = a.y, v[2] = b.x, v[3] = b.y;
}

// VEC channels per thread, `rows` rows per block; within a run of rows of one request the last taps inputs stay in
// registers, so every row is read once per block.
template <typename TW, typename TO, int TAPS, int VEC>
__global__ void __launch_bounds__(256)
input_conv_kernel(const float* __restrict__ x, const TW* __restrict__ w, float* __restrict__ state, TO* __restrict__ out,
                  int C, const int* __restrict__ row_req, const int* __restrict__ req_row_start,
                  const int* __restrict__ req_n_rows, const int* __restrict__ req_state_slot, int T, int rows, int writes) {
  kf_pdl_trigger();
  const int c0 = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  if (c0 >= C) return;
  constexpr int TAIL = TAPS - 1;
  constexpr int FAST = TAPS <= 4 ? IC_FAST_ROWS : 0;
  float wv[VEC][TAPS];                                 // the filters of VEC channels stand one after another
  if constexpr (VEC == 4) {
    float flat[4 * TAPS];
#pragma unroll
    for (int q = 0; q < TAPS; ++q) ic_load4(w + (size_t)c0 * TAPS + 4 * q, flat + 4 * q);
#pragma unroll
    for (int v = 0; v < 4; ++v)
#pragma unroll
      for (int j = 0; j < TAPS; ++j) wv[v][j] = flat[v * TAPS + j];
  } else {
#pragma unroll
    for (int j = 0; j < TAPS; ++j) wv[0][j] = kf_load(w, (size_t)c0 * TAPS + j);
  }
  kf_pdl_wait();
  x = kf_produced(x);
  float u[TAPS][VEC];                                  // the inputs of the row in hand, oldest first
  auto emit = [&](int t) {
    float y[VEC];
#pragma unroll
    for (int v = 0; v < VEC; ++v) {
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) acc = fmaf(wv[v][j], u[j][v], acc);
      y[v] = u[TAPS - 1][v] + acc;
    }
    ic_store<VEC>(out + (size_t)t * C + c0, y);
  };
  auto shift = [&]() {
#pragma unroll
    for (int j = 0; j + 1 < TAPS; ++j)
#pragma unroll
      for (int v = 0; v < VEC; ++v) u[j][v] = u[j + 1][v];
  };
  const int t_first = blockIdx.x * rows, t_end = min(T, t_first + rows);
  // The ordinary block of a long prompt: all its rows belong to one request and see only this step's inputs.  Every load is
  // then requested before the first sum.
  if (FAST > 0 && t_end - t_first == FAST && rows == FAST) {
    const int req = row_req[t_first];
    if (req >= 0 && row_req[t_end - 1] == req && t_first - req_row_start[req] >= (TAIL > 0 ? TAIL : 1)) {
      float in[FAST > 0 ? FAST + TAIL : 1][VEC];
#pragma unroll
      for (int j = 0; j < FAST + TAIL; ++j) ic_load<VEC>(x + (size_t)(t_first - TAIL + j) * C + c0, in[j]);
#pragma unroll
      for (int r = 0; r < FAST; ++r) {
        float y[VEC];
#pragma unroll
        for (int v = 0; v < VEC; ++v) {
          float acc = 0.f;
#pragma unroll
          for (int j = 0; j < TAPS; ++j) acc = fmaf(wv[v][j], in[r + j][v], acc);
          y[v] = in[r + TAIL][v] + acc;
        }
        ic_store<VEC>(out + (size_t)(t_first + r) * C + c0, y);
      }
      return;
    }
  }
  int held = -2;                                       // the row whose inputs u holds (-2: none)
  for (int t = t_first; t < t_end; ++t) {
    const int req = row_req[t];
    if (req < 0) { held = -2; continue; }
    const int row0 = req_row_start[req], i = t - row0;
    if (i >= TAIL && i > 0) {                          // every input lies in this step
      if (held == t - 1) {
        shift();
        ic_load<VEC>(x + (size_t)t * C + c0, u[TAPS - 1]);
      } else {
#pragma unroll
        for (int j = 0; j < TAPS; ++j) ic_load<VEC>(x + (size_t)(t - TAIL + j) * C + c0, u[j]);
      }
      held = t;
      emit(t);
      continue;
    }
    if (i > 0) { held = -2; continue; }                // the owner of the request's first row computes this one
    const int n = req_n_rows[req];
    float* st = state + (size_t)req_state_slot[req] * TAIL * C + c0;
#pragma unroll
    for (int s = 0; s < TAIL; ++s) ic_load<VEC>(st + (size_t)s * C, u[s]);
    ic_load<VEC>(x + (size_t)row0 * C + c0, u[TAPS - 1]);
    emit(row0);
#pragma unroll
    for (int r = 1; r < TAIL; ++r)
      if (r < n) {
        shift();
        ic_load<VEC>(x + (size_t)(row0 + r) * C + c0, u[TAPS - 1]);
        emit(row0 + r);
      }
    held = -2;
    if (TAIL > 0 && writes) {
      if (n >= TAIL) {
#pragma unroll
        for (int s = 0; s < TAIL; ++s) {
          float v[VEC];
          ic_load<VEC>(x + (size_t)(row0 + n - TAIL + s) * C + c0, v);
          ic_store<VEC>(st + (size_t)s * C, v);
        }
      } else {                                         // u ends with row n - 1: its last TAIL inputs are the new tail
#pragma unroll
        for (int s = 0; s < TAIL; ++s) ic_store<VEC>(st + (size_t)s * C, u[s + 1]);
      }
    }
  }
}

// One block per row, every request of the step with at most one row: the row, its tail and the filters in registers.
template <typename TW, typename TO, int TAPS, int NPT>
__global__ void __launch_bounds__(512)
add_rmsnorm_conv_kernel(const float* a, const TW* __restrict__ w1, float eps, float* x, const TW* __restrict__ w,
                        float* state, TO* __restrict__ out, int H, const int* __restrict__ row_req,
                        const int* __restrict__ req_state_slot, int writes) {
  kf_pdl_trigger();
  __shared__ float red[33];
  constexpr int TAIL = TAPS - 1;
  const int r = blockIdx.x;
  const int req = row_req[r];                          // the step's integers, weights and earlier steps' tails: readable at once
  float g[NPT], wv[NPT][TAPS], tail[NPT][TAIL > 0 ? TAIL : 1];
  float* st = state + (size_t)(req >= 0 ? req_state_slot[req] : 0) * TAIL * H;
#pragma unroll
  for (int k = 0; k < NPT; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    g[k] = i < H ? kf_load(w1, i) : 0.f;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) wv[k][j] = i < H ? kf_load(w, (size_t)i * TAPS + j) : 0.f;
#pragma unroll
    for (int s = 0; s < TAIL; ++s) tail[k][s] = (i < H && req >= 0) ? st[(size_t)s * H + i] : 0.f;
  }
  kf_pdl_wait();
  a = kf_produced(a), x = kf_produced(x);
  const float* ar = a + (size_t)r * H;
  float* xr = x + (size_t)r * H;
  float v[NPT], xv[NPT];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < NPT; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    v[k] = i < H ? ar[i] : 0.f;
    xv[k] = i < H ? xr[i] : 0.f;
    ss += v[k] * v[k];
  }
  ss = kf_block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / (float)H + eps);
#pragma unroll
  for (int k = 0; k < NPT; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < H) {
      const float h = xv[k] + v[k] * inv * g[k];
      xr[i] = h;
      float acc = 0.f;
#pragma unroll
      for (int s = 0; s < TAIL; ++s) acc = fmaf(wv[k][s], tail[k][s], acc);
      acc = fmaf(wv[k][TAPS - 1], h, acc);
      kf_store(out, (size_t)r * H + i, h + acc);
      if (req >= 0 && writes) {
#pragma unroll
        for (int s = 0; s < TAIL; ++s) st[(size_t)s * H + i] = s + 1 < TAIL ? tail[k][s + 1] : h;
      }
    }
  }
}

}  // namespace

#define KF_TAPS_SWITCH(taps, GO)                                                                                    \
  switch (taps) {                                                                                                   \
    case 1: GO(1); break; case 2: GO(2); break; case 3: GO(3); break; case 4: GO(4); break;                         \
    case 5: GO(5); break; case 6: GO(6); break; case 7: GO(7); break; case 8: GO(8); break;                         \
    default: return KF_ERR_SIZE;                                                                                    \
  }

// x [T, C] 32-bit, w [C, taps], state [slots, taps - 1, C] 32-bit (null when taps is 1), out [T, C]; taps 1 to 8.
KF_API int kf_input_conv(const float* x, const void* w, int w_dtype, int C, int taps, float* state, void* out, int out_dtype,
                         const int* row_req, const int* req_row_start, const int* req_n_rows, const int* req_state_slot,
                         int T, int writes, cudaStream_t stream) {
  if (T <= 0 || C <= 0) return KF_OK;
  if (taps < 1 || taps > IC_MAX_TAPS || (taps > 1 && !state)) return KF_ERR_SIZE;
  const bool vec = C % 4 == 0 && (((uintptr_t)x | (uintptr_t)w | (uintptr_t)state | (uintptr_t)out) & 15) == 0;
  const int per_thread = vec ? 4 : 1;
  const int threads = C / per_thread >= 256 ? 256 : 128;
  const int rows = T >= 512 ? IC_FAST_ROWS : (T >= 64 ? 4 : 1);
  const dim3 grid(kf_ceil_div(T, rows), kf_ceil_div(C, threads * per_thread));
#define KF_LAUNCH(TW, TO, TAPS, VEC)                                                                                  \
  kf_launch(input_conv_kernel<TW, TO, TAPS, VEC>, grid, dim3(threads), 0, stream, x, (const TW*)w, state, (TO*)out, C, row_req, \
            req_row_start, req_n_rows, req_state_slot, T, rows, writes)
#define KF_GO_FF(N) do { if (vec) KF_LAUNCH(float, float, N, 4); else KF_LAUNCH(float, float, N, 1); } while (0)
#define KF_GO_BB(N) do { if (vec) KF_LAUNCH(__nv_bfloat16, __nv_bfloat16, N, 4); else KF_LAUNCH(__nv_bfloat16, __nv_bfloat16, N, 1); } while (0)
  if (w_dtype == KF_F32 && out_dtype == KF_F32) { KF_TAPS_SWITCH(taps, KF_GO_FF) }
  else if (w_dtype == KF_BF16 && out_dtype == KF_BF16) { KF_TAPS_SWITCH(taps, KF_GO_BB) }
  else return KF_ERR_DTYPE;
#undef KF_GO_FF
#undef KF_GO_BB
#undef KF_LAUNCH
  KF_CHECK_LAUNCH();
  return KF_OK;
}

// Rows of up to 4096 elements (above, a thread's part of the row, its tails and filters no longer fit its registers); w1 (the norm's weights) and w share one element type.
KF_API int kf_add_rmsnorm_conv_supported(int H, int taps) { return H >= 1 && H <= 4096 && taps >= 1 && taps <= 4; }

KF_API int kf_add_rmsnorm_conv(const float* a, const void* w1, const void* w, int w_dtype, float eps, float* x, int taps,
                               float* state, void* out, int out_dtype, const int* row_req, const int* req_state_slot, int T,
                               int H, int writes, cudaStream_t stream) {
  if (T <= 0) return KF_OK;
  if (!kf_add_rmsnorm_conv_supported(H, taps) || (taps > 1 && !state)) return KF_ERR_SIZE;
  const int threads = H > 1024 ? 512 : (H >= 512 ? 256 : 128);
  const int npt = kf_ceil_div(H, threads);
#define KF_LAUNCH(TW, TO, TAPS, NPT)                                                                                   \
  kf_launch(add_rmsnorm_conv_kernel<TW, TO, TAPS, NPT>, dim3(T), dim3(threads), 0, stream, a, (const TW*)w1, eps, x, \
            (const TW*)w, state, (TO*)out, H, row_req, req_state_slot, writes)
#define KF_PICK(TW, TO, TAPS)                                                                                         \
  do {                                                                                                                \
    if (npt <= 4) KF_LAUNCH(TW, TO, TAPS, 4);                                                               \
    else KF_LAUNCH(TW, TO, TAPS, 8);                                                                             \
  } while (0)
#define KF_GO(TW, TO)                                                                                                 \
  do {                                                                                                                \
    if (taps == 1) KF_PICK(TW, TO, 1); else if (taps == 2) KF_PICK(TW, TO, 2);                                        \
    else if (taps == 3) KF_PICK(TW, TO, 3); else KF_PICK(TW, TO, 4);                                                  \
  } while (0)
  if (w_dtype == KF_F32 && out_dtype == KF_F32) KF_GO(float, float);
  else if (w_dtype == KF_BF16 && out_dtype == KF_BF16) KF_GO(__nv_bfloat16, __nv_bfloat16);
  else return KF_ERR_DTYPE;
#undef KF_GO
#undef KF_PICK
#undef KF_LAUNCH
  KF_CHECK_LAUNCH();
  return KF_OK;
}
