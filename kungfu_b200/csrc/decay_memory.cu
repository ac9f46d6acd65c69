// Linear attention with one fixed decay per head, over the rows of every request of a step, from and into a 32-bit state:
//   S_t = a_h S_(t-1) + k_t v_t^T      (S: d x dv per head, zero at admission)
//   o_t = S_t^T q_t
// q, k, v are column ranges of rows laid out head by head: either 32-bit projection results, to which an activation is
// applied as they are read (act 1: silu), or bfloat16 rows that have been through it.  Results are 32-bit [rows, H dv].
// q and k may be turned as they are read (32-bit rows): pairs (i, i + rot/2) of every head's first `rot` elements by the
// step's cos/sin table, k then multiplied by `kscale`; decay_rotate_kernel does the same ahead of the tensor cores.
// `powers` [H, n_powers] holds a_h^0, a_h^1, ... (made in 64-bit on the host): a decay is never the result of a device-side
// power, and ratios a^i / a^j never appear, so any decay in [0, 1] is exact.
//
// Three kernels:
//   decay_decode_kernel   no request of the step has more than one row: a block per (row, head, 32 value columns); the
//                         state goes through registers once, 16 bytes at a time.
//   decay_walk_kernel     any sizes and element types, row by row in 32-bit arithmetic.
//   decay_chunk_kernel    bfloat16 rows on the tensor cores, 64 rows at a time:  with S the state before the 64 rows,
//                         i, j rows of them (0-based) and n their number,
//                           O_i   = a^(i+1) (q_i S) + sum_(j<=i) a^(i-j) (q_i . k_j) v_j
//                           S    <- a^n S + sum_j (a^(n-1-j) k_j) v_j^T
//                         S stays in 32-bit accumulators.  Operands that are not 16-bit numbers to begin with (S, the decayed
//                         keys, the decayed scores) enter their products as the sum of two bfloat16 numbers, so that
//                         nothing of the recurrence is rounded to 8 bits.
//                         A step with few (request, head) pairs is cut into chunks of rows that are walked side by side:
//                         a first pass gives every chunk's own contribution to the state, decay_chunk_starts_kernel turns
//                         them into the states the chunks start from, and the second pass walks the chunks from those.
#include "common.cuh"
#include "mma_tiles.cuh"

namespace {

__device__ __forceinline__ float dm_act(float x, int act) { return act ? x / (1.f + expf(-x)) : x; }

struct DecayArgs {
  const void* q; const void* k; const void* v;       // row 0, column 0 of head 0
  int ldq, ldk, ldv, act;
  const float* powers; int n_powers;
  float* state;                                       // [slots, H, d, dv]
  float* out;                                         // [rows, H dv]
  int H, d, dv, n_reqs;
  const int* row_start; const int* n_rows; const int* slot;
  int writes;
  const float* cos; const float* sin; int rot;       // 0: nothing is turned
  float kscale;
};

// Element i of a head of q or k at row t: activated, then turned.
template <typename T>
__device__ __forceinline__ float dm_turned(const DecayArgs& a, const T* p, const float* cos, const float* sin, int t, int i) {
  const float x = dm_act(kf_load(p, i), a.act);
  if (i >= a.rot) return x;
  const int half = a.rot >> 1, e = i < half ? i : i - half;
  const float y = dm_act(kf_load(p, i < half ? i + half : e), a.act);
  const float c = cos[(size_t)t * half + e], s = sin[(size_t)t * half + e];
  return i < half ? fmaf(x, c, -y * s) : fmaf(x, c, y * s);
}

// ---- one row per request -------------------------------------------------------------------------------------------

constexpr int DD_COLS = 32;
constexpr int DD_THREADS = 256;

template <typename T, int NR>                          // NR rows of the state per thread: d <= 32 NR
__global__ void __launch_bounds__(DD_THREADS) decay_decode_kernel(DecayArgs p) {
  kf_pdl_trigger();
  __shared__ float qs[32 * NR], ks[32 * NR];
  __shared__ __align__(16) float vs[DD_COLS];
  __shared__ __align__(16) float4 red[8][8];
  const int tiles = (p.dv + DD_COLS - 1) / DD_COLS;
  const int tile = blockIdx.x % tiles, rh = blockIdx.x / tiles;
  const int h = rh % p.H, r = rh / p.H;
  if (p.n_rows[r] <= 0 || p.slot[r] < 0) return;
  const int t = p.row_start[r];
  const int tid = threadIdx.x, c4 = tid & 7, r0 = tid >> 3;
  const int col = tile * DD_COLS + c4 * 4;
  const bool live = col < p.dv;                        // dv is a multiple of four
  float* S = p.state + ((size_t)p.slot[r] * p.H + h) * p.d * p.dv + col;
  const float a = p.powers[(size_t)h * p.n_powers + 1];
  float4 s[NR];                                        // an earlier step left the state: readable at once
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int row = r0 + 32 * j;
    s[j] = (live && row < p.d) ? *reinterpret_cast<const float4*>(S + (size_t)row * p.dv) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  kf_pdl_wait();
  const T* q = kf_produced((const T*)p.q) + (size_t)t * p.ldq + h * p.d;
  const T* k = kf_produced((const T*)p.k) + (size_t)t * p.ldk + h * p.d;
  const T* v = kf_produced((const T*)p.v) + (size_t)t * p.ldv + h * p.dv;
  const float* cos = kf_produced(p.cos);
  const float* sin = kf_produced(p.sin);
  for (int i = tid; i < p.d; i += DD_THREADS) {
    qs[i] = dm_turned(p, q, cos, sin, t, i);
    ks[i] = dm_turned(p, k, cos, sin, t, i) * p.kscale;
  }
  if (tid < DD_COLS && tile * DD_COLS + tid < p.dv) vs[tid] = dm_act(kf_load(v, tile * DD_COLS + tid), p.act);
  __syncthreads();
  const float4 vv = live ? *reinterpret_cast<const float4*>(vs + c4 * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int row = r0 + 32 * j;
    if (live && row < p.d) {
      const float kk = ks[row], qq = qs[row];
      s[j].x = fmaf(a, s[j].x, kk * vv.x); s[j].y = fmaf(a, s[j].y, kk * vv.y);
      s[j].z = fmaf(a, s[j].z, kk * vv.z); s[j].w = fmaf(a, s[j].w, kk * vv.w);
      acc.x = fmaf(qq, s[j].x, acc.x); acc.y = fmaf(qq, s[j].y, acc.y);
      acc.z = fmaf(qq, s[j].z, acc.z); acc.w = fmaf(qq, s[j].w, acc.w);
      if (p.writes) *reinterpret_cast<float4*>(S + (size_t)row * p.dv) = s[j];
    }
  }
#pragma unroll
  for (int o = 8; o <= 16; o <<= 1) {
    acc.x += __shfl_xor_sync(0xffffffffu, acc.x, o); acc.y += __shfl_xor_sync(0xffffffffu, acc.y, o);
    acc.z += __shfl_xor_sync(0xffffffffu, acc.z, o); acc.w += __shfl_xor_sync(0xffffffffu, acc.w, o);
  }
  if ((tid & 31) < 8) red[tid >> 5][c4] = acc;
  __syncthreads();
  if (tid < 8 && live) {
    float4 o = red[0][tid];
#pragma unroll
    for (int w = 1; w < 8; ++w) { o.x += red[w][tid].x; o.y += red[w][tid].y; o.z += red[w][tid].z; o.w += red[w][tid].w; }
    *reinterpret_cast<float4*>(p.out + (size_t)t * p.H * p.dv + h * p.dv + col) = o;
  }
}

// ---- any sizes, row by row -----------------------------------------------------------------------------------------

constexpr int DW_R = 8;                                // rows of the state per thread
constexpr int DW_COLS = 16;                            // value columns per block
constexpr int DW_CHUNK = 16;                           // rows of the step staged at a time

template <typename T, int LANES>
__global__ void __launch_bounds__(LANES * DW_COLS) decay_walk_kernel(DecayArgs p) {
  kf_pdl_trigger();
  kf_pdl_wait();
  constexpr int THREADS = LANES * DW_COLS, DP = DW_R * LANES;
  __shared__ __align__(16) float qs[DW_CHUNK][DP];
  __shared__ __align__(16) float ks[DW_CHUNK][DP];
  __shared__ float vs[DW_CHUNK][DW_COLS];
  const int col_blocks = (p.dv + DW_COLS - 1) / DW_COLS;
  const int cb = blockIdx.x % col_blocks, rh = blockIdx.x / col_blocks;
  const int h = rh % p.H, r = rh / p.H;
  const int n = p.n_rows[r], row0 = p.row_start[r], slot = p.slot[r];
  if (n <= 0 || slot < 0) return;
  const int tid = threadIdx.x, l = tid % LANES, cl = tid / LANES;
  const int col = cb * DW_COLS + cl;
  const bool live = col < p.dv;
  float* Sg = p.state + ((size_t)slot * p.H + h) * p.d * p.dv;
  const float a = p.powers[(size_t)h * p.n_powers + 1];
  const T* qg = (const T*)p.q + h * p.d;
  const T* kg = (const T*)p.k + h * p.d;
  const T* vg = (const T*)p.v + h * p.dv;
  float S[DW_R];
#pragma unroll
  for (int j = 0; j < DW_R; ++j) {
    const int row = ((j >> 2) * LANES + l) * 4 + (j & 3);
    S[j] = (live && row < p.d) ? Sg[(size_t)row * p.dv + col] : 0.f;
  }
  for (int c0 = 0; c0 < n; c0 += DW_CHUNK) {
    const int rows = min(DW_CHUNK, n - c0);
    __syncthreads();
    for (int i = tid; i < rows * DP; i += THREADS) {
      const int t = i / DP, e = i - t * DP;
      const size_t row = (size_t)(row0 + c0 + t);
      qs[t][e] = e < p.d ? dm_turned(p, qg + row * p.ldq, p.cos, p.sin, (int)row, e) : 0.f;
      ks[t][e] = e < p.d ? dm_turned(p, kg + row * p.ldk, p.cos, p.sin, (int)row, e) * p.kscale : 0.f;
    }
    for (int i = tid; i < rows * DW_COLS; i += THREADS) {
      const int t = i / DW_COLS, c = cb * DW_COLS + (i - t * DW_COLS);
      vs[t][i - t * DW_COLS] = c < p.dv ? dm_act(kf_load(vg, (size_t)(row0 + c0 + t) * p.ldv + c), p.act) : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < rows; ++t) {
      const float vv = vs[t][cl];
      float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int g = 0; g < DW_R / 4; ++g) {
        const float4 kk = *reinterpret_cast<const float4*>(&ks[t][(g * LANES + l) * 4]);
        const float4 qq = *reinterpret_cast<const float4*>(&qs[t][(g * LANES + l) * 4]);
        const float kv[4] = {kk.x, kk.y, kk.z, kk.w}, qv[4] = {qq.x, qq.y, qq.z, qq.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          S[4 * g + e] = fmaf(a, S[4 * g + e], kv[e] * vv);
          acc[e] = fmaf(S[4 * g + e], qv[e], acc[e]);
        }
      }
      float o = (acc[0] + acc[1]) + (acc[2] + acc[3]);
#pragma unroll
      for (int m = LANES / 2; m > 0; m >>= 1) o += __shfl_xor_sync(0xffffffffu, o, m);
      if (l == 0 && live) p.out[(size_t)(row0 + c0 + t) * p.H * p.dv + h * p.dv + col] = o;
    }
  }
  if (!p.writes) return;
#pragma unroll
  for (int j = 0; j < DW_R; ++j) {
    const int row = ((j >> 2) * LANES + l) * 4 + (j & 3);
    if (live && row < p.d) Sg[(size_t)row * p.dv + col] = S[j];
  }
}

// ---- 64 rows at a time on the tensor cores -----------------------------------------------------------------------------

constexpr int DC_ROWS = 64;
enum { DC_WHOLE = 0, DC_STATES = 1, DC_FROM_STATES = 2 };

// The chunk a block walks: chunks of `chunk_rows` rows are numbered request by request (requests without rows have none).
__device__ __forceinline__ bool dc_find(const DecayArgs& p, int chunk_rows, int number, int* req, int* chunk, int* n_chunks) {
  for (int r = 0; r < p.n_reqs; ++r) {
    const int n = p.n_rows[r];
    const int c = n > 0 ? (n + chunk_rows - 1) / chunk_rows : 0;
    if (number < c) { *req = r; *chunk = number; *n_chunks = c; return true; }
    number -= c;
  }
  return false;
}

__device__ __forceinline__ void dc_split(float x, float y, uint32_t* hi, uint32_t* lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  *hi = *reinterpret_cast<const uint32_t*>(&h);
  *lo = kf_mma::pack_bf16(x - f.x, y - f.y);
}

// D: the key size rounded up to a size with an instance (tails zero); VT: value columns per block; WARPS: 4 or 8 (eight keep
// the parts of a 256-row state in registers; below that four are the faster ones, having less to recompute).
// mode DC_WHOLE: from and into the request's state.  DC_STATES: every chunk but a request's last, from zero, no results, into
// chunk_state[number].  DC_FROM_STATES: from chunk_state[number]; a request's last chunk into its state.
template <int D, int VT, int WARPS>
__global__ void __launch_bounds__(WARPS * 32)
decay_chunk_kernel(DecayArgs p, int mode, int chunk_rows, float* __restrict__ chunk_state) {
  using namespace kf_mma;
  kf_pdl_trigger();
  constexpr int KS = D / 16;                           // k-steps along the key size
  constexpr int NT = VT / 8;                           // 8-column tiles of the values
  // The state: RG groups of rows x CG groups of columns, one per warp.  The results: four tiles of 16 rows x OG groups of
  // columns (the warps of a row tile all compute its scores).
  constexpr int RG = (WARPS == 8 && D >= 128) ? 8 : 4, CG = WARPS / RG, OG = WARPS / 4;
  constexpr int MT = D / RG / 16;                      // 16-row tiles of the state per warp
  constexpr int NTS = NT / CG;                         // ... and its 8-column tiles
  constexpr int NTO = NT / OG;                         // 8-column tiles of the results per warp
  constexpr int QK_TILE = DC_ROWS * D, V_TILE = DC_ROWS * VT;
  extern __shared__ __align__(128) uint8_t dc_smem[];
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(dc_smem);         // [2][64][D]
  __nv_bfloat16* sK = sQ + 2 * QK_TILE;                                   // [2][64][D]
  __nv_bfloat16* sV = sK + 2 * QK_TILE;                                   // [2][64][VT]
  __nv_bfloat16* sH = sV + 2 * V_TILE;                                    // [D][VT] the state's upper halves
  __nv_bfloat16* sL = sH + D * VT;                                        // [D][VT] ... and what they leave
  float* pw = reinterpret_cast<float*>(sL + D * VT);                      // a^0 .. a^64

  const int tiles = (p.dv + VT - 1) / VT;
  const int tile = blockIdx.x % tiles, rh = blockIdx.x / tiles;
  const int h = rh % p.H, number = rh / p.H;
  int req, chunk, n_chunks;
  if (!dc_find(p, chunk_rows, number, &req, &chunk, &n_chunks)) return;
  const int slot = p.slot[req];
  if (slot < 0) return;
  const bool last_chunk = chunk == n_chunks - 1;
  if (mode == DC_STATES && last_chunk) return;         // nobody starts from what a request's last chunk adds
  const int first = p.row_start[req] + chunk * chunk_rows;
  const int n = min(chunk_rows, p.n_rows[req] - chunk * chunk_rows);
  const int col0 = tile * VT;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
  const int wr = warp & 3, oc = (warp >> 2) * NTO;     // this warp's tile of rows, its first column tile of the results
  const int sr = (warp % RG) * (D / RG), sc = (warp / RG) * NTS;   // its first row and first column tile of the state
  for (int i = tid; i <= DC_ROWS; i += WARPS * 32) pw[i] = p.powers[(size_t)h * p.n_powers + i];
  kf_pdl_wait();

  const __nv_bfloat16* qg = kf_produced((const __nv_bfloat16*)p.q) + h * p.d;
  const __nv_bfloat16* kg = kf_produced((const __nv_bfloat16*)p.k) + h * p.d;
  const __nv_bfloat16* vg = kf_produced((const __nv_bfloat16*)p.v) + h * p.dv + col0;
  const bool with_out = mode != DC_STATES;
  auto load = [&](int c0, int st) {
    constexpr int CH = D / 8, CV = VT / 8;
    const int rows = n - c0;
    for (int i = tid; i < DC_ROWS * CH; i += WARPS * 32) {
      const int t = i / CH, c = i - t * CH;
      const bool ok = t < rows && c * 8 < p.d;
      const size_t row = (size_t)(first + c0 + (ok ? t : 0));
      const int cc = ok ? c * 8 : 0;
      cp_async16(tile_ptr<D>(sK + st * QK_TILE, t, c), kg + row * p.ldk + cc, ok);
      if (with_out) cp_async16(tile_ptr<D>(sQ + st * QK_TILE, t, c), qg + row * p.ldq + cc, ok);
    }
    for (int i = tid; i < DC_ROWS * CV; i += WARPS * 32) {
      const int t = i / CV, c = i - t * CV;
      const bool ok = t < rows && col0 + c * 8 < p.dv;
      const size_t row = (size_t)(first + c0 + (ok ? t : 0));
      cp_async16(tile_ptr<VT>(sV + st * V_TILE, t, c), vg + row * p.ldv + (ok ? c * 8 : 0), ok);
    }
  };
  load(0, 0);
  cp_async_commit();

  // this warp's part of the state: rows sr + mt * 16 + {g, g + 8}, columns (sc + nt) * 8 + tq * 2 + {0, 1}
  float S[MT][NTS][4];
  float* own = p.state + ((size_t)slot * p.H + h) * p.d * p.dv;
  float* kept = chunk_state + ((size_t)number * p.H + h) * p.d * p.dv;
  const float* from = mode == DC_WHOLE ? own : kept;
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < NTS; ++nt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int row = sr + mt * 16 + g + 8 * e, col = col0 + (sc + nt) * 8 + tq * 2;
        float2 v = make_float2(0.f, 0.f);
        if (mode != DC_STATES && row < p.d && col < p.dv) v = *reinterpret_cast<const float2*>(from + (size_t)row * p.dv + col);
        S[mt][nt][2 * e] = v.x, S[mt][nt][2 * e + 1] = v.y;
      }

  int st = 0;
  for (int c0 = 0; c0 < n; c0 += DC_ROWS, st ^= 1) {
    const int rows = min(DC_ROWS, n - c0);
    if (c0 + DC_ROWS < n) load(c0 + DC_ROWS, st ^ 1);
    cp_async_commit();
    if (with_out) {                                    // the state before these rows, as two bfloat16 numbers per element
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nt = 0; nt < NTS; ++nt)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            uint32_t hi, lo;
            dc_split(S[mt][nt][2 * e], S[mt][nt][2 * e + 1], &hi, &lo);
            const int row = sr + mt * 16 + g + 8 * e;
            reinterpret_cast<uint32_t*>(tile_ptr<VT>(sH, row, sc + nt))[tq] = hi;
            reinterpret_cast<uint32_t*>(tile_ptr<VT>(sL, row, sc + nt))[tq] = lo;
          }
    }
    cp_async_wait<1>();
    __syncthreads();
    __nv_bfloat16* k_s = sK + st * QK_TILE;
    __nv_bfloat16* v_s = sV + st * V_TILE;
    if (with_out && wr * 16 < rows) {
      __nv_bfloat16* q_s = sQ + st * QK_TILE;
      float O[NTO][4], P[DC_ROWS / 8][4];
#pragma unroll
      for (int nt = 0; nt < NTO; ++nt) O[nt][0] = O[nt][1] = O[nt][2] = O[nt][3] = 0.f;
#pragma unroll
      for (int nt = 0; nt < DC_ROWS / 8; ++nt) P[nt][0] = P[nt][1] = P[nt][2] = P[nt][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        uint32_t a[4];
        ldmatrix_x4(a, tile_ptr<D>(q_s, wr * 16 + (lane & 15), ks * 2 + (lane >> 4)));
#pragma unroll
        for (int np = 0; np < NTO / 2; ++np) {
          uint32_t b[4];
          ldmatrix_x4_trans(b, tile_ptr<VT>(sH, ks * 16 + (lane & 7) + (((lane >> 3) & 1) << 3), oc + np * 2 + (lane >> 4)));
          mma_bf16(O[2 * np], a, b[0], b[1]);
          mma_bf16(O[2 * np + 1], a, b[2], b[3]);
          ldmatrix_x4_trans(b, tile_ptr<VT>(sL, ks * 16 + (lane & 7) + (((lane >> 3) & 1) << 3), oc + np * 2 + (lane >> 4)));
          mma_bf16(O[2 * np], a, b[0], b[1]);
          mma_bf16(O[2 * np + 1], a, b[2], b[3]);
        }
#pragma unroll
        for (int np = 0; np < DC_ROWS / 16; ++np) {
          if (np > wr) continue;                     // keys after every row of this warp
          uint32_t b[4];
          ldmatrix_x4(b, tile_ptr<D>(k_s, np * 16 + (lane & 7) + ((lane >> 4) << 3), ks * 2 + ((lane >> 3) & 1)));
          mma_bf16(P[2 * np], a, b[0], b[1]);
          mma_bf16(P[2 * np + 1], a, b[2], b[3]);
        }
      }
      const int i0 = wr * 16 + g;
      const float d0 = pw[i0 + 1], d1 = pw[i0 + 9];
#pragma unroll
      for (int nt = 0; nt < NTO; ++nt) { O[nt][0] *= d0; O[nt][1] *= d0; O[nt][2] *= d1; O[nt][3] *= d1; }
#pragma unroll
      for (int nt = 0; nt < DC_ROWS / 8; ++nt) {
        if (nt > 2 * wr + 1) continue;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int gap = i0 + 8 * (e >> 1) - (nt * 8 + tq * 2 + (e & 1));
          P[nt][e] = gap >= 0 ? P[nt][e] * pw[gap] : 0.f;
        }
      }
#pragma unroll
      for (int ks = 0; ks < DC_ROWS / 16; ++ks) {
        if (ks > wr) continue;
        uint32_t hi[4], lo[4];
        dc_split(P[2 * ks][0], P[2 * ks][1], &hi[0], &lo[0]);
        dc_split(P[2 * ks][2], P[2 * ks][3], &hi[1], &lo[1]);
        dc_split(P[2 * ks + 1][0], P[2 * ks + 1][1], &hi[2], &lo[2]);
        dc_split(P[2 * ks + 1][2], P[2 * ks + 1][3], &hi[3], &lo[3]);
#pragma unroll
        for (int np = 0; np < NTO / 2; ++np) {
          uint32_t b[4];
          ldmatrix_x4_trans(b, tile_ptr<VT>(v_s, ks * 16 + (lane & 7) + (((lane >> 3) & 1) << 3), oc + np * 2 + (lane >> 4)));
          mma_bf16(O[2 * np], hi, b[0], b[1]);
          mma_bf16(O[2 * np + 1], hi, b[2], b[3]);
          mma_bf16(O[2 * np], lo, b[0], b[1]);
          mma_bf16(O[2 * np + 1], lo, b[2], b[3]);
        }
      }
#pragma unroll
      for (int nt = 0; nt < NTO; ++nt)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int i = i0 + 8 * e, col = col0 + (oc + nt) * 8 + tq * 2;
          if (i < rows && col < p.dv)
            *reinterpret_cast<float2*>(p.out + (size_t)(first + c0 + i) * p.H * p.dv + h * p.dv + col) =
                make_float2(O[nt][2 * e], O[nt][2 * e + 1]);
        }
    }
    // ---- the state after these rows ---------------------------------------------------------------------------------
    const float dn = pw[rows];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int nt = 0; nt < NTS; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[mt][nt][e] *= dn;
#pragma unroll
    for (int ks = 0; ks < DC_ROWS / 16; ++ks) {
      if (ks * 16 >= rows) continue;
      float f[4];                                      // the decays of this thread's four rows of the k-step
#pragma unroll
      for (int e = 0; e < 4; ++e) f[e] = pw[max(rows - 1 - (ks * 16 + tq * 2 + (e & 1) + 8 * (e >> 1)), 0)];
      uint32_t hi[MT][4], lo[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        uint32_t a[4];
        ldmatrix_x4_trans(a, tile_ptr<D>(k_s, ks * 16 + (lane & 7) + ((lane >> 4) << 3), sr / 8 + mt * 2 + ((lane >> 3) & 1)));
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 kk = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a[e]));
          dc_split(kk.x * f[2 * (e >> 1)], kk.y * f[2 * (e >> 1) + 1], &hi[mt][e], &lo[mt][e]);
        }
      }
#pragma unroll
      for (int np = 0; np < NTS / 2; ++np) {
        uint32_t b[4];
        ldmatrix_x4_trans(b, tile_ptr<VT>(v_s, ks * 16 + (lane & 7) + (((lane >> 3) & 1) << 3), sc + np * 2 + (lane >> 4)));
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          mma_bf16(S[mt][2 * np], hi[mt], b[0], b[1]);
          mma_bf16(S[mt][2 * np + 1], hi[mt], b[2], b[3]);
          mma_bf16(S[mt][2 * np], lo[mt], b[0], b[1]);
          mma_bf16(S[mt][2 * np + 1], lo[mt], b[2], b[3]);
        }
      }
    }
    __syncthreads();                                   // the other stage and the state's halves may be overwritten next turn
  }
  cp_async_wait<0>();
  float* to = mode == DC_STATES ? kept : own;
  if (mode != DC_STATES && !(last_chunk && p.writes)) return;
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < NTS; ++nt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int row = sr + mt * 16 + g + 8 * e, col = col0 + (sc + nt) * 8 + tq * 2;
        if (row < p.d && col < p.dv)
          *reinterpret_cast<float2*>(to + (size_t)row * p.dv + col) = make_float2(S[mt][nt][2 * e], S[mt][nt][2 * e + 1]);
      }
}

// chunk_state[number] <- the state before that chunk, for every chunk of every request: a running sum over the chunks, one
// thread per four elements of the state.
__global__ void __launch_bounds__(256)
decay_chunk_starts_kernel(DecayArgs p, int chunk_rows, float* __restrict__ chunk_state) {
  kf_pdl_trigger();
  kf_pdl_wait();
  const int per_head = p.d * p.dv / 4;                 // dv is a multiple of four
  const int r = blockIdx.y, h = blockIdx.z;
  const int e = blockIdx.x * blockDim.x + threadIdx.x;
  const int n = p.n_rows[r], slot = p.slot[r];
  if (n <= 0 || slot < 0 || e >= per_head) return;
  int number = 0;
  for (int q = 0; q < r; ++q) number += p.n_rows[q] > 0 ? (p.n_rows[q] + chunk_rows - 1) / chunk_rows : 0;
  const int n_chunks = (n + chunk_rows - 1) / chunk_rows;
  const float a = p.powers[(size_t)h * p.n_powers + chunk_rows];          // every chunk but the last is full
  float4 s = reinterpret_cast<const float4*>(p.state + ((size_t)slot * p.H + h) * p.d * p.dv)[e];
  for (int c0 = 0; c0 < n_chunks; c0 += 8) {
    float4 add[8];
#pragma unroll
    for (int u = 0; u < 8; ++u)
      if (c0 + u < n_chunks - 1)
        add[u] = reinterpret_cast<const float4*>(chunk_state + ((size_t)(number + c0 + u) * p.H + h) * p.d * p.dv)[e];
#pragma unroll
    for (int u = 0; u < 8; ++u) {
      if (c0 + u >= n_chunks) break;
      reinterpret_cast<float4*>(chunk_state + ((size_t)(number + c0 + u) * p.H + h) * p.d * p.dv)[e] = s;
      if (c0 + u < n_chunks - 1) {
        s.x = fmaf(a, s.x, add[u].x); s.y = fmaf(a, s.y, add[u].y);
        s.z = fmaf(a, s.z, add[u].z); s.w = fmaf(a, s.w, add[u].w);
      }
    }
  }
}

// From 32-bit projection rows to the bfloat16 rows [q | k | v] the tensor-core kernel reads: q and k turned, k scaled.
// One thread per four neighbouring elements (V = 4: rot and d multiples of eight, dv and the columns of four), or per element.
template <int V>
__global__ void __launch_bounds__(256)
decay_rotate_kernel(const float* __restrict__ in, int ld, int q0, int k0, int v0, const float* __restrict__ cos,
                    const float* __restrict__ sin, int rot, float kscale, int H, int d, int dv, __nv_bfloat16* __restrict__ out,
                    int T) {
  kf_pdl_trigger();
  kf_pdl_wait();
  const int nq = H * d, width = 2 * nq + H * dv, per = width / V, half = rot >> 1;
  const long item = (long)blockIdx.x * blockDim.x + threadIdx.x;
  if (item >= (long)T * per) return;
  const int t = (int)(item / per), c = (int)(item - (long)t * per) * V;
  const float* row = in + (size_t)t * ld;
  float x[V];
  auto read = [&](const float* p, float* o) {
    if constexpr (V == 4) { const float4 f = *reinterpret_cast<const float4*>(p); o[0] = f.x, o[1] = f.y, o[2] = f.z, o[3] = f.w; }
    else o[0] = *p;
  };
  if (c >= 2 * nq) {
    read(row + v0 + c - 2 * nq, x);
  } else {
    const bool key = c >= nq;
    const int cc = key ? c - nq : c, i = cc % d;
    const float* src = row + (key ? k0 : q0) + cc;
    read(src, x);
    if (i < rot) {
      const bool low = i < half;
      const int e = low ? i : i - half;
      float y[V], cs[V], sn[V];
      read(src + (low ? half : -half), y);
      read(cos + (size_t)t * half + e, cs);
      read(sin + (size_t)t * half + e, sn);
#pragma unroll
      for (int u = 0; u < V; ++u) x[u] = fmaf(x[u], cs[u], low ? -y[u] * sn[u] : y[u] * sn[u]);
    }
    if (key) {
#pragma unroll
      for (int u = 0; u < V; ++u) x[u] *= kscale;
    }
  }
  __nv_bfloat16* o = out + (size_t)t * width + c;
  if constexpr (V == 4) *reinterpret_cast<uint2*>(o) = make_uint2(kf_mma::pack_bf16(x[0], x[1]), kf_mma::pack_bf16(x[2], x[3]));
  else *o = __float2bfloat16_rn(x[0]);
}

template <int D, int VT, int WARPS>
int launch_chunks(const DecayArgs& p, int mode, int chunk_rows, int n_numbers, float* chunk_state, cudaStream_t stream) {
  const size_t smem = (size_t)(4 * DC_ROWS * D + 2 * DC_ROWS * VT + 2 * D * VT) * 2 + (DC_ROWS + 1) * sizeof(float);
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(decay_chunk_kernel<D, VT, WARPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
      kf_record_cuda_error(cudaGetLastError());
      return KF_ERR_SETUP;
    }
    configured = true;
  }
  const dim3 grid((unsigned)((long)n_numbers * p.H * kf_ceil_div(p.dv, VT)));
  kf_launch(decay_chunk_kernel<D, VT, WARPS>, grid, dim3(WARPS * 32), smem, stream, p, mode, chunk_rows, chunk_state);
  KF_CHECK_LAUNCH();
  return KF_OK;
}

int chunk_pass(const DecayArgs& p, int mode, int chunk_rows, int n_numbers, float* chunk_state, cudaStream_t stream) {
  if (p.d <= 64) return launch_chunks<64, 64, 4>(p, mode, chunk_rows, n_numbers, chunk_state, stream);
  if (p.d <= 128) return launch_chunks<128, 64, 4>(p, mode, chunk_rows, n_numbers, chunk_state, stream);
  return launch_chunks<256, 32, 8>(p, mode, chunk_rows, n_numbers, chunk_state, stream);
}

}  // namespace

// Whether the tensor-core kernel takes these sizes: key and value sizes that are multiples of eight elements, rows and column
// ranges that start on 16-byte boundaries.
KF_API int kf_decay_chunk_supported(int d, int dv, int ld) {
  return d >= 8 && d <= 256 && d % 8 == 0 && dv >= 8 && dv % 8 == 0 && ld % 8 == 0;
}
// Blocks per (request, head) of that kernel.
KF_API int kf_decay_chunk_tiles(int d, int dv) { return kf_ceil_div(dv, d <= 128 ? 64 : 32); }

// in [T, ld] 32-bit with q, k, v in columns q0, k0, v0; out [T, 2 H d + H dv] bfloat16.
KF_API int kf_decay_rotate(const float* in, int ld, int q0, int k0, int v0, const float* cos, const float* sin, int rot, float kscale,
                           int H, int d, int dv, void* out, int T, cudaStream_t stream) {
  if (T <= 0) return KF_OK;
  if (H < 1 || d < 1 || dv < 1 || rot < 0 || rot > d || (rot & 1) || (rot && (!cos || !sin))) return KF_ERR_SIZE;
  const bool by4 = rot % 8 == 0 && d % 8 == 0 && dv % 4 == 0 && ((ld | q0 | k0 | v0) & 3) == 0 &&
                   (((uintptr_t)in | (uintptr_t)out | (uintptr_t)cos | (uintptr_t)sin) & 15) == 0;
  const long n = (long)T * (2 * H * d + H * dv) / (by4 ? 4 : 1);
  const dim3 grid((unsigned)((n + 255) / 256));
  if (by4) kf_launch(decay_rotate_kernel<4>, grid, dim3(256), 0, stream, in, ld, q0, k0, v0, cos, sin, rot, kscale, H, d, dv, (__nv_bfloat16*)out, T);
  else kf_launch(decay_rotate_kernel<1>, grid, dim3(256), 0, stream, in, ld, q0, k0, v0, cos, sin, rot, kscale, H, d, dv, (__nv_bfloat16*)out, T);
  KF_CHECK_LAUNCH();
  return KF_OK;
}

// rows: the base of the matrix that holds q, k and v in columns q0, k0, v0 (`ld` columns); dtype: its element type.
// chunk_rows > 0 (a multiple of 64, below n_powers): chunks side by side; chunk_state then holds n_numbers * H * d * dv
// floats, n_numbers at least the number of chunks of the step.  single: no request has more than one row.
KF_API int kf_decay_memory(const void* rows, int dtype, int ld, int q0, int k0, int v0, int act, const float* powers,
                           int n_powers, float* state, float* out, int H, int d, int dv, int n_reqs, const int* row_start,
                           const int* n_rows, const int* slot, int writes, int single, int chunk_rows, int n_numbers,
                           float* chunk_state, const float* cos, const float* sin, int rot, float kscale, cudaStream_t stream) {
  if (n_reqs <= 0) return KF_OK;
  if (rot < 0 || rot > d || (rot & 1) || (rot && (!cos || !sin))) return KF_ERR_SIZE;
  if (d < 1 || d > 256 || dv < 1 || H < 1 || n_powers < DC_ROWS + 1) return KF_ERR_SIZE;
  if (dtype != KF_F32 && dtype != KF_BF16) return KF_ERR_DTYPE;
  const size_t es = dtype == KF_F32 ? 4 : 2;
  const char* base = (const char*)rows;
  DecayArgs p{base + q0 * es, base + k0 * es, base + v0 * es, ld, ld, ld, act, powers, n_powers, state, out, H, d, dv, n_reqs,
              row_start, n_rows, slot, writes, cos, sin, rot, kscale};
  if (single && dv % 4 == 0 && (((uintptr_t)state | (uintptr_t)out) & 15) == 0) {
    const dim3 grid((unsigned)((long)n_reqs * H * kf_ceil_div(dv, DD_COLS)));
#define KF_GO(NR)                                                                                               \
    do {                                                                                                        \
      if (dtype == KF_F32) kf_launch(decay_decode_kernel<float, NR>, grid, dim3(DD_THREADS), 0, stream, p);     \
      else kf_launch(decay_decode_kernel<__nv_bfloat16, NR>, grid, dim3(DD_THREADS), 0, stream, p);             \
    } while (0)
    if (d <= 32) KF_GO(1); else if (d <= 64) KF_GO(2); else if (d <= 128) KF_GO(4); else KF_GO(8);
#undef KF_GO
    KF_CHECK_LAUNCH();
    return KF_OK;
  }
  if (dtype == KF_BF16 && act == 0 && rot == 0 && kscale == 1.f && kf_decay_chunk_supported(d, dv, ld) && ((q0 | k0 | v0) & 7) == 0 &&
      (((uintptr_t)rows | (uintptr_t)state | (uintptr_t)chunk_state) & 15) == 0) {
    if (chunk_rows <= 0) return chunk_pass(p, DC_WHOLE, 1 << 30, n_reqs, state, stream);
    if (chunk_rows % DC_ROWS || chunk_rows >= n_powers || !chunk_state || n_numbers < 1) return KF_ERR_SIZE;
    int rc = chunk_pass(p, DC_STATES, chunk_rows, n_numbers, chunk_state, stream);
    if (rc != KF_OK) return rc;
    kf_launch(decay_chunk_starts_kernel, dim3(kf_ceil_div((long)d * dv / 4, 256), n_reqs, H), dim3(256), 0, stream, p, chunk_rows,
              chunk_state);
    KF_CHECK_LAUNCH();
    return chunk_pass(p, DC_FROM_STATES, chunk_rows, n_numbers, chunk_state, stream);
  }
  const dim3 grid((unsigned)((long)n_reqs * H * kf_ceil_div(dv, DW_COLS)));
#define KF_GO(LL)                                                                                                          \
  do {                                                                                                                     \
    if (dtype == KF_F32) kf_launch(decay_walk_kernel<float, LL>, grid, dim3(LL * DW_COLS), 0, stream, p);                  \
    else kf_launch(decay_walk_kernel<__nv_bfloat16, LL>, grid, dim3(LL * DW_COLS), 0, stream, p);                          \
  } while (0)
  if (d <= 32) KF_GO(4); else if (d <= 64) KF_GO(8); else if (d <= 128) KF_GO(16); else KF_GO(32);
#undef KF_GO
  KF_CHECK_LAUNCH();
  return KF_OK;
}
