// Time mixing over a matrix state per head whose rows decay by a number of their own per token, with a bonus
// for the current token:
//
//   o_t = (S + diag(u) k_t v_t^T)^T r_t,   S <- diag(w_t) S + k_t v_t^T            (S: [D, E], float32)
//
// token_shift: every projection of the mixer reads its own blend of a row and the row before it,
//   h + (h' - h) mu_s; all blends of a row in one launch.  The row before a request's first row of the step
//   comes from its state row ([W] float32, zeros for a request's first token), which the launch moves on:
//   the thread that reads it there also writes the request's last row of the step, so nothing races.
// low_rank_decay: w = exp(-exp(w0 + W2 tanh(x))) per channel, x the narrow projection's float32 rows; float32
//   multiply-adds, a block a tile of tokens and channels.
// wkv_steps: the recurrence token by token (steps of single tokens, key heads over 256 wide).  A block takes
//   (request, head, slice of value columns); PARTS neighbouring lanes share a column of S and hold RPT of its
//   rows each.  r, k and v are read as the projections left them.
// wkv_chunks and the scan of chunk_scan.cuh: prompt portions, sixteen tokens at a time.  With P(i, j) the
//   product of the decays after token i and before token j, token j reads r_j . P(i, j) k_i of token i's v
//   (i < j) and r_j . u k_j of its own.  All decay products are products of numbers in (0, 1], no ratio is
//   formed, so nothing can overflow.
// The state is laid out [head][column][key channel]: the lanes of a column move consecutive 16-byte pieces.
#include "chunk_scan.cuh"
#include "common.cuh"
#include "pdl.cuh"

using namespace pbe;

namespace {
constexpr int MAX_BLENDS = 8;
constexpr int MAX_HEAD = 512;

// ------------------------------------------------------------------ token_shift
struct ShiftParams {
  const void* h;             // [T, W]
  const float* mu;           // [S, W]
  float* state;              // [slots, W]
  void* out;                 // [S, T, W]
  const int32_t* request_of_row;
  const int32_t* q_start;
  const int32_t* q_len;
  const int32_t* slots;
  int T, R, W, S, update;
};

template <typename T, int V>
__global__ void token_shift_kernel(ShiftParams p) {
  pdl_launch_dependents();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  pdl_wait();
  if (c >= p.W) return;
  const int t = blockIdx.x;
  const int r = p.request_of_row[t];
  const bool live = r >= 0 && r < p.R && p.q_len[r] > 0;       // not a padding row of a captured step
  const T* h = (const T*)p.h;
  float now[V], before[V];
#pragma unroll
  for (int k = 0; k < V; ++k) now[k] = before[k] = 0.f;
  if (live) {
    load_v<V>(h + (size_t)t * p.W + c, now);
    if (t > p.q_start[r]) {
      load_v<V>(h + (size_t)(t - 1) * p.W + c, before);
    } else {
      float* st = p.state + (size_t)p.slots[r] * p.W + c;
      load_v<V>(st, before);
      if (p.update) {
        float last[V];
        load_v<V>(h + (size_t)(t + p.q_len[r] - 1) * p.W + c, last);
        put_v<V>(st, last);
      }
    }
  }
#pragma unroll 1
  for (int s = 0; s < p.S; ++s) {
    float mu[V], y[V];
    load_v<V>(p.mu + (size_t)s * p.W + c, mu);
#pragma unroll
    for (int k = 0; k < V; ++k) y[k] = fmaf(before[k] - now[k], mu[k], now[k]);
    put_v<V>((T*)p.out + ((size_t)s * p.T + t) * p.W + c, y);
  }
}

// ------------------------------------------------------------------ low_rank_decay
constexpr int LR_TOKENS = 8, LR_THREADS = 128, LR_RANK = 32;

struct LowRankParams {
  const float* x;            // [T, ldx], the narrow projection before tanh
  int ldx;
  const void* w2t;           // [rank, C]
  const float* w0;           // [C]
  float* decay;              // [T, C]
  int T, C, rank;
};

// grid (tiles of LR_TOKENS tokens, tiles of LR_THREADS * V channels)
template <typename TW, int V>
__global__ void __launch_bounds__(LR_THREADS) low_rank_decay_kernel(LowRankParams p) {
  __shared__ __align__(16) float th[LR_RANK][LR_TOKENS];
  pdl_launch_dependents();
  const int c = (blockIdx.y * LR_THREADS + threadIdx.x) * V;
  const bool live = c < p.C;
  float acc[V][LR_TOKENS];
#pragma unroll
  for (int k = 0; k < V; ++k) {
    const float w0 = live ? p.w0[c + k] : 0.f;       // C is a multiple of V
#pragma unroll
    for (int i = 0; i < LR_TOKENS; ++i) acc[k][i] = w0;
  }
  pdl_wait();
  const int t0 = blockIdx.x * LR_TOKENS;
  for (int j0 = 0; j0 < p.rank; j0 += LR_RANK) {
    const int n = min(LR_RANK, p.rank - j0);
    __syncthreads();
    for (int i = threadIdx.x; i < LR_TOKENS * LR_RANK; i += LR_THREADS) {
      const int tt = i / LR_RANK, j = i - tt * LR_RANK;
      th[j][tt] = (j < n && t0 + tt < p.T) ? tanhf(p.x[(size_t)(t0 + tt) * p.ldx + j0 + j]) : 0.f;
    }
    __syncthreads();
    if (live) {
      const TW* w2 = (const TW*)p.w2t + (size_t)j0 * p.C + c;
#pragma unroll 8
      for (int j = 0; j < n; ++j) {
        float w[V];
        if constexpr (V == 2 && sizeof(TW) == 2) {
          const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(w2 + (size_t)j * p.C));
          w[0] = f.x; w[1] = f.y;
        } else {
#pragma unroll
          for (int k = 0; k < V; ++k) w[k] = to_float(w2[(size_t)j * p.C + k]);
        }
#pragma unroll
        for (int i = 0; i < LR_TOKENS; i += 4) {
          const float4 y = *reinterpret_cast<const float4*>(&th[j][i]);
#pragma unroll
          for (int k = 0; k < V; ++k) {
            acc[k][i] = fmaf(w[k], y.x, acc[k][i]);
            acc[k][i + 1] = fmaf(w[k], y.y, acc[k][i + 1]);
            acc[k][i + 2] = fmaf(w[k], y.z, acc[k][i + 2]);
            acc[k][i + 3] = fmaf(w[k], y.w, acc[k][i + 3]);
          }
        }
      }
    }
  }
  if (!live) return;
#pragma unroll
  for (int i = 0; i < LR_TOKENS; ++i) {
    if (t0 + i >= p.T) break;
    float* out = p.decay + (size_t)(t0 + i) * p.C + c;
    if constexpr (V == 2) {
      *reinterpret_cast<float2*>(out) = make_float2(expf(-expf(acc[0][i])), expf(-expf(acc[1][i])));
    } else {
#pragma unroll
      for (int k = 0; k < V; ++k) out[k] = expf(-expf(acc[k][i]));
    }
  }
}

// ------------------------------------------------------------------ the recurrence, token by token
struct WkvParams {
  const void* r;             // [T, H * D]
  const void* k;             // [T, H * D]
  const void* v;             // [T, H * E]
  int ld_r, ld_k, ld_v;      // row strides, elements
  const float* decay;        // [T, H * D]
  const float* bonus;        // [H * D]
  float* out;                // [T, H * E]
  float* state;              // [slots, H, E, D]
  const int32_t* q_start;
  const int32_t* q_len;
  const int32_t* slots;
  int R, H, D, E, write_state;
};

template <typename T, int RPT, int PARTS, int V>
__global__ void __launch_bounds__(128) wkv_steps_kernel(WkvParams p) {
  constexpr int COLS = 128 / PARTS;
  constexpr int PIECES = RPT / V;              // pieces of V neighbouring rows a lane holds
  pdl_launch_dependents();
  const int r = blockIdx.x, h = blockIdx.y;
  const int part = threadIdx.x % PARTS, col = threadIdx.x / PARTS;
  const int e = blockIdx.z * COLS + col;
  const int D = p.D, E = p.E, H = p.H;
  const bool live = e < E;
  float u[PIECES][V];
#pragma unroll
  for (int j = 0; j < PIECES; ++j) {
    const int d = (j * PARTS + part) * V;
#pragma unroll
    for (int x = 0; x < V; ++x) u[j][x] = 0.f;
    if (d < D) load_v<V>(p.bonus + (size_t)h * D + d, u[j]);
  }
  pdl_wait();
  const int n = p.q_len[r];
  if (n <= 0) return;
  const int t0 = p.q_start[r];
  float* st = p.state + (((size_t)p.slots[r] * H + h) * E + (live ? e : 0)) * D;
  float S[PIECES][V];
#pragma unroll
  for (int j = 0; j < PIECES; ++j) {
    const int d = (j * PARTS + part) * V;
#pragma unroll
    for (int x = 0; x < V; ++x) S[j][x] = 0.f;
    if (live && d < D) load_v<V>(st + d, S[j]);
  }
#pragma unroll 1
  for (int t = t0; t < t0 + n; ++t) {
    const T* rp = (const T*)p.r + (size_t)t * p.ld_r + h * D;
    const T* kp = (const T*)p.k + (size_t)t * p.ld_k + h * D;
    const float* wp = p.decay + (size_t)t * H * D + h * D;
    const float v = live ? to_float(((const T*)p.v)[(size_t)t * p.ld_v + h * E + e]) : 0.f;
    float read = 0.f, own = 0.f;
#pragma unroll
    for (int j = 0; j < PIECES; ++j) {
      const int d = (j * PARTS + part) * V;
      float rv[V], kv[V], wv[V];
#pragma unroll
      for (int x = 0; x < V; ++x) rv[x] = kv[x] = wv[x] = 0.f;
      if (d < D) {
        load_v<V>(rp + d, rv);
        load_v<V>(kp + d, kv);
        load_v<V>(wp + d, wv);
      }
#pragma unroll
      for (int x = 0; x < V; ++x) {
        read = fmaf(S[j][x], rv[x], read);
        own = fmaf(u[j][x] * kv[x], rv[x], own);
        S[j][x] = fmaf(wv[x], S[j][x], kv[x] * v);
      }
    }
#pragma unroll
    for (int m = 1; m < PARTS; m <<= 1) {
      read += __shfl_xor_sync(0xffffffffu, read, m);
      own += __shfl_xor_sync(0xffffffffu, own, m);
    }
    if (live && part == 0) p.out[((size_t)t * H + h) * E + e] = fmaf(own, v, read);
  }
  if (live && p.write_state) {
#pragma unroll
    for (int j = 0; j < PIECES; ++j) {
      const int d = (j * PARTS + part) * V;
      if (d < D) put_v<V>(st + d, S[j]);
    }
  }
}

// ------------------------------------------------------------------ chunks of sixteen tokens
// grid (records, H), a block of 128 threads a chunk and head
template <typename T, int DP>
__global__ void __launch_bounds__(128) wkv_chunks_kernel(WkvParams p, float* records) {
  extern __shared__ __align__(16) float smem[];
  float* K = smem;                        // [CH][DP]
  float* Q = K + CH * DP;                 // [CH][DP] the read vectors
  float* W = Q + CH * DP;                 // [CH][DP] decays
  pdl_launch_dependents();
  pdl_wait();
  const int rec = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int D = p.D, H = p.H;
  const int r = record_owner<128>(rec, p.q_start, p.q_len, p.R);
  if (r < 0) return;
  const int c = rec - first_record(p.q_start[r], r);
  const int count = min(CH, p.q_len[r] - c * CH);
  const size_t row0 = (size_t)p.q_start[r] + c * CH;
  const T* rp = (const T*)p.r + h * D;
  const T* kp = (const T*)p.k + h * D;
  const float* wp = p.decay + (size_t)h * D;
  const bool quads = (D & 3) == 0 && ((p.ld_r | p.ld_k) & 3) == 0 &&
                     (((uintptr_t)p.r | (uintptr_t)p.k) & (4 * sizeof(T) - 1)) == 0;
  if (quads) {
#pragma unroll
    for (int n = 0; n < CH * DP / 512; ++n) {
      const int i = (tid + n * 128) * 4;
      const int j = i / DP, d = i % DP;
      float rv[4] = {0.f, 0.f, 0.f, 0.f}, kv[4] = {0.f, 0.f, 0.f, 0.f}, wv[4] = {1.f, 1.f, 1.f, 1.f};
      if (j < count && d < D) {
        load_v<4>(rp + (row0 + j) * p.ld_r + d, rv);
        load_v<4>(kp + (row0 + j) * p.ld_k + d, kv);
        load_v<4>(wp + (row0 + j) * H * D + d, wv);
      }
      put_v<4>(Q + i, rv);
      put_v<4>(K + i, kv);
      put_v<4>(W + i, wv);
    }
  } else {
    for (int i = tid; i < CH * DP; i += 128) {
      const int j = i / DP, d = i % DP;
      const bool ok = j < count && d < D;
      Q[i] = ok ? to_float(rp[(row0 + j) * p.ld_r + d]) : 0.f;
      K[i] = ok ? to_float(kp[(row0 + j) * p.ld_k + d]) : 0.f;
      W[i] = ok ? wp[(row0 + j) * H * D + d] : 1.f;
    }
  }
  __syncthreads();
  float* out = records + ((size_t)rec * H + h) * record_floats(DP, false);
  float* mq = out + rec_mq(DP);
  {
    // eight lanes share a token i, DP / 8 channels each; x runs over k_i times the decays after i
    constexpr int MPT = DP / 8;
    const int i = tid >> 3, slice = tid & 7;
    float x[MPT];
#pragma unroll
    for (int m = 0; m < MPT; ++m) x[m] = K[i * DP + slice + 8 * m];
    for (int j = 0; j < CH; ++j) {
      float cq = 0.f;
      if (j == i) {
#pragma unroll
        for (int m = 0; m < MPT; ++m) {
          const int d = slice + 8 * m;
          if (d < D) cq = fmaf(p.bonus[(size_t)h * D + d] * x[m], Q[j * DP + d], cq);
        }
      } else if (j > i) {
#pragma unroll
        for (int m = 0; m < MPT; ++m) {
          const int d = j * DP + slice + 8 * m;
          cq = fmaf(x[m], Q[d], cq);
          x[m] *= W[d];
        }
      }
#pragma unroll
      for (int m = 1; m < 8; m <<= 1) cq += __shfl_xor_sync(0xffffffffu, cq, m);
      if (slice == 0) mq[i * CH + j] = cq;
    }
    float* kd = out + rec_kd(DP) + i * DP;
#pragma unroll
    for (int m = 0; m < MPT; ++m) kd[slice + 8 * m] = x[m];
  }
  for (int d = tid; d < DP; d += 128) {
    float up = 1.f;
#pragma unroll
    for (int j = 0; j < CH; ++j) {
      out[j * DP + d] = Q[j * DP + d] * up;
      up *= W[j * DP + d];
    }
    out[rec_decay(DP) + d] = up;
  }
}

// How long portions are cut into segments (all null: they are not)
struct Segments {
  const int32_t* first;      // [n_first, 4] the segments whose own contributions are needed
  int n_first;
  const int32_t* starts;     // [n_starts, 4]
  int n_starts;
  const int32_t* second;     // [n_second, 4] every segment, and the requests that are not cut
  int n_second;
  float* scratch;            // [entries, H, E, D]
  float* own_decay;          // [entries, H, D]
  const int32_t* request_of_row;
};

template <typename T, int RPT, int CPT, int WARPS>
int launch_chunks(const WkvParams& g, float* records, int count, const Segments& s, cudaStream_t stream) {
  constexpr int DP = 16 * RPT, COLS = 2 * WARPS * CPT;
  constexpr size_t smem_g = sizeof(float) * 3 * CH * DP, smem_p = sizeof(float) * 2 * record_floats(DP, false);
  static bool opted = false;
  if (!opted) {
    cudaFuncSetAttribute(wkv_chunks_kernel<T, DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_g);
    cudaFuncSetAttribute(scan_chunks_kernel<RPT, CPT, WARPS, false, true, T>,
                         cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_p);
    const cudaError_t e = cudaFuncSetAttribute(scan_chunks_kernel<RPT, CPT, WARPS, false, false, T>,
                                               cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_p);
    if (e != cudaSuccess) return (int)e;
    opted = true;
  }
  launch_k(wkv_chunks_kernel<T, DP>, dim3(count, g.H), 128, smem_g, stream, g, records);
  int err = launch_status();
  if (err != 0) return err;
  ChunkScanParams<T> p{records, (const T*)g.v, g.ld_v, g.out, g.state, g.q_start, g.q_len, g.slots,
                       g.H, g.D, g.E, g.write_state};
  const int slices = (g.E + COLS - 1) / COLS;
  if (s.second == nullptr) {
    launch_spread(scan_chunks_kernel<RPT, CPT, WARPS, false, false, T>, dim3(g.R, g.H, slices), 32 * WARPS, smem_p,
                  stream, p);
    return launch_status();
  }
  p.scratch = s.scratch;
  p.own_decay = s.own_decay;
  p.request_of_row = s.request_of_row;
  p.items = s.first;
  launch_spread(scan_chunks_kernel<RPT, CPT, WARPS, false, true, T>, dim3(s.n_first, g.H, slices), 32 * WARPS, smem_p,
                stream, p);
  err = launch_status();
  if (err != 0) return err;
  launch_k(segment_starts_kernel, dim3(s.n_starts, g.H, (unsigned)(((size_t)g.D * g.E + 255) / 256)), 256, 0, stream,
           (const float*)g.state, s.scratch, (const float*)s.own_decay, s.starts, g.H, g.D, g.E);
  err = launch_status();
  if (err != 0) return err;
  p.items = s.second;
  launch_spread(scan_chunks_kernel<RPT, CPT, WARPS, false, false, T>, dim3(s.n_second, g.H, slices), 32 * WARPS, smem_p,
                stream, p);
  return launch_status();
}

template <typename T, int V>
int launch_steps(const WkvParams& p, cudaStream_t stream) {
#define PBE_WKV(RPT, PARTS) \
  launch_k(wkv_steps_kernel<T, RPT, PARTS, V>, dim3(p.R, p.H, (p.E + 128 / PARTS - 1) / (128 / PARTS)), 128, 0, stream, p)
  if (p.D <= 32) PBE_WKV(4, 8);
  else if (p.D <= 64) PBE_WKV(8, 8);
  else if (p.D <= 128) PBE_WKV(16, 8);
  else if (p.D <= 256) PBE_WKV(16, 16);
  else PBE_WKV(16, 32);
#undef PBE_WKV
  return launch_status();
}
}  // namespace

PBE_EXPORT int pbe_token_shift(const void* h, int dtype, const float* mu, float* state, void* out,
                               const int32_t* request_of_row, const int32_t* q_start, const int32_t* q_len,
                               const int32_t* slots, int T, int R, int W, int S, int update, cudaStream_t stream) {
  if (T <= 0 || W <= 0) return 0;
  if (S < 1 || S > MAX_BLENDS) return (int)cudaErrorInvalidValue;
  ShiftParams p{h, mu, state, out, request_of_row, q_start, q_len, slots, T, R, W, S, update};
  const bool vec4 = W % 4 == 0 && (((uintptr_t)mu | (uintptr_t)state) & 15) == 0 &&
                    (((uintptr_t)h | (uintptr_t)out) & (dtype == PBE_F32 ? 15 : 7)) == 0;
  const int per = vec4 ? 4 : 1;
  const int lanes = (W + per - 1) / per;
  const int threads = lanes >= 256 ? 256 : (lanes + 31) / 32 * 32;
  dim3 grid(T, (lanes + threads - 1) / threads);
  if (dtype == PBE_F32) {
    if (vec4) launch_k(token_shift_kernel<float, 4>, grid, threads, 0, stream, p);
    else launch_k(token_shift_kernel<float, 1>, grid, threads, 0, stream, p);
  } else {
    if (vec4) launch_k(token_shift_kernel<__nv_bfloat16, 4>, grid, threads, 0, stream, p);
    else launch_k(token_shift_kernel<__nv_bfloat16, 1>, grid, threads, 0, stream, p);
  }
  return launch_status();
}

PBE_EXPORT int pbe_low_rank_decay(const float* x, int ldx, const void* w2t, int w_dtype, const float* w0, float* decay,
                                  int T, int C, int rank, cudaStream_t stream) {
  if (T <= 0 || C <= 0) return 0;
  if (rank < 1) return (int)cudaErrorInvalidValue;
  LowRankParams p{x, ldx, w2t, w0, decay, T, C, rank};
  const bool pair = C % 2 == 0 && ((uintptr_t)w2t & 3) == 0 && ((uintptr_t)decay & 7) == 0;
  const int per = LR_THREADS * (pair ? 2 : 1);
  dim3 grid((T + LR_TOKENS - 1) / LR_TOKENS, (C + per - 1) / per);
  if (w_dtype == PBE_F32) {
    if (pair) launch_k(low_rank_decay_kernel<float, 2>, grid, LR_THREADS, 0, stream, p);
    else launch_k(low_rank_decay_kernel<float, 1>, grid, LR_THREADS, 0, stream, p);
  } else {
    if (pair) launch_k(low_rank_decay_kernel<__nv_bfloat16, 2>, grid, LR_THREADS, 0, stream, p);
    else launch_k(low_rank_decay_kernel<__nv_bfloat16, 1>, grid, LR_THREADS, 0, stream, p);
  }
  return launch_status();
}

PBE_EXPORT int pbe_wkv_steps(const void* r, const void* k, const void* v, int ld_r, int ld_k, int ld_v, int dtype,
                             const float* decay, const float* bonus, float* out, float* state, const int32_t* q_start,
                             const int32_t* q_len, const int32_t* slots, int R, int H, int D, int E, int write_state,
                             cudaStream_t stream) {
  if (R <= 0) return 0;
  if (D < 1 || E < 1 || H < 1 || D > MAX_HEAD) return (int)cudaErrorInvalidValue;
  WkvParams p{r, k, v, ld_r, ld_k, ld_v, decay, bonus, out, state, q_start, q_len, slots, R, H, D, E, write_state};
  const bool vec4 = D % 4 == 0 && ((ld_r | ld_k) & 3) == 0 &&
                    (((uintptr_t)decay | (uintptr_t)bonus | (uintptr_t)state) & 15) == 0 &&
                    (((uintptr_t)r | (uintptr_t)k) & (dtype == PBE_F32 ? 15 : 7)) == 0;
  if (dtype == PBE_F32) return vec4 ? launch_steps<float, 4>(p, stream) : launch_steps<float, 1>(p, stream);
  return vec4 ? launch_steps<__nv_bfloat16, 4>(p, stream) : launch_steps<__nv_bfloat16, 1>(p, stream);
}

// Floats of a chunk's record (a head), for key heads of D channels (0: too wide for the chunked form).
PBE_EXPORT int pbe_wkv_record_floats(int D) {
  return D <= 64 ? record_floats(64, false) : D <= 128 ? record_floats(128, false) : D <= 256 ? record_floats(256, false) : 0;
}
PBE_EXPORT int pbe_wkv_chunk_tokens() { return CH; }

// The same for steps with prompt portions, sixteen tokens of a request at a time: two launches.
// records: [T / 16 + R][H][pbe_wkv_record_floats(D)] floats of scratch memory.  With `second` (segments of whole
// chunks, see chunk_scan.cuh) long portions run as segments side by side: two launches more.
PBE_EXPORT int pbe_wkv_chunks(const void* r, const void* k, const void* v, int ld_r, int ld_k, int ld_v, int dtype,
                              const float* decay, const float* bonus, float* out, float* state, float* records,
                              const int32_t* q_start, const int32_t* q_len, const int32_t* slots, int T, int R, int H,
                              int D, int E, int write_state, const int32_t* first, int n_first, const int32_t* starts,
                              int n_starts, const int32_t* second, int n_second, float* scratch, float* own_decay,
                              const int32_t* request_of_row, cudaStream_t stream) {
  if (R <= 0 || T <= 0) return 0;
  if (second != nullptr && (!first || !starts || !scratch || !own_decay || !request_of_row || n_first < 1 || n_starts < 1))
    return (int)cudaErrorInvalidValue;
  if (((uintptr_t)scratch & 15) != 0) return (int)cudaErrorMisalignedAddress;
  const Segments s{first, n_first, starts, n_starts, second, n_second, scratch, own_decay, request_of_row};
  if (D < 1 || D > 256 || E < 1 || H < 1 || records == nullptr) return (int)cudaErrorInvalidValue;
  if ((((uintptr_t)state | (uintptr_t)records | (uintptr_t)decay) & 15) != 0) return (int)cudaErrorMisalignedAddress;
  WkvParams p{r, k, v, ld_r, ld_k, ld_v, decay, bonus, out, state, q_start, q_len, slots, R, H, D, E, write_state};
  const int n = T / CH + R;
  if (dtype == PBE_F32) {
    if (D <= 64) return launch_chunks<float, 4, 4, 4>(p, records, n, s, stream);
    if (D <= 128) return launch_chunks<float, 8, 4, 4>(p, records, n, s, stream);
    return launch_chunks<float, 16, 2, 4>(p, records, n, s, stream);
  }
  if (D <= 64) return launch_chunks<__nv_bfloat16, 4, 4, 4>(p, records, n, s, stream);
  if (D <= 128) return launch_chunks<__nv_bfloat16, 8, 4, 4>(p, records, n, s, stream);
  return launch_chunks<__nv_bfloat16, 16, 2, 4>(p, records, n, s, stream);
}
