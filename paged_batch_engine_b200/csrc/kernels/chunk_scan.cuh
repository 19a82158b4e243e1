// A recurrence over a matrix state per head, sixteen tokens at a time: what the gated delta rule and the
// time mixing with a bonus share.
//
// Both make, in a launch of their own, a record per chunk of sixteen tokens and head: with S ([D, E],
// float32) the state at the chunk's start and a decay per row of S and token,
//   QG  the read vectors times the decays from the chunk's start,
//   KD  the written keys times the decays to the chunk's end,
//   decay  the product of all the chunk's decays,
//   MQ[i][j]  what token j reads of token i's write (i <= j),
//   W  (only where writes are corrected by what S predicts) the vectors that turn the given rows U into the
//      written ones, u = U - S^T W; elsewhere u = U.
// The scan over a request's chunks is then o_j = S^T qg_j + sum_{i<=j} MQ_ij u_i and
// S <- decay S + sum_j kd_j u_j^T: products of small matrices, float32 pairs (fma.rn.f32x2), one
// reduce-scatter for sixteen tokens.
//
// Writes without corrections are linear in the state, so long portions may be cut into segments (whole chunks)
// that run side by side, given as work items: a pass without read-outs (OWN) leaves each segment's own
// contribution and decay product, segment_starts_kernel turns these into the states at the segments' starts, and
// a second pass runs every segment from its start state.
#pragma once
#include "common.cuh"
#include "pdl.cuh"
#include "vec.cuh"

namespace pbe {


__device__ __forceinline__ void cp_async16(void* smem, const void* gmem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(s), "l"(gmem));
}
__device__ __forceinline__ void cp_async4(void* smem, const void* gmem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(s), "l"(gmem));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_group 0;\n" ::); }


constexpr int CH = 16;

// A record: QG and KD [CH][DP] each, the decay product [DP], MQ [CH][CH], and with corrections W [CH][DP].
__host__ __device__ constexpr int rec_kd(int dp) { return CH * dp; }
__host__ __device__ constexpr int rec_decay(int dp) { return 2 * CH * dp; }
__host__ __device__ constexpr int rec_mq(int dp) { return 2 * CH * dp + dp; }
__host__ __device__ constexpr int rec_w(int dp) { return 2 * CH * dp + dp + CH * CH; }
__host__ __device__ constexpr int record_floats(int dp, bool correct) { return rec_w(dp) + (correct ? CH * dp : 0); }
// The records of a request that starts at row q of the step: they begin at q / CH + r, which leaves every
// request room for all its chunks (the last of them may be short) without overlap.
__device__ __forceinline__ int first_record(int q_start, int r) { return q_start / CH + r; }

// Which request record `rec` belongs to (-1: none); called by all threads of a block of NT.
template <int NT>
__device__ __forceinline__ int record_owner(int rec, const int32_t* q_start, const int32_t* q_len, int R) {
  __shared__ int owner;
  if (threadIdx.x == 0) owner = -1;
  __syncthreads();
  for (int i = threadIdx.x; i < R; i += NT) {      // each thread looks at some of the requests, one finds it
    const int first = first_record(q_start[i], i);
    if (rec >= first && rec < first + (q_len[i] + CH - 1) / CH) owner = i;
  }
  __syncthreads();
  return owner;
}

typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ f32x2 pack2(float x, float y) {
  f32x2 d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(x), "f"(y));
  return d;
}
__device__ __forceinline__ void unpack2(f32x2 a, float& x, float& y) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(a));
}

template <typename TU>
struct ChunkScanParams {
  const float* records;
  const TU* u;               // [T, ld_u], column h * E + e
  int ld_u;
  float* out;                // [T, H * E]
  float* state;              // [slots, H, E, D]
  const int32_t* q_start;
  const int32_t* q_len;
  const int32_t* slots;
  int H, D, E, write_state;
  // work items instead of requests when not null: [n, 4] = first batch row, rows, where the state comes from,
  // where it goes; a place is a row of `state` (v >= 0), nothing / zeros (-1), or entry -(v + 2) of `scratch`
  const int32_t* items = nullptr;
  float* scratch = nullptr;            // [entries, H, E, D]
  float* own_decay = nullptr;          // [entries, H, D]: the segments' decay products, left by the OWN pass
  const int32_t* request_of_row = nullptr;
};

// x: a value per token (16) of each of the sixteen lanes of a half warp; lane p ends with the sum over the
// lanes of its token p
__device__ __forceinline__ float scatter_sum(float (&x)[CH], int part) {
#pragma unroll
  for (int half = CH / 2; half > 0; half >>= 1) {
    const bool upper = (part & half) != 0;
#pragma unroll
    for (int j = 0; j < half; ++j) {
      const float mine = upper ? x[j + half] : x[j];
      const float give = upper ? x[j] : x[j + half];
      x[j] = mine + __shfl_xor_sync(0xffffffffu, give, half);
    }
  }
  return x[0];
}

// A half warp shares CPT columns: lane p holds RPT key channels of each (DP = 16 RPT), and stands for the
// chunk's token p where the chunk's own numbers are concerned.
template <int RPT, int CPT, int WARPS, bool CORRECT, bool OWN, typename TU>
__global__ void __launch_bounds__(32 * WARPS, CPT > 2 ? 3 : 1) scan_chunks_kernel(ChunkScanParams<TU> p) {
  constexpr int NT = 32 * WARPS;
  constexpr int DP = 16 * RPT;
  constexpr int QUADS = RPT / 4;
  constexpr int COLS = 2 * WARPS * CPT;
  constexpr int REC = record_floats(DP, CORRECT);
  constexpr int TG = CPT > 2 ? 8 : 16;                   // tokens whose products are summed at a time (registers)
  extern __shared__ __align__(16) float smem[];          // two records
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.y;
  const int tid = threadIdx.x;
  int r = blockIdx.x, t0, n, src, dst;
  if (p.items) {
    const int32_t* it = p.items + (size_t)blockIdx.x * 4;
    t0 = it[0]; n = it[1]; src = it[2]; dst = it[3];
    r = p.request_of_row[t0];
  } else {
    n = p.q_len[r];
    t0 = p.q_start[r];
    src = dst = n > 0 ? p.slots[r] : -1;
  }
  if (n <= 0) return;
  const int D = p.D, E = p.E, H = p.H;
  const int part = tid & 15;
  const int e0 = blockIdx.z * COLS + (tid >> 4) * CPT;   // this half warp's first column
  const int nc = (n + CH - 1) / CH;
  const int q0 = p.q_start[r];
  const float* rec0 = p.records + ((size_t)(first_record(q0, r) + (t0 - q0) / CH) * H + h) * REC;
  auto fetch = [&](int c) {
    const float* src = rec0 + (size_t)c * H * REC;
    float* dst = smem + (c & 1) * REC;
    for (int i = tid; i < REC / 4; i += NT) cp_async16(dst + 4 * i, src + 4 * i);
  };
  fetch(0);
  cp_async_commit();
  auto place = [&](int v) -> float* {
    if (v == -1) return nullptr;
    return (v >= 0 ? p.state + ((size_t)v * H + h) * E * D : p.scratch + ((size_t)(-(v + 2)) * H + h) * E * D);
  };
  const float* st_in = place(src);
  const bool quads = (D & 3) == 0;
  f32x2 S[CPT][RPT / 2];
#pragma unroll
  for (int c = 0; c < CPT; ++c) {
#pragma unroll
    for (int j = 0; j < QUADS; ++j) {
      const int d = (j * 16 + part) * 4;
      float x[4] = {0.f, 0.f, 0.f, 0.f};
      if (st_in && e0 + c < E) {
        const float* st = st_in + (size_t)(e0 + c) * D;
        if (quads && d < D) {
          const float4 s4 = *reinterpret_cast<const float4*>(st + d);
          x[0] = s4.x; x[1] = s4.y; x[2] = s4.z; x[3] = s4.w;
        } else if (!quads) {
#pragma unroll
          for (int k = 0; k < 4; ++k)
            if (d + k < D) x[k] = st[d + k];
        }
      }
      S[c][2 * j] = pack2(x[0], x[1]);
      S[c][2 * j + 1] = pack2(x[2], x[3]);
    }
  }
  // this lane's token of a chunk: its U in this half warp's columns, requested a chunk ahead
  float u_next[CPT];
  auto request_u = [&](int c) {
    const int t = c * CH + part;
#pragma unroll
    for (int k = 0; k < CPT; ++k)
      u_next[k] = (t < n && e0 + k < E) ? to_float(p.u[(size_t)(t0 + t) * p.ld_u + h * E + e0 + k]) : 0.f;
  };
  request_u(0);
  f32x2 product[OWN ? RPT / 2 : 1];        // of the decays of this lane's key channels
#pragma unroll
  for (int j = 0; j < (OWN ? RPT / 2 : 1); ++j) product[j] = pack2(1.f, 1.f);

#pragma unroll 1
  for (int c = 0; c < nc; ++c) {
    cp_async_wait_all();
    __syncthreads();       // chunk c has landed, chunk c - 1 is computed by all (its buffer is free)
    if (c + 1 < nc) fetch(c + 1);
    cp_async_commit();
    float x[CPT];          // token `part`: U, then u
#pragma unroll
    for (int k = 0; k < CPT; ++k) x[k] = u_next[k];
    if (c + 1 < nc) request_u(c + 1);
    const float* rec = smem + (c & 1) * REC;
    // the chunk's products with the state at its start: which = 0: W, 1: QG
    float dot[2][CPT];
#pragma unroll
    for (int which = CORRECT ? 0 : 1; which < (OWN ? 1 : 2); ++which) {
      float v[CPT][CH];
      const float* base = rec + (which == 0 ? rec_w(DP) : 0) + part * 4;
#pragma unroll
      for (int first = 0; first < CH; first += TG) {
        f32x2 acc[CPT][TG];
#pragma unroll
        for (int k = 0; k < CPT; ++k)
#pragma unroll
          for (int j = 0; j < TG; ++j) acc[k][j] = 0ull;
#pragma unroll
        for (int j = 0; j < QUADS; ++j) {
#pragma unroll
          for (int tt = 0; tt < TG; ++tt) {
            const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(base + (first + tt) * DP + j * 64);
#pragma unroll
            for (int k = 0; k < CPT; ++k) {
              acc[k][tt] = fma2(S[k][2 * j], w.x, acc[k][tt]);
              acc[k][tt] = fma2(S[k][2 * j + 1], w.y, acc[k][tt]);
            }
          }
        }
#pragma unroll
        for (int k = 0; k < CPT; ++k)
#pragma unroll
          for (int tt = 0; tt < TG; ++tt) {
            float lo, hi;
            unpack2(acc[k][tt], lo, hi);
            v[k][first + tt] = lo + hi;
          }
      }
#pragma unroll
      for (int k = 0; k < CPT; ++k) dot[which][k] = scatter_sum(v[k], part);
    }
    if (CORRECT) {
#pragma unroll
      for (int k = 0; k < CPT; ++k) x[k] -= dot[0][k];
    }
    // S <- decays * S + sum over the tokens of kd u^T; the read-outs add what the chunk's own writes give
#pragma unroll
    for (int j = 0; j < QUADS; ++j) {
      const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(rec + rec_decay(DP) + part * 4 + j * 64);
      if (OWN) {
        product[2 * j] = mul2(product[2 * j], w.x);
        product[2 * j + 1] = mul2(product[2 * j + 1], w.y);
      }
#pragma unroll
      for (int k = 0; k < CPT; ++k) {
        S[k][2 * j] = mul2(S[k][2 * j], w.x);
        S[k][2 * j + 1] = mul2(S[k][2 * j + 1], w.y);
      }
    }
    const float* mq = rec + rec_mq(DP) + part;
    const float* kd = rec + rec_kd(DP) + part * 4;
#pragma unroll
    for (int i = 0; i < CH; ++i) {
      const float m = OWN ? 0.f : mq[i * CH];
      f32x2 u[CPT];
#pragma unroll
      for (int k = 0; k < CPT; ++k) {
        const float ui = __shfl_sync(0xffffffffu, x[k], i, 16);     // every lane gets token i's u
        if (!OWN) dot[1][k] = fmaf(m, ui, dot[1][k]);
        u[k] = pack2(ui, ui);
      }
#pragma unroll
      for (int j = 0; j < QUADS; ++j) {
        const ulonglong2 y = *reinterpret_cast<const ulonglong2*>(kd + i * DP + j * 64);
#pragma unroll
        for (int k = 0; k < CPT; ++k) {
          S[k][2 * j] = fma2(y.x, u[k], S[k][2 * j]);
          S[k][2 * j + 1] = fma2(y.y, u[k], S[k][2 * j + 1]);
        }
      }
    }
    const int t = c * CH + part;
    if (!OWN && t < n) {
      float* o = p.out + ((size_t)(t0 + t) * H + h) * E + e0;
#pragma unroll
      for (int k = 0; k < CPT; ++k)
        if (e0 + k < E) o[k] = dot[1][k];
    }
  }
  float* st_out = place(dst);
  if (OWN && dst <= -2 && blockIdx.z == 0 && (tid >> 4) == 0) {
    float* out = p.own_decay + ((size_t)(-(dst + 2)) * H + h) * D;
#pragma unroll
    for (int j = 0; j < QUADS; ++j) {
      const int d = (j * 16 + part) * 4;
      float x[4];
      unpack2(product[2 * j], x[0], x[1]);
      unpack2(product[2 * j + 1], x[2], x[3]);
#pragma unroll
      for (int k = 0; k < 4; ++k)
        if (d + k < D) out[d + k] = x[k];
    }
  }
  if (!st_out || (dst >= 0 && !p.write_state)) return;
#pragma unroll
  for (int c = 0; c < CPT; ++c) {
    if (e0 + c >= E) continue;
    float* st = st_out + (size_t)(e0 + c) * D;
#pragma unroll
    for (int j = 0; j < QUADS; ++j) {
      const int d = (j * 16 + part) * 4;
      float x[4];
      unpack2(S[c][2 * j], x[0], x[1]);
      unpack2(S[c][2 * j + 1], x[2], x[3]);
      if (quads && d < D) {
        *reinterpret_cast<float4*>(st + d) = make_float4(x[0], x[1], x[2], x[3]);
      } else if (!quads) {
#pragma unroll
        for (int k = 0; k < 4; ++k)
          if (d + k < D) st[d + k] = x[k];
      }
    }
  }
}

// The states at the segments' starts from the segments' own contributions, in place.  desc [m, 4]: state row,
// first scratch entry, segments, rows of a segment.
static __global__ void segment_starts_kernel(const float* state, float* scratch, const float* own_decay,
                                             const int32_t* desc, int H, int D, int E) {
  pdl_launch_dependents();
  pdl_wait();
  const int32_t* d = desc + (size_t)blockIdx.x * 4;
  const int h = blockIdx.y;
  const size_t per_head = (size_t)E * D, i = (size_t)blockIdx.z * blockDim.x + threadIdx.x;
  if (i >= per_head) return;
  float S = state[((size_t)d[0] * H + h) * per_head + i];
  for (int c = 0; c < d[2]; ++c) {
    const size_t entry = (size_t)(d[1] + c) * H + h;
    float* u = scratch + entry * per_head + i;
    const bool more = c + 1 < d[2];               // the last segment leaves no contribution
    const float own = more ? *u : 0.f, w = more ? own_decay[entry * D + i % D] : 0.f;
    *u = S;
    S = fmaf(w, S, own);
  }
}

// Launched without the programmatic dependency: its few long-running blocks would else be placed while the
// kernel before still fills most multiprocessors, several on the same one.
template <typename... KArgs, typename... Args>
void launch_spread(void (*kernel)(KArgs...), dim3 grid, int threads, size_t smem, cudaStream_t stream, Args... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = dim3(threads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...);
}


}  // namespace pbe
