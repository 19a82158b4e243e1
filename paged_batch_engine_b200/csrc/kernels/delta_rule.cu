// The gated delta rule: a matrix state per head that decays and is corrected by the error of what it
// predicts for the current key,
//
//   S <- g * S,   u = beta (v - S^T k),   S <- S + k u^T,   o = S^T q            (S: [D, E], float32)
//
// with a decay g per head, or one per head and key channel (the rows of S).  q and k are unit vectors
// behind a short causal convolution and silu, shared by neighbouring heads; v passes the same.
//
// delta_inputs: everything that enters the recurrence, in float32 and once per token: the
//   convolutions (taps inputs per channel: the projection's rows of this step, before them the
//   request's state row), silu, the unit norms, k . q, beta = sigmoid, g = exp(-exp(A) softplus(a + c)).
//   A warp takes one query/key head (both vectors, so their product costs nothing more) or one value
//   head of one token.  A request that brings one token has its convolution state moved on in the same
//   launch: each channel is read and written by one thread only.  delta_conv_state moves the others.
// delta_scan: the recurrence.  A block takes (request, head, slice of value columns); PARTS
//   neighbouring lanes share a column of S and hold RPT of its rows each in registers.  Both dot
//   products of a token are taken from the decayed state before its correction - the read-out is
//   S^T q = (g S)^T q + (k . q) u - so one round of shuffles serves both, and a token's dependent
//   chain is: the lanes' multiply-adds, log2(PARTS) shuffles, u, the update.  Tokens are staged TB at a
//   time in two shared-memory buffers by cp.async.  The state is laid out [head][column][key channel],
//   so that the lanes of a column read and write consecutive 16-byte pieces.  Steps of single tokens
//   take this kernel.
// delta_chunks / delta_scan_chunks: the same recurrence for prompt portions, sixteen tokens of a request at
//   a time.  With S the state at a chunk's start, kg_j and qg_j token j's key and query times all decays up
//   to j, kd_j its key times the decays after j, and
//       L_ji = beta_j k_j . (decays after i up to j) k_i  (i < j),    M_ij = k_i . (decays after i up to j) q_j  (i <= j),
//   the corrections solve (I + L) u = beta (v - S^T kg), a triangular system of sixteen unknowns whose
//   matrix belongs to the head, not to the column: delta_chunks inverts it and forms
//       W = (I + L)^-1 beta kg   and   U = (I + L)^-1 beta v,
//   so that the scan over chunks is u = U - S^T W, o_j = S^T qg_j + sum_{i<=j} M_ij u_i and
//   S <- (all decays) S + sum_j kd_j u_j^T: products of small matrices, one round of shuffles for sixteen
//   tokens.  All decay products are products of numbers in (0, 1], no ratio is formed, so nothing can
//   overflow; the inverse's entries are bounded by one because every step of the rule is a contraction
//   for keys of at most unit length.  Everything is float32.
#include "common.cuh"
#include "pdl.cuh"

using namespace pbe;

namespace {
constexpr int MAX_TAPS = 16;
constexpr int MAX_HEAD = 512;        // widest key or value head

struct InputParams {
  const void* proj;          // [T, ld]: queries at column 0, keys at G * D, values at 2 G D
  int ld;
  const float* conv_t;       // [taps, C], C = 2 G D + H E; the last tap is the current token's
  float* conv_state;         // [slots, taps - 1, C], the newest input last
  const float* small;        // [T, ld_small] float32: beta's pre-activations at column 0, (per head) decay's at H
  int ld_small;
  const float* chan;         // [T, ld_chan] float32 pre-activations of the channels' decays, or null (one per head)
  int ld_chan;
  const float* dt_bias;      // [H] or [H * D]
  const float* a_log;        // [H]
  float* qk;                 // [T, G, 2, D]
  float* kq;                 // [T, G]
  float* v;                  // [T, H * E]
  float* beta;               // [T, H]
  float* decay;              // [T, H] or [T, H * D]
  const int32_t* request_of_row;
  const int32_t* q_start;
  const int32_t* q_len;
  const int32_t* slots;
  int T, R, G, H, D, E, taps, update;
  float q_scale, unit_eps;
};

__device__ __forceinline__ float softplus_(float x) { return x > 20.f ? x : log1pf(expf(x)); }

template <int V>
__device__ __forceinline__ void load_v(const float* p, float (&a)[V]) {
  if constexpr (V == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    a[0] = v.x; a[1] = v.y; a[2] = v.z; a[3] = v.w;
  } else {
    a[0] = *p;
  }
}
template <int V>
__device__ __forceinline__ void load_v(const __nv_bfloat16* p, float (&a)[V]) {
  if constexpr (V == 4) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    a[0] = lo.x; a[1] = lo.y; a[2] = hi.x; a[3] = hi.y;
  } else {
    a[0] = __bfloat162float(*p);
  }
}
template <int V>
__device__ __forceinline__ void store_v(float* p, const float (&a)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(a[0], a[1], a[2], a[3]);
  else *p = a[0];
}

// The convolution of V neighbouring channels from column c of one token, with silu.
template <typename T, int V>
__device__ __forceinline__ void conv_silu(const InputParams& p, int t, int i, const float* st_in, float* st_out, int C,
                                          int c, float (&acc)[V]) {
#pragma unroll
  for (int k = 0; k < V; ++k) acc[k] = 0.f;
  const int taps = p.taps;
  const T* in = (const T*)p.proj + c;
  for (int j = 0; j < taps; ++j) {
    const int off = i - (taps - 1) + j;          // the input's place among this step's rows; negative: before them
    float u[V], w[V];
    if (off >= 0) load_v<V>(in + (size_t)(t - (taps - 1) + j) * p.ld, u);
    else load_v<V>(st_in + (size_t)(taps - 1 + off) * C + c, u);
    load_v<V>(p.conv_t + (size_t)j * C + c, w);
#pragma unroll
    for (int k = 0; k < V; ++k) acc[k] = fmaf(w[k], u[k], acc[k]);
    if (st_out && j > 0) store_v<V>(st_out + (size_t)(j - 1) * C + c, u);     // entry j - 1 was read the turn before
  }
#pragma unroll
  for (int k = 0; k < V; ++k) acc[k] = acc[k] / (1.0f + expf(-acc[k]));
}

constexpr int IN_WARPS = 4;

// grid (rows, ceil((G + H) / IN_WARPS) + 1): a warp per head of a token; the last block of a row makes
// beta and the decays.  N: groups of 32 * V channels a head has at most.
template <typename T, int V, int N>
__global__ void __launch_bounds__(IN_WARPS * 32) delta_inputs_kernel(InputParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const int G = p.G, H = p.H, D = p.D, E = p.E;
  const int C = 2 * G * D + H * E;
  const int r = p.request_of_row[t];
  const bool live = r >= 0 && r < p.R && p.q_len[r] > 0;        // not a padding row of a captured step
  if (blockIdx.y == gridDim.y - 1) {
    for (int h = threadIdx.x; h < H; h += blockDim.x) {
      const float b = live ? p.small[(size_t)t * p.ld_small + h] : 0.f;
      p.beta[(size_t)t * H + h] = 1.0f / (1.0f + expf(-b));
      if (!p.chan) {
        const float a = live ? p.small[(size_t)t * p.ld_small + H + h] + p.dt_bias[h] : 0.f;
        p.decay[(size_t)t * H + h] = expf(-expf(p.a_log[h]) * softplus_(a));
      }
    }
    if (p.chan) {
      for (int i = threadIdx.x; i < H * D; i += blockDim.x) {
        const float a = live ? p.chan[(size_t)t * p.ld_chan + i] + p.dt_bias[i] : 0.f;
        p.decay[(size_t)t * H * D + i] = expf(-expf(p.a_log[i / D]) * softplus_(a));
      }
    }
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.y * IN_WARPS + warp;
  if (head >= G + H) return;
  const bool is_qk = head < G;
  const int i = live ? t - p.q_start[r] : 0;
  float* st = live && p.taps > 1 ? p.conv_state + (size_t)p.slots[r] * (p.taps - 1) * C : nullptr;
  float* st_out = (live && p.update && p.q_len[r] == 1) ? st : nullptr;
  if (is_qk) {
    float q[N][V], k[N][V];
    float qq = 0.f, kk = 0.f;
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int d = (n * 32 + lane) * V;
#pragma unroll
      for (int e = 0; e < V; ++e) q[n][e] = k[n][e] = 0.f;
      if (d < D && live) {
        conv_silu<T, V>(p, t, i, st, st_out, C, head * D + d, q[n]);
        conv_silu<T, V>(p, t, i, st, st_out, C, G * D + head * D + d, k[n]);
      }
#pragma unroll
      for (int e = 0; e < V; ++e) {
        qq = fmaf(q[n][e], q[n][e], qq);
        kk = fmaf(k[n][e], k[n][e], kk);
      }
    }
    const float qs = p.q_scale / sqrtf(warp_sum(qq) + p.unit_eps), ks = 1.0f / sqrtf(warp_sum(kk) + p.unit_eps);
    float dot = 0.f;
    float* out = p.qk + ((size_t)t * G + head) * 2 * D;
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int d = (n * 32 + lane) * V;
#pragma unroll
      for (int e = 0; e < V; ++e) {
        q[n][e] *= qs;
        k[n][e] *= ks;
        dot = fmaf(q[n][e], k[n][e], dot);
      }
      if (d < D) {
        store_v<V>(out + d, q[n]);
        store_v<V>(out + D + d, k[n]);
      }
    }
    dot = warp_sum(dot);
    if (lane == 0) p.kq[(size_t)t * G + head] = dot;
  } else {
    const int h = head - G;
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int e = (n * 32 + lane) * V;
      if (e < E) {
        float v[V];
#pragma unroll
        for (int k = 0; k < V; ++k) v[k] = 0.f;
        if (live) conv_silu<T, V>(p, t, i, st, st_out, C, 2 * G * D + h * E + e, v);
        store_v<V>(p.v + (size_t)t * H * E + h * E + e, v);
      }
    }
  }
}

// The convolution state after a portion of two or more tokens (one token: delta_inputs did it).
template <typename T>
__global__ void delta_conv_state_kernel(InputParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x;
  const int C = 2 * p.G * p.D + p.H * p.E;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  const int n = p.q_len[r];
  if (c >= C || n <= 1) return;
  const int keep = p.taps - 1;
  float* st = p.conv_state + (size_t)p.slots[r] * keep * C + c;
  const T* in = (const T*)p.proj + c;
  const int t0 = p.q_start[r];
  for (int i = 0; i < keep; ++i) {                 // ascending: entry i + n > i is still the old one
    const int li = n - keep + i;
    st[(size_t)i * C] = li >= 0 ? to_float(in[(size_t)(t0 + li) * p.ld]) : st[(size_t)(i + n) * C];
  }
}

// ------------------------------------------------------------------ delta_scan
struct ScanParams {
  const float* qk;           // [T, G, 2, D]
  const float* kq;           // [T, G]
  const float* v;            // [T, H * E]
  const float* beta;         // [T, H]
  const float* decay;        // [T, H] or [T, H * D]
  float* out;                // [T, H * E]
  float* state;              // [slots, H, E, D]
  const int32_t* q_start;
  const int32_t* q_len;
  const int32_t* slots;
  int G, H, D, E, write_state;
};

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

template <int RPT, int PARTS, int WARPS, int TB, bool CHAN>
__global__ void __launch_bounds__(32 * WARPS) delta_scan_kernel(ScanParams p) {
  constexpr int NT = 32 * WARPS;
  constexpr int COLS = NT / PARTS;
  constexpr int DMAX = RPT * PARTS;
  constexpr int QUADS = RPT / 4;               // 16-byte pieces of a column a lane holds
  constexpr int VECS = CHAN ? 3 : 2;           // staged vectors of D: q, k (and the channels' decays)
  __shared__ __align__(16) float vec[2][TB][VECS][DMAX];
  __shared__ float vs[2][TB][COLS], outs[2][TB][COLS];
  __shared__ float sc[2][TB][3];               // beta, k . q, the head's decay
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x, h = blockIdx.y;
  const int tid = threadIdx.x;
  const int n = p.q_len[r];
  if (n <= 0) return;
  const int t0 = p.q_start[r];
  const int D = p.D, E = p.E, H = p.H, G = p.G;
  const int kvh = h / (H / G);
  const int part = tid % PARTS, col = tid / PARTS;
  const int e0 = blockIdx.z * COLS, e = e0 + col;
  const bool live = e < E;
  const bool quads = (D & 3) == 0;

  auto fetch = [&](int b) {                    // batch b into buffer b & 1
    const int buf = b & 1;
    const int first = b * TB, count = min(TB, n - first);
    const size_t row0 = (size_t)t0 + first;
    if (quads) {
      const int dq = D >> 2;
      for (int i = tid; i < count * 2 * dq; i += NT) {
        const int tt = i / (2 * dq), j = i - tt * 2 * dq;
        const int which = j >= dq, d = (j - which * dq) * 4;
        cp_async16(&vec[buf][tt][which][d], p.qk + (((row0 + tt) * G + kvh) * 2 + which) * D + d);
      }
      if (CHAN)
        for (int i = tid; i < count * dq; i += NT) {
          const int tt = i / dq, d = (i - tt * dq) * 4;
          cp_async16(&vec[buf][tt][VECS - 1][d], p.decay + ((row0 + tt) * H + h) * D + d);
        }
    } else {
      for (int i = tid; i < count * 2 * D; i += NT) {
        const int tt = i / (2 * D), j = i - tt * 2 * D;
        const int which = j >= D, d = j - which * D;
        cp_async4(&vec[buf][tt][which][d], p.qk + (((row0 + tt) * G + kvh) * 2 + which) * D + d);
      }
      if (CHAN)
        for (int i = tid; i < count * D; i += NT) {
          const int tt = i / D, d = i - tt * D;
          cp_async4(&vec[buf][tt][VECS - 1][d], p.decay + ((row0 + tt) * H + h) * D + d);
        }
    }
    for (int i = tid; i < count * COLS; i += NT) {
      const int tt = i / COLS, c = i - tt * COLS;
      if (e0 + c < E) cp_async4(&vs[buf][tt][c], p.v + ((row0 + tt) * H + h) * E + e0 + c);
    }
    for (int tt = tid; tt < count; tt += NT) {
      cp_async4(&sc[buf][tt][0], p.beta + (row0 + tt) * H + h);
      cp_async4(&sc[buf][tt][1], p.kq + (row0 + tt) * G + kvh);
      if (!CHAN) cp_async4(&sc[buf][tt][2], p.decay + (row0 + tt) * H + h);
    }
  };

  // channels beyond D stay zero in both buffers (a copy never touches them)
  if (D < DMAX) {
    for (int i = tid; i < 2 * TB * VECS * (DMAX - D); i += NT) {
      const int v = i / (DMAX - D), d = D + i - v * (DMAX - D);
      (&vec[0][0][0][0])[v * DMAX + d] = 0.f;
    }
  }
  fetch(0);
  cp_async_commit();
  float* st = p.state + (((size_t)p.slots[r] * H + h) * E + (live ? e : 0)) * D;
  float S[RPT];
#pragma unroll
  for (int j = 0; j < QUADS; ++j) {
    const int d = (j * PARTS + part) * 4;
    if (quads && live && d < D) {
      const float4 s4 = *reinterpret_cast<const float4*>(st + d);
      S[4 * j] = s4.x; S[4 * j + 1] = s4.y; S[4 * j + 2] = s4.z; S[4 * j + 3] = s4.w;
    } else {
#pragma unroll
      for (int k = 0; k < 4; ++k) S[4 * j + k] = (live && d + k < D) ? st[d + k] : 0.f;
    }
  }

  // one token of buffer `buf`; returns the read-out of this thread's column
  auto step = [&](int buf, int tt) -> float {
    float kv[RPT];
    float a0 = 0.f, a1 = 0.f, b0 = 0.f, b1 = 0.f;
    const float g = CHAN ? 1.f : sc[buf][tt][2];
#pragma unroll
    for (int j = 0; j < QUADS; ++j) {
      const int d = (j * PARTS + part) * 4;
      const float4 q4 = *reinterpret_cast<const float4*>(&vec[buf][tt][0][d]);
      const float4 k4 = *reinterpret_cast<const float4*>(&vec[buf][tt][1][d]);
      kv[4 * j] = k4.x; kv[4 * j + 1] = k4.y; kv[4 * j + 2] = k4.z; kv[4 * j + 3] = k4.w;
      if (CHAN) {
        const float4 g4 = *reinterpret_cast<const float4*>(&vec[buf][tt][VECS - 1][d]);
        S[4 * j] *= g4.x; S[4 * j + 1] *= g4.y; S[4 * j + 2] *= g4.z; S[4 * j + 3] *= g4.w;
      } else {
        S[4 * j] *= g; S[4 * j + 1] *= g; S[4 * j + 2] *= g; S[4 * j + 3] *= g;
      }
      a0 = fmaf(S[4 * j], k4.x, a0);
      a1 = fmaf(S[4 * j + 1], k4.y, a1);
      a0 = fmaf(S[4 * j + 2], k4.z, a0);
      a1 = fmaf(S[4 * j + 3], k4.w, a1);
      b0 = fmaf(S[4 * j], q4.x, b0);
      b1 = fmaf(S[4 * j + 1], q4.y, b1);
      b0 = fmaf(S[4 * j + 2], q4.z, b0);
      b1 = fmaf(S[4 * j + 3], q4.w, b1);
    }
    float a = a0 + a1, b = b0 + b1;
#pragma unroll
    for (int m = 1; m < PARTS; m <<= 1) {
      a += __shfl_xor_sync(0xffffffffu, a, m);
      b += __shfl_xor_sync(0xffffffffu, b, m);
    }
    const float u = sc[buf][tt][0] * (vs[buf][tt][col] - a);
#pragma unroll
    for (int i = 0; i < RPT; ++i) S[i] = fmaf(kv[i], u, S[i]);
    return fmaf(sc[buf][tt][1], u, b);
  };
  auto flush = [&](int b) {                    // the read-outs of batch b, a slice's columns side by side
    const int first = b * TB, count = min(TB, n - first);
    for (int i = tid; i < count * COLS; i += NT) {
      const int tt = i / COLS, c = i - tt * COLS;
      if (e0 + c < E) p.out[((size_t)(t0 + first + tt) * H + h) * E + e0 + c] = outs[b & 1][tt][c];
    }
  };

  const int nb = (n + TB - 1) / TB;
  for (int b = 0; b < nb; ++b) {
    cp_async_wait_all();
    __syncthreads();       // batch b has landed, batch b - 1 is computed (its buffer is free, its read-outs are written)
    if (b + 1 < nb) fetch(b + 1);
    cp_async_commit();
    if (b > 0) flush(b - 1);
    const int buf = b & 1, count = min(TB, n - b * TB);
    float o[TB];
    if (count == TB) {
#pragma unroll
      for (int tt = 0; tt < TB; ++tt) o[tt] = step(buf, tt);
#pragma unroll
      for (int tt = 0; tt < TB; ++tt)
        if (part == 0) outs[buf][tt][col] = o[tt];
    } else {
      for (int tt = 0; tt < count; ++tt) {
        const float y = step(buf, tt);
        if (part == 0) outs[buf][tt][col] = y;
      }
    }
  }
  __syncthreads();
  flush(nb - 1);
  if (live && p.write_state) {
#pragma unroll
    for (int j = 0; j < QUADS; ++j) {
      const int d = (j * PARTS + part) * 4;
      if (quads && d < D) {
        *reinterpret_cast<float4*>(st + d) = make_float4(S[4 * j], S[4 * j + 1], S[4 * j + 2], S[4 * j + 3]);
      } else if (!quads) {
#pragma unroll
        for (int k = 0; k < 4; ++k)
          if (d + k < D) st[d + k] = S[4 * j + k];
      }
    }
  }
}

// ------------------------------------------------------------------ chunks of sixteen tokens
constexpr int CH = 16;

// A record holds a chunk of one head: W, QG and KD [CH][DP] each, the chunk's decay product [DP], MQ [CH][CH].
__host__ __device__ constexpr int record_floats(int dp) { return 3 * CH * dp + dp + CH * CH; }
// The records of a request that starts at row q of the step: they begin at q / CH + r, which leaves every
// request room for all its chunks (the last of them may be short) without overlap.
__device__ __forceinline__ int first_record(int q_start, int r) { return q_start / CH + r; }

struct ChunkParams {
  const float* qk;           // [T, G, 2, D]
  const float* decay;        // [T, H] or [T, H * D]
  const float* beta;         // [T, H]
  float* v;                  // [T, H * E]: v in, U out
  float* records;            // [first_record(T, R)][H][record_floats(DP)]
  const int32_t* q_start;
  const int32_t* q_len;
  int R, G, H, D, E;
};

// grid (records, H), a block of 128 threads a chunk and head
template <int DP, bool CHAN>
__global__ void __launch_bounds__(128, 4) delta_chunks_kernel(ChunkParams p) {
  extern __shared__ __align__(16) float smem[];
  float* K = smem;                        // [CH][DP]
  float* Q = K + CH * DP;                 // [CH][DP]
  float* W = Q + CH * DP;                 // [CH][DP] decays
  __shared__ float Lk[CH][CH + 1];        // [j][i]: beta_j k_i . (decays after i up to j) k_j, i < j
  __shared__ __align__(16) float Tb[CH][CH];   // (I + Lk)^-1, columns times beta
  __shared__ float beta[CH];
  pdl_launch_dependents();
  pdl_wait();
  const int rec = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int D = p.D, E = p.E, H = p.H, G = p.G;
  // whose chunk this is: each thread looks at some of the requests, one of them finds it
  __shared__ int owner;
  if (tid == 0) owner = -1;
  __syncthreads();
  for (int i = tid; i < p.R; i += 128) {
    const int first = first_record(p.q_start[i], i);
    if (rec >= first && rec < first + (p.q_len[i] + CH - 1) / CH) owner = i;
  }
  __syncthreads();
  const int r = owner;
  if (r < 0) return;
  const int c = rec - first_record(p.q_start[r], r);
  const int count = min(CH, p.q_len[r] - c * CH);
  const size_t row0 = (size_t)p.q_start[r] + c * CH;
  const int g = h / (H / G);
  if ((D & 3) == 0) {                     // sixteen bytes a load, all of a thread's loads in flight
#pragma unroll
    for (int n = 0; n < CH * DP / 512; ++n) {
      const int i = (tid + n * 128) * 4;
      const int j = i / DP, d = i % DP;
      const bool ok = j < count && d < D;
      float4 q4 = make_float4(0.f, 0.f, 0.f, 0.f), k4 = q4, w4 = make_float4(1.f, 1.f, 1.f, 1.f);
      if (ok) {
        const float* src = p.qk + ((row0 + j) * G + g) * 2 * D + d;
        q4 = *reinterpret_cast<const float4*>(src);
        k4 = *reinterpret_cast<const float4*>(src + D);
        if (CHAN) {
          w4 = *reinterpret_cast<const float4*>(p.decay + ((row0 + j) * H + h) * D + d);
        } else {
          const float w = p.decay[(row0 + j) * H + h];
          w4 = make_float4(w, w, w, w);
        }
      }
      *reinterpret_cast<float4*>(Q + i) = q4;
      *reinterpret_cast<float4*>(K + i) = k4;
      *reinterpret_cast<float4*>(W + i) = w4;
    }
  } else {
    for (int i = tid; i < CH * DP; i += 128) {
      const int j = i / DP, d = i % DP;
      const bool ok = j < count && d < D;
      const float* src = p.qk + ((row0 + (ok ? j : 0)) * G + g) * 2 * D + (ok ? d : 0);
      Q[i] = ok ? src[0] : 0.f;
      K[i] = ok ? src[D] : 0.f;
      W[i] = ok ? (CHAN ? p.decay[((row0 + j) * H + h) * D + d] : p.decay[(row0 + j) * H + h]) : 1.f;
    }
  }
  if (tid < CH) beta[tid] = tid < count ? p.beta[(row0 + tid) * H + h] : 0.f;
  __syncthreads();
  float* out = p.records + ((size_t)rec * H + h) * record_floats(DP);
  float* mq = out + 3 * CH * DP + DP;
  {
    // eight lanes share a token i, DP / 8 channels each; x runs over k_i times the decays after i
    constexpr int MPT = DP / 8;
    const int i = tid >> 3, slice = tid & 7;
    float x[MPT];
#pragma unroll
    for (int m = 0; m < MPT; ++m) x[m] = K[i * DP + slice + 8 * m];
    for (int j = 0; j < CH; ++j) {
      float ck = 0.f, cq = 0.f;
      if (j >= i) {
#pragma unroll
        for (int m = 0; m < MPT; ++m) {
          const int d = j * DP + slice + 8 * m;
          if (j > i) x[m] *= W[d];
          ck = fmaf(x[m], K[d], ck);
          cq = fmaf(x[m], Q[d], cq);
        }
      }
#pragma unroll
      for (int m = 1; m < 8; m <<= 1) {
        ck += __shfl_xor_sync(0xffffffffu, ck, m);
        cq += __shfl_xor_sync(0xffffffffu, cq, m);
      }
      if (slice == 0) {
        Lk[j][i] = j > i ? beta[j] * ck : 0.f;
        mq[i * CH + j] = j >= i ? cq : 0.f;
      }
    }
    float* kd = out + 2 * CH * DP + i * DP;
#pragma unroll
    for (int m = 0; m < MPT; ++m) kd[slice + 8 * m] = x[m];
  }
  __syncthreads();
  if (tid < CH) {                          // a thread a column of the inverse, by substitution
    float t[CH];
#pragma unroll
    for (int j = 0; j < CH; ++j) {
      float s = j == tid ? 1.f : 0.f;
#pragma unroll
      for (int i = 0; i < j; ++i) s = fmaf(-Lk[j][i], t[i], s);      // t[i] is 0 above the diagonal
      t[j] = s;
      Tb[j][tid] = s * beta[tid];
    }
  }
  __syncthreads();
  // rows j of Tb times a column of sixteen numbers
  auto times_tb = [&](const float (&y)[CH], auto&& put) {
#pragma unroll
    for (int j = 0; j < CH; ++j) {
      float s = 0.f;
#pragma unroll
      for (int i = 0; i <= j; i += 4) {
        const float4 t4 = *reinterpret_cast<const float4*>(&Tb[j][i]);
        s = fmaf(t4.x, y[i], s);
        if (i + 1 <= j) s = fmaf(t4.y, y[i + 1], s);
        if (i + 2 <= j) s = fmaf(t4.z, y[i + 2], s);
        if (i + 3 <= j) s = fmaf(t4.w, y[i + 3], s);
      }
      put(j, s);
    }
  };
  for (int d = tid; d < DP; d += 128) {
    float kg[CH];
    float up = 1.f;
#pragma unroll
    for (int j = 0; j < CH; ++j) {
      up *= W[j * DP + d];
      kg[j] = K[j * DP + d] * up;
      out[CH * DP + j * DP + d] = Q[j * DP + d] * up;
    }
    out[3 * CH * DP + d] = up;
    times_tb(kg, [&](int j, float s) { out[j * DP + d] = s; });
  }
  for (int e = tid; e < E; e += 128) {
    float y[CH];
#pragma unroll
    for (int j = 0; j < CH; ++j) y[j] = j < count ? p.v[((row0 + j) * H + h) * E + e] : 0.f;
    times_tb(y, [&](int j, float s) {
      if (j < count) p.v[((row0 + j) * H + h) * E + e] = s;
    });
  }
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

struct ChunkScanParams {
  const float* records;
  const float* u;            // [T, H * E]
  float* out;                // [T, H * E]
  float* state;              // [slots, H, E, D]
  const int32_t* q_start;
  const int32_t* q_len;
  const int32_t* slots;
  int H, D, E, write_state;
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
template <int RPT, int CPT, int WARPS>
__global__ void __launch_bounds__(32 * WARPS) delta_scan_chunks_kernel(ChunkScanParams p) {
  constexpr int NT = 32 * WARPS;
  constexpr int DP = 16 * RPT;
  constexpr int QUADS = RPT / 4;
  constexpr int COLS = 2 * WARPS * CPT;
  constexpr int REC = record_floats(DP);
  extern __shared__ __align__(16) float smem[];          // two records
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x, h = blockIdx.y;
  const int tid = threadIdx.x;
  const int n = p.q_len[r];
  if (n <= 0) return;
  const int t0 = p.q_start[r];
  const int D = p.D, E = p.E, H = p.H;
  const int part = tid & 15;
  const int e0 = blockIdx.z * COLS + (tid >> 4) * CPT;   // this half warp's first column
  const int nc = (n + CH - 1) / CH;
  const float* rec0 = p.records + ((size_t)first_record(t0, r) * H + h) * REC;
  auto fetch = [&](int c) {
    const float* src = rec0 + (size_t)c * H * REC;
    float* dst = smem + (c & 1) * REC;
    for (int i = tid; i < REC / 4; i += NT) cp_async16(dst + 4 * i, src + 4 * i);
  };
  fetch(0);
  cp_async_commit();
  float* st_head = p.state + ((size_t)p.slots[r] * H + h) * E * D;
  const bool quads = (D & 3) == 0;
  f32x2 S[CPT][RPT / 2];
#pragma unroll
  for (int c = 0; c < CPT; ++c) {
#pragma unroll
    for (int j = 0; j < QUADS; ++j) {
      const int d = (j * 16 + part) * 4;
      float x[4] = {0.f, 0.f, 0.f, 0.f};
      if (e0 + c < E) {
        const float* st = st_head + (size_t)(e0 + c) * D;
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
      u_next[k] = (t < n && e0 + k < E) ? p.u[((size_t)(t0 + t) * H + h) * E + e0 + k] : 0.f;
  };
  request_u(0);

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
    for (int which = 0; which < 2; ++which) {
      f32x2 acc[CPT][CH];
#pragma unroll
      for (int k = 0; k < CPT; ++k)
#pragma unroll
        for (int j = 0; j < CH; ++j) acc[k][j] = 0ull;
      const float* base = rec + which * CH * DP + part * 4;
#pragma unroll
      for (int j = 0; j < QUADS; ++j) {
#pragma unroll
        for (int tt = 0; tt < CH; ++tt) {
          const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(base + tt * DP + j * 64);
#pragma unroll
          for (int k = 0; k < CPT; ++k) {
            acc[k][tt] = fma2(S[k][2 * j], w.x, acc[k][tt]);
            acc[k][tt] = fma2(S[k][2 * j + 1], w.y, acc[k][tt]);
          }
        }
      }
#pragma unroll
      for (int k = 0; k < CPT; ++k) {
        float v[CH];
#pragma unroll
        for (int tt = 0; tt < CH; ++tt) {
          float a, b;
          unpack2(acc[k][tt], a, b);
          v[tt] = a + b;
        }
        dot[which][k] = scatter_sum(v, part);
      }
    }
#pragma unroll
    for (int k = 0; k < CPT; ++k) x[k] -= dot[0][k];
    // every lane gets every token's u; the read-outs add what the chunk's own writes give
    const float* mq = rec + 3 * CH * DP + DP + part;
    f32x2 u[CPT][CH];
#pragma unroll
    for (int i = 0; i < CH; ++i) {
      const float m = mq[i * CH];
#pragma unroll
      for (int k = 0; k < CPT; ++k) {
        const float ui = __shfl_sync(0xffffffffu, x[k], i, 16);
        dot[1][k] = fmaf(m, ui, dot[1][k]);
        u[k][i] = pack2(ui, ui);
      }
    }
    const int t = c * CH + part;
    if (t < n) {
      float* o = p.out + ((size_t)(t0 + t) * H + h) * E + e0;
#pragma unroll
      for (int k = 0; k < CPT; ++k)
        if (e0 + k < E) o[k] = dot[1][k];
    }
    // S <- decays * S + sum over the tokens of kd u^T
    const float* kd = rec + 2 * CH * DP + part * 4;
#pragma unroll
    for (int j = 0; j < QUADS; ++j) {
      const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(rec + 3 * CH * DP + part * 4 + j * 64);
#pragma unroll
      for (int k = 0; k < CPT; ++k) {
        S[k][2 * j] = mul2(S[k][2 * j], w.x);
        S[k][2 * j + 1] = mul2(S[k][2 * j + 1], w.y);
      }
#pragma unroll
      for (int tt = 0; tt < CH; ++tt) {
        const ulonglong2 y = *reinterpret_cast<const ulonglong2*>(kd + tt * DP + j * 64);
#pragma unroll
        for (int k = 0; k < CPT; ++k) {
          S[k][2 * j] = fma2(y.x, u[k][tt], S[k][2 * j]);
          S[k][2 * j + 1] = fma2(y.y, u[k][tt], S[k][2 * j + 1]);
        }
      }
    }
  }
  if (!p.write_state) return;
#pragma unroll
  for (int c = 0; c < CPT; ++c) {
    if (e0 + c >= E) continue;
    float* st = st_head + (size_t)(e0 + c) * D;
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

template <int RPT, int CPT, int WARPS>
int launch_chunks(const ChunkParams& g, const ChunkScanParams& p, int records, bool chan, cudaStream_t stream) {
  constexpr int DP = 16 * RPT, COLS = 2 * WARPS * CPT;
  constexpr size_t smem_g = sizeof(float) * 3 * CH * DP, smem_p = sizeof(float) * 2 * record_floats(DP);
  static bool opted = false;
  if (!opted) {
    cudaFuncSetAttribute(delta_chunks_kernel<DP, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_g);
    cudaFuncSetAttribute(delta_chunks_kernel<DP, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_g);
    const cudaError_t e = cudaFuncSetAttribute(delta_scan_chunks_kernel<RPT, CPT, WARPS>,
                                               cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_p);
    if (e != cudaSuccess) return (int)e;
    opted = true;
  }
  const dim3 grid(records, g.H);
  if (chan) launch_k(delta_chunks_kernel<DP, true>, grid, 128, smem_g, stream, g);
  else launch_k(delta_chunks_kernel<DP, false>, grid, 128, smem_g, stream, g);
  const int err = launch_status();
  if (err != 0) return err;
  launch_spread(delta_scan_chunks_kernel<RPT, CPT, WARPS>, dim3(g.R, g.H, (g.E + COLS - 1) / COLS), 32 * WARPS, smem_p,
                stream, p);
  return launch_status();
}

template <int RPT, int PARTS, int WARPS, int TB>
void launch_scan(const ScanParams& p, int R, bool chan, cudaStream_t stream) {
  constexpr int COLS = 32 * WARPS / PARTS;
  dim3 grid(R, p.H, (p.E + COLS - 1) / COLS);
  if (chan) launch_k(delta_scan_kernel<RPT, PARTS, WARPS, TB, true>, grid, 32 * WARPS, 0, stream, p);
  else launch_k(delta_scan_kernel<RPT, PARTS, WARPS, TB, false>, grid, 32 * WARPS, 0, stream, p);
}

template <typename T, int V>
int launch_inputs(const InputParams& p, bool many, cudaStream_t stream) {
  const int wide = p.D > p.E ? p.D : p.E;
  dim3 grid(p.T, (p.G + p.H + IN_WARPS - 1) / IN_WARPS + 1);
  const int per = (wide + 32 * V - 1) / (32 * V);
  if (per <= 1) launch_k(delta_inputs_kernel<T, V, 1>, grid, IN_WARPS * 32, 0, stream, p);
  else if (per <= 2) launch_k(delta_inputs_kernel<T, V, 2>, grid, IN_WARPS * 32, 0, stream, p);
  else if (per <= 4) launch_k(delta_inputs_kernel<T, V, 4>, grid, IN_WARPS * 32, 0, stream, p);
  else if (per <= 16 / V) launch_k(delta_inputs_kernel<T, V, 16 / V>, grid, IN_WARPS * 32, 0, stream, p);
  else return (int)cudaErrorInvalidValue;
  int err = launch_status();
  if (err != 0 || !many || !p.update || p.taps == 1) return err;
  const int C = 2 * p.G * p.D + p.H * p.E;
  launch_k(delta_conv_state_kernel<T>, dim3(p.R, (C + 127) / 128), 128, 0, stream, p);
  return launch_status();
}
}  // namespace

// many: some request of the step brings more than one token (its convolution state moves in a launch of its own)
PBE_EXPORT int pbe_delta_inputs(const void* proj, int ld, int dtype, const float* conv_t, float* conv_state,
                                const float* small, int ld_small, const float* chan, int ld_chan, const float* dt_bias,
                                const float* a_log, float* qk, float* kq, float* v, float* beta, float* decay,
                                const int32_t* request_of_row, const int32_t* q_start, const int32_t* q_len,
                                const int32_t* slots, int T, int R, int G, int H, int D, int E, int taps, int update,
                                int many, float q_scale, float unit_eps, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (taps < 1 || taps > MAX_TAPS || D < 1 || E < 1 || D > MAX_HEAD || E > MAX_HEAD || G < 1 || H % G != 0)
    return (int)cudaErrorInvalidValue;
  InputParams p{proj, ld, conv_t, conv_state, small, ld_small, chan, ld_chan, dt_bias, a_log, qk, kq, v, beta, decay,
                request_of_row, q_start, q_len, slots, T, R, G, H, D, E, taps, update, q_scale, unit_eps};
  const bool vec4 = D % 4 == 0 && E % 4 == 0 && ld % 4 == 0 &&
                    (((uintptr_t)conv_t | (uintptr_t)conv_state | (uintptr_t)qk | (uintptr_t)v) & 15) == 0 &&
                    ((uintptr_t)proj & (dtype == PBE_F32 ? 15 : 7)) == 0;
  if (dtype == PBE_F32) return vec4 ? launch_inputs<float, 4>(p, many, stream) : launch_inputs<float, 1>(p, many, stream);
  return vec4 ? launch_inputs<__nv_bfloat16, 4>(p, many, stream) : launch_inputs<__nv_bfloat16, 1>(p, many, stream);
}

PBE_EXPORT int pbe_delta_scan(const float* qk, const float* kq, const float* v, const float* beta, const float* decay,
                              int per_channel, float* out, float* state, const int32_t* q_start, const int32_t* q_len,
                              const int32_t* slots, int R, int G, int H, int D, int E, int write_state,
                              cudaStream_t stream) {
  if (R <= 0) return 0;
  if (D < 1 || E < 1 || G < 1 || H % G != 0) return (int)cudaErrorInvalidValue;
  if ((D & 3) == 0 && (((uintptr_t)qk | (uintptr_t)state | (per_channel ? (uintptr_t)decay : 0)) & 15) != 0)
    return (int)cudaErrorMisalignedAddress;
  ScanParams p{qk, kq, v, beta, decay, out, state, q_start, q_len, slots, G, H, D, E, write_state};
  const bool chan = per_channel != 0;
  if (D <= 32) launch_scan<4, 8, 4, 8>(p, R, chan, stream);
  else if (D <= 64) launch_scan<8, 8, 4, 8>(p, R, chan, stream);
  else if (D <= 128) launch_scan<16, 8, 4, 8>(p, R, chan, stream);
  else if (D <= 256) launch_scan<16, 16, 4, 4>(p, R, chan, stream);
  else if (D <= MAX_HEAD) launch_scan<16, 32, 4, 2>(p, R, chan, stream);
  else return (int)cudaErrorInvalidValue;
  return launch_status();
}

// Floats of a chunk's record (a head), for key heads of D channels (0: too wide for the chunked form).
PBE_EXPORT int pbe_delta_record_floats(int D) {
  return D <= 64 ? record_floats(64) : D <= 128 ? record_floats(128) : D <= 256 ? record_floats(256) : 0;
}
PBE_EXPORT int pbe_delta_chunk_tokens() { return CH; }

// The same for steps with prompt portions, sixteen tokens of a request at a time: two launches.  v is
// overwritten.  records: [T / 16 + R][H][pbe_delta_record_floats(D)] floats of scratch memory.
PBE_EXPORT int pbe_delta_scan_chunks(const float* qk, float* v, const float* beta, const float* decay, int per_channel,
                                     float* out, float* state, float* records, const int32_t* q_start,
                                     const int32_t* q_len, const int32_t* slots, int T, int R, int G, int H, int D,
                                     int E, int write_state, cudaStream_t stream) {
  if (R <= 0 || T <= 0) return 0;
  if (D < 1 || D > 256 || E < 1 || G < 1 || H % G != 0 || records == nullptr) return (int)cudaErrorInvalidValue;
  if ((((uintptr_t)state | (uintptr_t)records) & 15) != 0) return (int)cudaErrorMisalignedAddress;
  if ((D & 3) == 0 && (((uintptr_t)qk | (per_channel ? (uintptr_t)decay : 0)) & 15) != 0)
    return (int)cudaErrorMisalignedAddress;
  const ChunkParams g{qk, decay, beta, v, records, q_start, q_len, R, G, H, D, E};
  const ChunkScanParams p{records, v, out, state, q_start, q_len, slots, H, D, E, write_state};
  const int n = T / CH + R;
  const bool chan = per_channel != 0;
  if (D <= 64) return launch_chunks<4, 2, 4>(g, p, n, chan, stream);
  if (D <= 128) return launch_chunks<8, 2, 4>(g, p, n, chan, stream);
  return launch_chunks<16, 2, 4>(g, p, n, chan, stream);
}
