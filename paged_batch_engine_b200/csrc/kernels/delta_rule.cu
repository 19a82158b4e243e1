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
// delta_chunks and the scan of chunk_scan.cuh: the same recurrence for prompt portions, sixteen tokens of a request at
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
#include "chunk_scan.cuh"
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
    if (st_out && j > 0) put_v<V>(st_out + (size_t)(j - 1) * C + c, u);     // entry j - 1 was read the turn before
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
        put_v<V>(out + d, q[n]);
        put_v<V>(out + D + d, k[n]);
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
        put_v<V>(p.v + (size_t)t * H * E + h * E + e, v);
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
  const int r = record_owner<128>(rec, p.q_start, p.q_len, p.R);
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
  float* out = p.records + ((size_t)rec * H + h) * record_floats(DP, true);
  float* mq = out + rec_mq(DP);
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
    float* kd = out + rec_kd(DP) + i * DP;
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
      out[j * DP + d] = Q[j * DP + d] * up;
    }
    out[rec_decay(DP) + d] = up;
    times_tb(kg, [&](int j, float s) { out[rec_w(DP) + j * DP + d] = s; });
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

template <int RPT, int CPT, int WARPS>
int launch_chunks(const ChunkParams& g, const ChunkScanParams<float>& p, int records, bool chan, cudaStream_t stream) {
  constexpr int DP = 16 * RPT, COLS = 2 * WARPS * CPT;
  constexpr size_t smem_g = sizeof(float) * 3 * CH * DP, smem_p = sizeof(float) * 2 * record_floats(DP, true);
  static bool opted = false;
  if (!opted) {
    cudaFuncSetAttribute(delta_chunks_kernel<DP, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_g);
    cudaFuncSetAttribute(delta_chunks_kernel<DP, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_g);
    const cudaError_t e = cudaFuncSetAttribute(scan_chunks_kernel<RPT, CPT, WARPS, true, false, float>,
                                               cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_p);
    if (e != cudaSuccess) return (int)e;
    opted = true;
  }
  const dim3 grid(records, g.H);
  if (chan) launch_k(delta_chunks_kernel<DP, true>, grid, 128, smem_g, stream, g);
  else launch_k(delta_chunks_kernel<DP, false>, grid, 128, smem_g, stream, g);
  const int err = launch_status();
  if (err != 0) return err;
  launch_spread(scan_chunks_kernel<RPT, CPT, WARPS, true, false, float>, dim3(g.R, g.H, (g.E + COLS - 1) / COLS), 32 * WARPS, smem_p,
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
  return D <= 64 ? record_floats(64, true) : D <= 128 ? record_floats(128, true) : D <= 256 ? record_floats(256, true) : 0;
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
  const ChunkScanParams<float> p{records, v, H * E, out, state, q_start, q_len, slots, H, D, E, write_state};
  const int n = T / CH + R;
  const bool chan = per_channel != 0;
  if (D <= 64) return launch_chunks<4, 2, 4>(g, p, n, chan, stream);
  if (D <= 128) return launch_chunks<8, 2, 4>(g, p, n, chan, stream);
  return launch_chunks<16, 2, 4>(g, p, n, chan, stream);
}
