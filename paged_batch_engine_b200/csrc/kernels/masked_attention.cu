// Grouped-query softmax attention over the paged cache with per-head query/key norms, keys and
// values of different widths, and a choice of what a row sees and what joins its softmax:
//
//   * mask: every earlier key, the last W keys (sliding window), or the earlier keys of the
//     row's own chunk of C positions (chunks counted from position 0 of the sequence);
//   * a bias per (head, distance) added to the scaled score: bias[h][min(i - j, rows - 1)], a table
//     the host expands from whatever rule the model has (buckets, slopes ...);
//   * a cap on the scaled score, c tanh(s / c);
//   * a sink: one more term in the softmax's denominator that carries no value, e^0 or e^(a learned
//     number of the head);
//   * values that were rotated by their position when they were cached: each head's output is turned
//     back by the row's position, pair by pair (e with e + E / 2), before the gate;
//   * a gate: the output of head h, element e, times sigmoid(gate[t][h * E + e]).
//
// head_norm_write: per token, the projection's bias, an RMS norm over each head's D query or key
//   elements with one gain vector shared by the heads (float32 throughout), optionally a factor per
//   query head (a learned temperature), a rotation of the first rot_dims dimensions of queries and
//   keys and one of whole values (halves paired: i with i + half), queries out in float32, keys and
//   values into the pages.  The angle's fraction of a turn is formed from the frequency as two
//   float32 numbers and the exact remainder of the product, so it is good to a few 1e-8 of a turn at
//   any position.  cos and sin of the values' angles are left in a table for the attention's epilogue.
// head_conv_norm_write: the same behind a short causal convolution on every channel of queries, keys and values
//   (taps inputs per channel: the projection's rows of this step, before them the request's state row).  A warp
//   a head of a token, V neighbouring channels a lane.  A request that brings one token has its convolution
//   state moved on in the same launch: each channel is read and written by one thread only.
// masked_attention: the float32-arithmetic kernel.  It reads the engine's attention work list
//   (request, row tile, key split, splits): the rows of a request are packed with the query heads
//   that share a key/value head, 16 packed rows a block, 32 keys a tile (a key a lane), online
//   softmax.  Scores, maxima, sums and weights are float32; queries are float32, keys and values
//   what the cache holds.
// masked_merge: the key splits of a row put together, with the sink and the gate.
#include "attention_params.cuh"
#include "common.cuh"
#include "masked_attention.cuh"
#include "pdl.cuh"
#include "vec.cuh"

using namespace pbe;

namespace {

// ------------------------------------------------------------------ head_norm_write
struct HeadNormParams {
  const void* proj;          // [T, ld]: queries at column q_off, keys at k_off, values at v_off
  int ld, q_off, k_off, v_off;
  const float* bias;         // indexed like the projection's columns, or null
  const float* q_gain;       // [D] or null: no norm
  const float* k_gain;       // [D] or null
  const float* q_head_scale; // [H] or null: head h's normed query is multiplied by it (a temperature per head)
  const int32_t* slots;      // [T] page * page_tokens + offset; negative: nothing is written
  float* q_out;              // [T, H * D]
  void* k_pages;             // [page][G][page_tokens][D] or null
  void* v_pages;             // [page][G][page_tokens][E]
  int H, G, D, E, page_tokens;
  float eps;
  const int32_t* positions;  // [T], read when something turns
  const float2* rot_freq;    // [rot_dims / 2] turns a position as (rounded, rest), or null: no rotation of q and k
  int rot_dims;
  const float2* v_freq;      // [E / 2] the same for values, or null
  float2* v_turn;            // [T, E / 2] (cos, sin) of the values' angles, written when v_freq is given
};

// (cos, sin) of 2 pi * position * freq
__device__ __forceinline__ float2 turn_of(int position, float2 freq) {
  const float p = (float)position;               // exact up to 2^24
  const float whole = rintf(p * freq.x);
  const float rest = fmaf(p, freq.x, -whole) + p * freq.y;
  float2 cs;
  sincospif(2.0f * rest, &cs.y, &cs.x);
  return cs;
}

constexpr int HN_MAX = 8;    // elements of a head a lane holds at most (D <= 256)

template <typename T, bool TURN>
__global__ void __launch_bounds__(128) head_norm_write_kernel(HeadNormParams p) {
  __shared__ float2 rot_cs[TURN ? 16 * HN_MAX : 1], v_cs[TURN ? 16 * HN_MAX : 1];   // heads are at most 256 wide
  __shared__ float held[TURN ? 4 : 1][TURN ? 32 * HN_MAX : 1];     // a warp's head between the norm and the turn
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  if (TURN) {
    const int half = p.rot_freq ? p.rot_dims / 2 : 0, vhalf = p.v_freq ? p.E / 2 : 0;
    const int pos = p.positions[t];
    for (int i = threadIdx.x; i < half + vhalf; i += blockDim.x) {
      if (i < half) {
        rot_cs[i] = turn_of(pos, p.rot_freq[i]);
      } else {
        const float2 cs = turn_of(pos, p.v_freq[i - half]);
        v_cs[i - half] = cs;
        p.v_turn[(size_t)t * vhalf + i - half] = cs;
      }
    }
    __syncthreads();
  }
  const int H = p.H, G = p.G, D = p.D, E = p.E, PT = p.page_tokens;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* row = (const T*)p.proj + (size_t)t * p.ld;
  const int slot = p.slots ? p.slots[t] : -1;
  const bool store = slot >= 0 && p.k_pages != nullptr;
  const int page = store ? slot / PT : 0, off = store ? slot - page * PT : 0;
  for (int hh = warp; hh < H + G; hh += 4) {
    const bool is_q = hh < H;
    const int head = is_q ? hh : hh - H;
    if (!is_q && !store) continue;
    const int col = (is_q ? p.q_off : p.k_off) + head * D;
    const float* gain = is_q ? p.q_gain : p.k_gain;
    float x[HN_MAX];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < HN_MAX; ++i) {
      const int d = lane + i * 32;
      x[i] = 0.f;
      if (d < D) {
        x[i] = to_float(row[col + d]) + (p.bias ? p.bias[col + d] : 0.f);
        ss = fmaf(x[i], x[i], ss);
      }
    }
    float sc = 1.f;
    if (gain) sc = 1.0f / sqrtf(warp_sum(ss) / (float)D + p.eps);
    const int half = (TURN && p.rot_freq) ? p.rot_dims / 2 : 0;
    if (half) {
      __syncwarp();                            // the warp's head before is read
#pragma unroll
      for (int i = 0; i < HN_MAX; ++i) {
        const int d = lane + i * 32;
        if (d < D) {
          x[i] = gain ? (x[i] * sc) * gain[d] : x[i];
          if (d < 2 * half) held[TURN ? warp : 0][TURN ? d : 0] = x[i];
        }
      }
      __syncwarp();
    }
#pragma unroll
    for (int i = 0; i < HN_MAX; ++i) {
      const int d = lane + i * 32;
      if (d < D) {
        float y = (gain && !half) ? (x[i] * sc) * gain[d] : x[i];
        if (d < 2 * half) {
          const bool first = d < half;
          const float other = held[TURN ? warp : 0][TURN ? (first ? d + half : d - half) : 0];
          const float2 cs = rot_cs[TURN ? (first ? d : d - half) : 0];
          y = first ? y * cs.x - other * cs.y : y * cs.x + other * cs.y;
        }
        if (is_q && p.q_head_scale) y *= p.q_head_scale[head];
        if (is_q) p.q_out[((size_t)t * H + head) * D + d] = y;
        else ((T*)p.k_pages)[(((size_t)page * G + head) * PT + off) * D + d] = from_float<T>(y);
      }
    }
  }
  if (TURN && store && p.v_pages && p.v_freq) {
    const int vhalf = E / 2;
    for (int i = threadIdx.x; i < G * vhalf; i += blockDim.x) {
      const int head = i / vhalf, m = i - head * vhalf, c = p.v_off + head * E + m;
      float u = to_float(row[c]), v = to_float(row[c + vhalf]);
      if (p.bias) {
        u += p.bias[c];
        v += p.bias[c + vhalf];
      }
      const float2 cs = v_cs[m];
      T* dst = (T*)p.v_pages + (((size_t)page * G + head) * PT + off) * E + m;
      dst[0] = from_float<T>(u * cs.x - v * cs.y);
      dst[vhalf] = from_float<T>(v * cs.x + u * cs.y);
    }
  } else if (store && p.v_pages) {
    for (int i = threadIdx.x; i < G * E; i += blockDim.x) {
      const int head = i / E, e = i - head * E;
      const float y = to_float(row[p.v_off + i]) + (p.bias ? p.bias[p.v_off + i] : 0.f);
      ((T*)p.v_pages)[(((size_t)page * G + head) * PT + off) * E + e] = from_float<T>(y);
    }
  }
}

// ------------------------------------------------------------------ head_conv_norm_write
struct HeadConvParams {
  HeadNormParams b;          // what head_norm_write reads (columns from 0: queries, keys, values side by side; no
                             // bias, no factor per head, no rotation of values)
  const float* conv_t;       // [taps, C], C = H D + G D + G E; the last tap is the current token's
  float* conv_state;         // [slots, taps - 1, C], the newest input last
  const int32_t* request_of_row;
  const int32_t* q_start;
  const int32_t* q_len;
  const int32_t* state_slots;
  int R, taps, update;
};

constexpr int HC_WARPS = 4;

// The convolution of V neighbouring channels from column c of one token.
template <typename T, int V>
__device__ __forceinline__ void conv_at(const HeadConvParams& p, int t, int i, const float* st_in, float* st_out, int C,
                                        int c, float (&acc)[V]) {
#pragma unroll
  for (int k = 0; k < V; ++k) acc[k] = 0.f;
  const int taps = p.taps;
  const T* in = (const T*)p.b.proj + c;
#pragma unroll 4
  for (int j = 0; j < taps; ++j) {
    const int off = i - (taps - 1) + j;          // the input's place among this step's rows; negative: before them
    float u[V], w[V];
    if (off >= 0) load_v<V>(in + (size_t)(t - (taps - 1) + j) * p.b.ld, u);
    else load_v<V>(st_in + (size_t)(taps - 1 + off) * C + c, u);
    load_v<V>(p.conv_t + (size_t)j * C + c, w);
#pragma unroll
    for (int k = 0; k < V; ++k) acc[k] = fmaf(w[k], u[k], acc[k]);
    if (st_out && j > 0) put_v<V>(st_out + (size_t)(j - 1) * C + c, u);     // entry j - 1 was read the turn before
  }
}

// grid (rows, groups of heads_here heads): queries, keys, then values.  N: groups of 32 V channels a head has at most.
template <typename T, int V, int N>
__global__ void __launch_bounds__(HC_WARPS * 32) head_conv_norm_write_kernel(HeadConvParams p, int heads_here) {
  __shared__ float2 rot_cs[16 * HN_MAX];
  __shared__ __align__(16) float held[HC_WARPS][32 * HN_MAX];      // a warp's head between the norm and the turn
  pdl_launch_dependents();
  pdl_wait();
  const HeadNormParams& b = p.b;
  const int t = blockIdx.x;
  const int H = b.H, G = b.G, D = b.D, E = b.E, PT = b.page_tokens;
  const int C = (H + G) * D + G * E;
  const int r = p.request_of_row[t];
  const bool live = r >= 0 && r < p.R && p.q_len[r] > 0;        // not a padding row of a captured step
  const int half = b.rot_freq ? b.rot_dims / 2 : 0;
  if (half) {
    const int pos = b.positions[t];
    for (int i = threadIdx.x; i < half; i += blockDim.x) rot_cs[i] = turn_of(pos, b.rot_freq[i]);
    __syncthreads();
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int slot = (live && b.slots) ? b.slots[t] : -1;
  const bool store = slot >= 0 && b.k_pages != nullptr;
  const int page = store ? slot / PT : 0, off = store ? slot - page * PT : 0;
  const int i = live ? t - p.q_start[r] : 0;
  float* st = live && p.taps > 1 ? p.conv_state + (size_t)p.state_slots[r] * (p.taps - 1) * C : nullptr;
  float* st_out = (live && p.update && p.q_len[r] == 1) ? st : nullptr;
  const int first = blockIdx.y * heads_here, last = min(H + 2 * G, first + heads_here);
  for (int hh = first + warp; hh < last; hh += HC_WARPS) {
    if (hh >= H + G) {                         // a value head
      const int head = hh - H - G;
      if (!store && !st_out) continue;
#pragma unroll
      for (int n = 0; n < N; ++n) {
        const int e = (n * 32 + lane) * V;
        if (e < E && live) {
          float v[V];
          conv_at<T, V>(p, t, i, st, st_out, C, (H + G) * D + head * E + e, v);
          if (store) put_v<V>((T*)b.v_pages + (((size_t)page * G + head) * PT + off) * E + e, v);
        }
      }
      continue;
    }
    const bool is_q = hh < H;
    const int head = is_q ? hh : hh - H;
    if (!is_q && !store && !st_out) continue;
    const float* gain = is_q ? b.q_gain : b.k_gain;
    float x[N][V];
    float ss = 0.f;
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int d = (n * 32 + lane) * V;
#pragma unroll
      for (int k = 0; k < V; ++k) x[n][k] = 0.f;
      if (d < D && live) conv_at<T, V>(p, t, i, st, st_out, C, hh * D + d, x[n]);
#pragma unroll
      for (int k = 0; k < V; ++k) ss = fmaf(x[n][k], x[n][k], ss);
    }
    const float sc = gain ? 1.0f / sqrtf(warp_sum(ss) / (float)D + b.eps) : 1.f;
    __syncwarp();                              // the warp's head before is read
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int d = (n * 32 + lane) * V;
      if (d < D) {
        if (gain) {
          float g[V];
          load_v<V>(gain + d, g);
#pragma unroll
          for (int k = 0; k < V; ++k) x[n][k] = (x[n][k] * sc) * g[k];
        }
        if (d < 2 * half) put_v<V>(&held[warp][d], x[n]);
      }
    }
    __syncwarp();
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int d = (n * 32 + lane) * V;
      if (d >= D) continue;
#pragma unroll
      for (int k = 0; k < V; ++k) {
        const int dd = d + k;
        if (dd < 2 * half) {
          const bool lower = dd < half;
          const float other = held[warp][lower ? dd + half : dd - half];
          const float2 cs = rot_cs[lower ? dd : dd - half];
          x[n][k] = lower ? x[n][k] * cs.x - other * cs.y : x[n][k] * cs.x + other * cs.y;
        }
      }
      if (is_q) put_v<V>(b.q_out + ((size_t)t * H + head) * D + d, x[n]);
      else if (store) put_v<V>((T*)b.k_pages + (((size_t)page * G + head) * PT + off) * D + d, x[n]);
    }
  }
}

template <typename T, int V>
int launch_head_conv(const HeadConvParams& p, int T_rows, cudaStream_t stream) {
  const int wide = p.b.D > p.b.E ? p.b.D : p.b.E, heads = p.b.H + 2 * p.b.G;
  // few rows: a block per group of four heads; many: a block keeps its row's angles for all heads
  const int here = T_rows >= 512 ? heads : HC_WARPS;
  dim3 grid(T_rows, (heads + here - 1) / here);
  const int per = (wide + 32 * V - 1) / (32 * V);
  if (per <= 1) launch_k(head_conv_norm_write_kernel<T, V, 1>, grid, HC_WARPS * 32, 0, stream, p, here);
  else if (per <= 2) launch_k(head_conv_norm_write_kernel<T, V, 2>, grid, HC_WARPS * 32, 0, stream, p, here);
  else if (per <= 8 / V) launch_k(head_conv_norm_write_kernel<T, V, 8 / V>, grid, HC_WARPS * 32, 0, stream, p, here);
  else return (int)cudaErrorInvalidValue;
  return launch_status();
}

// ------------------------------------------------------------------ masked_attention
constexpr int BM = 16;       // packed rows per block
constexpr int BN = 32;       // keys per tile, one per lane
constexpr int NWARPS = 4;
constexpr int ROWS_PER_WARP = BM / NWARPS;

template <typename T, int EPL>
__global__ void __launch_bounds__(NWARPS * 32) masked_attention_kernel(AttnParams p, MaskedExtra x) {
  extern __shared__ __align__(16) float smem[];
  const int D = x.D, E = x.E;
  const int QS = (D + 3) & ~3;            // query rows start on 16-byte boundaries
  const int KS = D + 1;
  float* Qs = smem;                       // [BM][QS]
  float* Ks = Qs + BM * QS;               // [BN][D + 1]
  float* Vs = Ks + BN * KS;               // [BN][E]
  __shared__ long long base[BN];          // (page * G + kv head) * page_tokens + offset of key j, -1: none

  pdl_launch_dependents();
  pdl_wait();
  const int32_t* work = p.work + (size_t)blockIdx.x * 4;
  const int r = work[0];
  if (r < 0) return;
  const int m_tile = work[1], split = work[2], nsplit = work[3];
  const int kvh = blockIdx.y;
  const int H = p.num_heads, KV = p.num_kv_heads, G = H / KV, P = p.page_tokens;
  const int qs = p.q_start[r], nq = p.q_len[r], sl = p.seq_len[r];
  const int n_packed = nq * G;
  const int pr0 = m_tile * BM;
  if (pr0 >= n_packed) return;
  const int row_lo = pr0 / G;
  const int row_hi = (min(n_packed, pr0 + BM) - 1) / G;
  const int pos0 = sl - nq;
  const int hi_key = pos0 + row_hi + 1;
  const int lo_key = first_visible(pos0 + row_lo, x.mask_kind, p.window);
  int k_begin = lo_key, k_end = hi_key;
  if (nsplit > 1) {
    // split boundaries are absolute multiples of split_keys, counted from the first split that a
    // window of this size at the request's first row can reach: the work list's own rule
    const int lo_req = x.mask_kind ? max(0, pos0 - p.window + 1) : 0;
    const int s0 = lo_req / p.split_keys;
    k_begin = max(lo_key, (s0 + split) * p.split_keys);
    k_end = min(hi_key, (s0 + split + 1) * p.split_keys);
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float* q = (const float*)p.q;
  const T* kc = (const T*)p.k_cache;
  const T* vc = (const T*)p.v_cache;
  const int32_t* bt = p.block_table + (size_t)r * p.bt_stride;

  for (int idx = threadIdx.x; idx < BM * D; idx += blockDim.x) {
    const int i = idx / D, d = idx - i * D;
    const int pr = pr0 + i;
    float v = 0.f;
    if (pr < n_packed) {
      const int row = pr / G, hg = pr - row * G;
      v = q[((size_t)(qs + row) * H + kvh * G + hg) * D + d];
    }
    Qs[i * QS + d] = v;
  }

  float m_run[ROWS_PER_WARP], l_run[ROWS_PER_WARP], acc[ROWS_PER_WARP][EPL];
#pragma unroll
  for (int j = 0; j < ROWS_PER_WARP; ++j) {
    m_run[j] = -INFINITY;
    l_run[j] = 0.f;
#pragma unroll
    for (int i = 0; i < EPL; ++i) acc[j][i] = 0.f;
  }
  // this warp's rows: position and head (fixed for the block)
  int row_pos[ROWS_PER_WARP], row_head[ROWS_PER_WARP];
#pragma unroll
  for (int j = 0; j < ROWS_PER_WARP; ++j) {
    const int pr = pr0 + warp + j * NWARPS;
    row_pos[j] = pr < n_packed ? pos0 + pr / G : -1;
    row_head[j] = kvh * G + (pr < n_packed ? pr % G : 0);
  }

  const int tile0 = (k_begin / BN) * BN;
  for (int ts = tile0; ts < k_end; ts += BN) {
    __syncthreads();   // the tile before is consumed (and Qs written, first time)
    if (threadIdx.x < BN) {
      const int key = ts + threadIdx.x;
      long long b = -1;
      if (key >= k_begin && key < k_end) {
        const int page = bt[key / P];
        if (page >= 0) b = ((long long)page * KV + kvh) * P + key % P;
      }
      base[threadIdx.x] = b;
    }
    __syncthreads();
    // keys and values of the tile as float32: four elements a thread and turn where the widths allow
    if ((D & 3) == 0) {
      const int dq = D >> 2;
      for (int i = threadIdx.x; i < BN * dq; i += blockDim.x) {
        const int j = i / dq, d = (i - j * dq) * 4;
        const long long b = base[j];
        float f[4] = {0.f, 0.f, 0.f, 0.f};
        if (b >= 0) {
#pragma unroll
          for (int u = 0; u < 4; ++u) f[u] = to_float(kc[b * D + d + u]);
        }
        float* kd = Ks + j * KS + d;
        kd[0] = f[0]; kd[1] = f[1]; kd[2] = f[2]; kd[3] = f[3];
      }
    } else {
      for (int i = threadIdx.x; i < BN * D; i += blockDim.x) {
        const int j = i / D, d = i - j * D;
        const long long b = base[j];
        Ks[j * KS + d] = b >= 0 ? to_float(kc[b * D + d]) : 0.f;
      }
    }
    for (int i = threadIdx.x; i < BN * E; i += blockDim.x) {
      const int j = i / E, e = i - j * E;
      const long long b = base[j];
      Vs[i] = b >= 0 ? to_float(vc[b * E + e]) : 0.f;
    }
    __syncthreads();
    float s[ROWS_PER_WARP];
#pragma unroll
    for (int j = 0; j < ROWS_PER_WARP; ++j) s[j] = 0.f;
    {
      const float* krow = Ks + lane * KS;
      int d = 0;
      for (; d + 3 < D; d += 4) {
        const float k0 = krow[d], k1 = krow[d + 1], k2 = krow[d + 2], k3 = krow[d + 3];
#pragma unroll
        for (int j = 0; j < ROWS_PER_WARP; ++j) {
          const float4 qv = *reinterpret_cast<const float4*>(Qs + (warp + j * NWARPS) * QS + d);
          float a = s[j];
          a = fmaf(qv.x, k0, a);
          a = fmaf(qv.y, k1, a);
          a = fmaf(qv.z, k2, a);
          a = fmaf(qv.w, k3, a);
          s[j] = a;
        }
      }
      for (; d < D; ++d) {
        const float k0 = krow[d];
#pragma unroll
        for (int j = 0; j < ROWS_PER_WARP; ++j) s[j] = fmaf(Qs[(warp + j * NWARPS) * QS + d], k0, s[j]);
      }
    }
    float pj[ROWS_PER_WARP];
    const int key = ts + lane;
    const bool have = base[lane] >= 0;
#pragma unroll
    for (int j = 0; j < ROWS_PER_WARP; ++j) {
      pj[j] = 0.f;
      const int pos = row_pos[j];
      if (pos < 0) continue;
      const bool visible = have && key <= pos && key >= first_visible(pos, x.mask_kind, p.window);
      float sc = -INFINITY;
      if (visible) {
        sc = s[j] * p.scale;
        if (x.softcap > 0.f) sc = x.softcap * tanhf(sc / x.softcap);
        if (x.bias) sc += __ldg(x.bias + (size_t)row_head[j] * x.bias_rows + min(pos - key, x.bias_rows - 1));
      }
      const float m_new = fmaxf(m_run[j], warp_max(sc));
      if (m_new == -INFINITY) continue;     // nothing visible so far
      pj[j] = visible ? expf(sc - m_new) : 0.f;
      const float alpha = expf(m_run[j] - m_new);
      l_run[j] = l_run[j] * alpha + warp_sum(pj[j]);
      m_run[j] = m_new;
#pragma unroll
      for (int ii = 0; ii < EPL; ++ii) acc[j][ii] *= alpha;
    }
    for (int kk = 0; kk < BN; ++kk) {
      float vv[EPL];
#pragma unroll
      for (int ii = 0; ii < EPL; ++ii) {
        const int e = lane + ii * 32;
        vv[ii] = e < E ? Vs[kk * E + e] : 0.f;
      }
#pragma unroll
      for (int j = 0; j < ROWS_PER_WARP; ++j) {
        const float pk = __shfl_sync(0xffffffffu, pj[j], kk);
#pragma unroll
        for (int ii = 0; ii < EPL; ++ii) acc[j][ii] = fmaf(pk, vv[ii], acc[j][ii]);
      }
    }
  }

  if (x.turn) __syncthreads();     // the values are read: their place holds a row of outputs a warp while it turns
#pragma unroll
  for (int j = 0; j < ROWS_PER_WARP; ++j) {
    const int pr = pr0 + warp + j * NWARPS;
    if (pr >= n_packed) continue;
    const int row = pr / G;
    const int head = row_head[j];
    const int t = qs + row;
    if (nsplit <= 1) {
      float m = m_run[j], l = l_run[j], rescale = 1.f;
      if (x.has_sink) add_sink(m, l, rescale, x.sink ? x.sink[head] : 0.f);
      const float inv = l > 0.f ? rescale / l : 0.f;
      T* o = (T*)p.out + ((size_t)t * H + head) * E;
      const T* g = x.gate ? (const T*)x.gate + (size_t)t * x.ldg + head * E : nullptr;
      float* held = Vs + warp * E;
      const int half = E / 2;
      if (x.turn) {
        __syncwarp();
#pragma unroll
        for (int ii = 0; ii < EPL; ++ii) {
          const int e = lane + ii * 32;
          if (e < E) held[e] = acc[j][ii] * inv;
        }
        __syncwarp();
      }
#pragma unroll
      for (int ii = 0; ii < EPL; ++ii) {
        const int e = lane + ii * 32;
        if (e < E) {
          float y = acc[j][ii] * inv;
          if (x.turn) {
            const bool first = e < half;
            const float2 cs = x.turn[(size_t)t * half + (first ? e : e - half)];
            const float other = held[first ? e + half : e - half];
            y = first ? y * cs.x + other * cs.y : y * cs.x - other * cs.y;
          }
          if (g) y *= sigmoidf_(to_float(g[e]));
          o[e] = from_float<T>(y);
        }
      }
    } else {
      const int srow = p.tok_split_row[t];
      const size_t b = ((size_t)srow * H + head) * p.max_splits + split;
      float* po = p.part_o + b * E;
#pragma unroll
      for (int ii = 0; ii < EPL; ++ii) {
        const int e = lane + ii * 32;
        if (e < E) po[e] = acc[j][ii];
      }
      if (lane == 0) {
        p.part_ml[b * 2] = m_run[j];
        p.part_ml[b * 2 + 1] = l_run[j];
      }
    }
  }
}

struct MaskedMergeExtra {
  int has_sink;
  const float* sink;
  const float2* turn;
  const void* gate;
  int ldg;
};

template <typename T>
__global__ void masked_merge_kernel(AttnMergeParams p, MaskedMergeExtra x) {
  pdl_launch_dependents();
  pdl_wait();
  const int srow = blockIdx.x, head = blockIdx.y;
  const int n = p.split_counts[srow];
  if (n <= 1) return;
  const int t = p.split_tokens[srow];
  const int E = p.head_dim;
  const size_t base = ((size_t)srow * p.num_heads + head) * p.max_splits;
  float m = -INFINITY;
  for (int s = 0; s < n; ++s) m = fmaxf(m, p.part_ml[(base + s) * 2]);
  const float s_sink = (x.has_sink && x.sink) ? x.sink[head] : 0.f;
  if (x.has_sink) m = fmaxf(m, s_sink);
  float l = x.has_sink ? expf(s_sink - m) : 0.f;
  for (int s = 0; s < n; ++s) {
    const float ms = p.part_ml[(base + s) * 2];
    if (ms != -INFINITY) l += p.part_ml[(base + s) * 2 + 1] * expf(ms - m);
  }
  const float inv = l > 0.f ? 1.0f / l : 0.f;
  T* o = (T*)p.out + ((size_t)t * p.num_heads + head) * E;
  const T* g = x.gate ? (const T*)x.gate + (size_t)t * x.ldg + head * E : nullptr;
  auto sum_at = [&](int e) {
    float a = 0.f;
    for (int s = 0; s < n; ++s) {
      const float ms = p.part_ml[(base + s) * 2];
      if (ms != -INFINITY) a += p.part_o[(base + s) * E + e] * expf(ms - m);
    }
    return a * inv;
  };
  if (x.turn) {
    const int half = E / 2;
    for (int e = threadIdx.x; e < half; e += blockDim.x) {
      float u = sum_at(e), v = sum_at(e + half);
      turn_back(u, v, x.turn[(size_t)t * half + e]);
      if (g) {
        u *= sigmoidf_(to_float(g[e]));
        v *= sigmoidf_(to_float(g[e + half]));
      }
      o[e] = from_float<T>(u);
      o[e + half] = from_float<T>(v);
    }
    return;
  }
  for (int e = threadIdx.x; e < E; e += blockDim.x) {
    float y = sum_at(e);
    if (g) y *= sigmoidf_(to_float(g[e]));
    o[e] = from_float<T>(y);
  }
}

size_t ma_smem(int D, int E) {
  return sizeof(float) * ((size_t)BM * ((D + 3) & ~3) + (size_t)BN * (D + 1) + (size_t)BN * E);
}

template <typename T, int EPL>
int launch_ma(const AttnParams& p, const MaskedExtra& x, int num_work, cudaStream_t stream) {
  const size_t smem = ma_smem(x.D, x.E);
  static size_t opted = 48 * 1024;
  if (smem > opted) {
    cudaFuncSetAttribute(masked_attention_kernel<T, EPL>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    opted = 200 * 1024;
  }
  launch_k(masked_attention_kernel<T, EPL>, dim3(num_work, p.num_kv_heads), NWARPS * 32, smem, stream, p, x);
  return launch_status();
}

template <typename T>
int dispatch_ma(const AttnParams& p, const MaskedExtra& x, int num_work, cudaStream_t stream) {
  const int epl = (x.E + 31) / 32;
  if (epl <= 1) return launch_ma<T, 1>(p, x, num_work, stream);
  if (epl <= 2) return launch_ma<T, 2>(p, x, num_work, stream);
  if (epl <= 4) return launch_ma<T, 4>(p, x, num_work, stream);
  return launch_ma<T, 8>(p, x, num_work, stream);
}
}  // namespace

PBE_EXPORT int pbe_masked_attention_tile_rows() { return BM; }
PBE_EXPORT int pbe_masked_attention_key_tile() { return BN; }

PBE_EXPORT int pbe_head_norm_write(const void* proj, int ld, int q_off, int k_off, int v_off, const float* bias,
                                   const float* q_gain, const float* k_gain, const float* q_head_scale,
                                   const int32_t* slots, float* q_out,
                                   void* k_pages, void* v_pages, int T, int H, int G, int D, int E, int page_tokens,
                                   float eps, const int32_t* positions, const float2* rot_freq, int rot_dims,
                                   const float2* v_freq, float2* v_turn, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (D > 32 * HN_MAX || D < 1 || E < 1) return (int)cudaErrorInvalidValue;
  const bool turns = rot_freq != nullptr || v_freq != nullptr;
  if (turns && positions == nullptr) return (int)cudaErrorInvalidValue;
  if (rot_freq && (rot_dims < 2 || (rot_dims & 1) || rot_dims > D)) return (int)cudaErrorInvalidValue;
  if (v_freq && (v_turn == nullptr || (E & 1) || E > 32 * HN_MAX)) return (int)cudaErrorInvalidValue;
  HeadNormParams p{proj, ld, q_off, k_off, v_off, bias, q_gain, k_gain, q_head_scale, slots, q_out, k_pages, v_pages,
                   H, G, D, E, page_tokens, eps, positions, rot_freq, rot_dims, v_freq, v_turn};
  if (dtype == PBE_F32) {
    if (turns) launch_k(head_norm_write_kernel<float, true>, T, 128, 0, stream, p);
    else launch_k(head_norm_write_kernel<float, false>, T, 128, 0, stream, p);
  } else {
    if (turns) launch_k(head_norm_write_kernel<__nv_bfloat16, true>, T, 128, 0, stream, p);
    else launch_k(head_norm_write_kernel<__nv_bfloat16, false>, T, 128, 0, stream, p);
  }
  return launch_status();
}

PBE_EXPORT int pbe_head_conv_norm_write(const void* proj, int ld, const float* conv_t, float* conv_state,
                                        const float* q_gain, const float* k_gain, const int32_t* slots, float* q_out,
                                        void* k_pages, void* v_pages, int T, int R, int H, int G, int D, int E,
                                        int page_tokens, float eps, const int32_t* positions, const float2* rot_freq,
                                        int rot_dims, int taps, int update, const int32_t* request_of_row,
                                        const int32_t* q_start, const int32_t* q_len, const int32_t* state_slots,
                                        int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (D > 32 * HN_MAX || E > 32 * HN_MAX || D < 1 || E < 1 || taps < 1 || taps > 16) return (int)cudaErrorInvalidValue;
  if (rot_freq && (positions == nullptr || rot_dims < 2 || (rot_dims & 1) || rot_dims > D)) return (int)cudaErrorInvalidValue;
  HeadConvParams p{};
  p.b = HeadNormParams{proj, ld, 0, H * D, (H + G) * D, nullptr, q_gain, k_gain, nullptr, slots, q_out, k_pages,
                       v_pages, H, G, D, E, page_tokens, eps, positions, rot_freq, rot_dims, nullptr, nullptr};
  p.conv_t = conv_t;
  p.conv_state = conv_state;
  p.request_of_row = request_of_row;
  p.q_start = q_start;
  p.q_len = q_len;
  p.state_slots = state_slots;
  p.R = R;
  p.taps = taps;
  p.update = update;
  const bool f32 = dtype == PBE_F32;
  const bool vec4 = D % 4 == 0 && E % 4 == 0 && ld % 4 == 0 &&
                    (((uintptr_t)conv_t | (uintptr_t)conv_state | (uintptr_t)q_out | (uintptr_t)q_gain | (uintptr_t)k_gain) & 15) == 0 &&
                    (((uintptr_t)proj | (uintptr_t)k_pages | (uintptr_t)v_pages) & (f32 ? 15 : 7)) == 0;
  if (f32) return vec4 ? launch_head_conv<float, 4>(p, T, stream) : launch_head_conv<float, 1>(p, T, stream);
  return vec4 ? launch_head_conv<__nv_bfloat16, 4>(p, T, stream) : launch_head_conv<__nv_bfloat16, 1>(p, T, stream);
}

PBE_EXPORT int pbe_masked_attention(const AttnParams* params, int D, int E, const float* bias, int bias_rows,
                                    int mask_kind, int has_sink, const float* sink, float softcap,
                                    const float2* turn, const void* gate, int ldg, int num_work, int dtype,
                                    cudaStream_t stream) {
  if (num_work <= 0) return 0;
  AttnParams p = *params;
  if (p.num_heads % p.num_kv_heads != 0 || p.tile_rows != BM || p.split_keys % BN != 0 || D < 1 || E < 1 ||
      E > 256 || (turn && (E & 1)) || mask_kind < 0 || mask_kind > 2 || (mask_kind != 0 && p.window < 1) || (bias && bias_rows < 1))
    return (int)cudaErrorInvalidValue;
  if (ma_smem(D, E) > 200 * 1024) return (int)cudaErrorInvalidValue;
  MaskedExtra x{bias, bias_rows, mask_kind, has_sink, sink, softcap, turn, gate, ldg, D, E};
  return dtype == PBE_F32 ? dispatch_ma<float>(p, x, num_work, stream)
                          : dispatch_ma<__nv_bfloat16>(p, x, num_work, stream);
}

PBE_EXPORT int pbe_masked_merge(const AttnMergeParams* params, int has_sink, const float* sink, const float2* turn,
                                const void* gate, int ldg, int split_rows, int dtype, cudaStream_t stream) {
  if (split_rows <= 0) return 0;
  AttnMergeParams p = *params;
  MaskedMergeExtra x{has_sink, sink, turn, gate, ldg};
  dim3 grid(split_rows, p.num_heads);
  const int threads = p.head_dim > 64 ? 128 : 64;
  if (dtype == PBE_F32) launch_k(masked_merge_kernel<float>, grid, threads, 0, stream, p, x);
  else launch_k(masked_merge_kernel<__nv_bfloat16>, grid, threads, 0, stream, p, x);
  return launch_status();
}
