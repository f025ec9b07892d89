// The selective scan: a recurrence whose step size, input and output vectors depend on the token.
//
//   conv_act_kernel           causal convolution per channel with bias and activation, rows in the compute
//                             dtype, and the last taps - 1 inputs of every sequence into its state
//   selective_scan_kernel     S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n,
//                             y_c = (sum_n S[c, n] C_n + D_c x_c) * silu(z_c)
//   selective_combine_kernel  the states that chunks of a long portion start from
//   selective_step_kernel     one token of every sequence in one launch, the step size's second small
//                             matrix included
//
// dt, decays, S and the sums over S are float32 whatever the storage type.  A sequence is rows q_start[s]
// .. q_start[s] + q_len[s] - 1 of the step, its state row seq_slots[s].  Every sum has an order that depends
// on the sizes only.
#include "common.cuh"
#include "recurrent.cuh"

namespace vx {

// Sixteen bytes of a row as floats, or one value.
template <typename T, int V>
struct RowVec;
template <>
struct RowVec<float, 4> {
  float4 raw;
  __device__ __forceinline__ void load(const float* p) { raw = *reinterpret_cast<const float4*>(p); }
  __device__ __forceinline__ void get(float (&v)[4]) const { v[0] = raw.x, v[1] = raw.y, v[2] = raw.z, v[3] = raw.w; }
  static __device__ __forceinline__ void store(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  }
};
template <>
struct RowVec<__nv_bfloat16, 8> {
  uint4 raw;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { raw = *reinterpret_cast<const uint4*>(p); }
  __device__ __forceinline__ void get(float (&v)[8]) const {
    const uint32_t w[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      v[2 * i] = __uint_as_float(w[i] << 16);
      v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[8]) {
    uint32_t w[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const __nv_bfloat162 h = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
      w[i] = *reinterpret_cast<const uint32_t*>(&h);
    }
    *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
  }
};
template <typename T>
struct RowVec<T, 1> {
  T raw;
  __device__ __forceinline__ void load(const T* p) { raw = *p; }
  __device__ __forceinline__ void get(float (&v)[1]) const { v[0] = to_float(raw); }
  static __device__ __forceinline__ void store(T* p, const float (&v)[1]) { *p = from_float<T>(v[0]); }
};

// ---------------------------------------------------------------------------------------------
// out_t = act(bias + sum_k w[k] x_(t - taps + 1 + k)) per channel.  state[slot][m][c], m = 0 .. taps - 2, is the
// input taps - 1 - m positions before the portion's first token (zero before the sequence's start).  w_t
// [taps][channels].  A thread takes V channels of a tile of CA_TILE tokens; only the first tile of a
// portion reads the state (CA_TILE >= taps - 1, or one tile holds the portion), and the same thread then
// writes the state that the portion leaves.
constexpr int CA_TILE = 8;

template <typename T, int V, int TAPS>
__global__ void __launch_bounds__(128)
conv_act_kernel(const T* __restrict__ x, long long x_stride, int channels, int taps, const float* __restrict__ w_t,
                const float* __restrict__ bias, float* __restrict__ state, long long state_stride, T* __restrict__ out,
                long long out_stride, const int* __restrict__ q_start, const int* __restrict__ q_len,
                const int* __restrict__ seq_slots, int tile, int act) {
  allow_dependents();
  const int c0 = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (c0 >= channels) return;
  float b[V];
#pragma unroll
  for (int v = 0; v < V; ++v) b[v] = bias[c0 + v];
  grid_dependency_wait();
  const int s = blockIdx.z, n = q_len[s], lo = blockIdx.y * tile;
  if (lo >= n) return;
  const int hi = min(n, lo + tile), start = q_start[s];
  float* st = state + (size_t)seq_slots[s] * state_stride + c0;
  const T* xc = x + (size_t)start * x_stride + c0;
  T* oc = out + (size_t)start * out_stride + c0;
  if constexpr (TAPS > 0) {
    // Up to TAPS taps, the window in registers.
    float w[TAPS][V], win[TAPS - 1][V];
#pragma unroll
    for (int k = 0; k < TAPS; ++k) {
      const int at = taps - TAPS + k;
#pragma unroll
      for (int v = 0; v < V; ++v) w[k][v] = at >= 0 ? w_t[(size_t)at * channels + c0 + v] : 0.f;
    }
    RowVec<T, V> raw[CA_TILE];
#pragma unroll
    for (int i = 0; i < CA_TILE; ++i) raw[i].load(xc + (size_t)min(lo + i, hi - 1) * x_stride);
#pragma unroll
    for (int m = 0; m < TAPS - 1; ++m) {
      const int j = lo - (TAPS - 1) + m;  // place of this input in the portion
      if (j >= 0) {
        RowVec<T, V> r;
        r.load(xc + (size_t)j * x_stride);
        r.get(win[m]);
      } else {
        const int at = taps - 1 + j;
#pragma unroll
        for (int v = 0; v < V; ++v) win[m][v] = at >= 0 ? st[(size_t)at * channels + v] : 0.f;
      }
    }
#pragma unroll
    for (int i = 0; i < CA_TILE; ++i) {
      if (lo + i < hi) {
        float now[V], acc[V];
        raw[i].get(now);
#pragma unroll
        for (int v = 0; v < V; ++v) {
          float a = fmaf(w[TAPS - 1][v], now[v], b[v]);
#pragma unroll
          for (int k = 0; k < TAPS - 1; ++k) a = fmaf(w[k][v], win[k][v], a);
          acc[v] = act_for<T>(a, act);
#pragma unroll
          for (int k = 0; k + 1 < TAPS - 1; ++k) win[k][v] = win[k + 1][v];
          win[TAPS - 2][v] = now[v];
        }
        RowVec<T, V>::store(oc + (size_t)(lo + i) * out_stride, acc);
      }
    }
  } else {
    for (int i = lo; i < hi; ++i) {
      float acc[V];
#pragma unroll
      for (int v = 0; v < V; ++v) acc[v] = b[v];
      for (int k = 0; k < taps; ++k) {
        const int j = i - (taps - 1) + k;
#pragma unroll
        for (int v = 0; v < V; ++v) {
          const float in = j >= 0 ? to_float(xc[(size_t)j * x_stride + v]) : st[(size_t)(taps - 1 + j) * channels + v];
          acc[v] = fmaf(w_t[(size_t)k * channels + c0 + v], in, acc[v]);
        }
      }
#pragma unroll
      for (int v = 0; v < V; ++v) acc[v] = act_for<T>(acc[v], act);
      RowVec<T, V>::store(oc + (size_t)i * out_stride, acc);
    }
  }
  if (lo != 0) return;
  // What the portion leaves; ascending m: what is read lies at or behind what has been written.
  for (int m = 0; m < taps - 1; ++m) {
    const int j = n - (taps - 1) + m;
#pragma unroll
    for (int v = 0; v < V; ++v)
      st[(size_t)m * channels + v] = j >= 0 ? to_float(xc[(size_t)j * x_stride + v]) : st[(size_t)(m + n) * channels + v];
  }
}

// ---------------------------------------------------------------------------------------------
// The scan.  Channels never meet, so a block takes SS_THREADS / L channels of one sequence: L lanes of a warp share
// a channel, each with NS of its states in registers.  Tokens come SS_TC at a time through shared memory (the next
// ones are on their way while these are used); a token of no step size and no input (behind the end) changes
// nothing.  Four tokens' shares of y meet by shuffles at once, each ending in another lane.
//
// Mode 0: a whole sequence in one block, from the slot's state.  Long portions of models with few channels run in
// chunks of `chunk` tokens side by side: every chunk from a zero state, keeping its last state and the sum of
// its step sizes (mode 1; a chunk's whole decay is exp(A sum dt)); the chunks' starting states in order
// (selective_combine_kernel); every chunk again from its starting state, writing y (mode 2).  The chunks of
// sequence s lie at places q_start[s] / chunk + s + c.
constexpr int SS_THREADS = 128;

struct SelectiveScan {
  const void* x;           // [tokens, inner] in the compute dtype
  long long x_stride;
  const float* dt;         // [tokens, inner] logits, bias not yet added
  long long dt_stride;
  const float* dt_bias;    // [inner]
  const float* a2;         // [inner, N]: A log2(e)
  const void* bc;          // rows B [N] | C [N] in the compute dtype
  long long bc_stride;
  const float* d_skip;     // [inner]
  const void* z;           // [tokens, inner]
  long long z_stride;
  void* out;
  long long out_stride;
  float* state;            // [slots][inner, N]
  long long state_stride;
  int inner, N, chunk;
  const int *q_start, *q_len, *seq_slots;
  float* chunk_states;     // [places][inner, N]
  float* chunk_dt;         // [places][inner]
};

template <typename T, int L, int NS, int MODE>
__global__ void __launch_bounds__(SS_THREADS) selective_scan_kernel(SelectiveScan p) {
  constexpr int CB = SS_THREADS / L, NP = L * NS;
  constexpr int TC = NP >= 256 ? 4 : NP >= 128 ? 8 : 16;
  constexpr int BUF = 2 * TC * CB + 2 * TC * NP;
  constexpr int CH_PER = (TC * CB + SS_THREADS - 1) / SS_THREADS;
  constexpr int BC_PER = 2 * TC * NP / SS_THREADS > 0 ? (2 * TC * NP + SS_THREADS - 1) / SS_THREADS : 1;
  extern __shared__ __align__(16) float ss_s[];
  allow_dependents();
  const int tid = threadIdx.x, r = tid % L, ch = tid / L;
  const int c0 = blockIdx.x * CB, c = c0 + ch, s = blockIdx.y;
  const bool live = c < p.inner;
  float a2[NS], S[NS];
#pragma unroll
  for (int k = 0; k < NS; ++k) {
    const int n = r * NS + k;
    a2[k] = live && n < p.N ? p.a2[(size_t)c * p.N + n] : 0.f;
  }
  grid_dependency_wait();
  const int seq_tokens = p.q_len[s], seq_start = p.q_start[s];
  const int lo = MODE == 0 ? 0 : (int)blockIdx.z * p.chunk;
  if (lo >= seq_tokens) return;
  const int n_tok = MODE == 0 ? seq_tokens : min(p.chunk, seq_tokens - lo);
  const size_t start = (size_t)seq_start + lo;
  const size_t place = MODE == 0 ? 0 : (size_t)(seq_start / p.chunk + s) + blockIdx.z;
  float* st = MODE == 0 ? p.state + (size_t)p.seq_slots[s] * p.state_stride : p.chunk_states + place * p.inner * p.N;
  st += (size_t)c * p.N;
#pragma unroll
  for (int k = 0; k < NS; ++k) {
    const int n = r * NS + k;
    S[k] = MODE != 1 && live && n < p.N ? st[n] : 0.f;
  }
  float dt_sum = 0.f;
  const T* x = (const T*)p.x + start * p.x_stride + c0;
  const T* z = (const T*)p.z + start * p.z_stride + c0;
  const T* bc = (const T*)p.bc + start * p.bc_stride;
  const float* dtl = p.dt + start * p.dt_stride + c0;
  T* out = (T*)p.out + start * p.out_stride + c0;
  // A thread's places of a tile: (token, channel) pairs tid + u SS_THREADS, the channel the same for all of them
  // where a tile's width divides the block.
  T pre_x[CH_PER], pre_z[CH_PER], pre_bc[BC_PER], cur_x[CH_PER], cur_z[CH_PER];
  float pre_dt[CH_PER];
  auto fetch = [&](int i0) {
    const int tc = min(TC, n_tok - i0);
#pragma unroll
    for (int u = 0; u < CH_PER; ++u) {
      const int idx = tid + u * SS_THREADS, k = idx / CB, q = idx - k * CB;
      const bool ok = k < tc && c0 + q < p.inner;
      // Loads from valid places, used or not: behind conditions they would be waited for one by one.
      const size_t row = (size_t)(i0 + (ok ? k : 0));
      const int col = ok ? q : 0;
      pre_x[u] = x[row * p.x_stride + col];
      pre_dt[u] = dtl[row * p.dt_stride + col];
      if (MODE != 1) pre_z[u] = z[row * p.z_stride + col];
    }
#pragma unroll
    for (int u = 0; u < BC_PER; ++u) {
      const int idx = tid + u * SS_THREADS, k = idx / (2 * NP), j = idx - k * (2 * NP), arr = j / NP, n = j - arr * NP;
      const bool ok = k < tc && n < p.N;
      pre_bc[u] = bc[(size_t)(i0 + (ok ? k : 0)) * p.bc_stride + (ok ? arr * p.N + n : 0)];
    }
  };
  auto put = [&](float* buf, int i0) {
    const int tc = min(TC, n_tok - i0);
#pragma unroll
    for (int u = 0; u < CH_PER; ++u) {
      const int idx = tid + u * SS_THREADS, k = idx / CB, q = idx - k * CB;
      const bool ok = k < tc && c0 + q < p.inner;
      if (idx < TC * CB) {
        const float dt = ok ? softplus_for<T>(pre_dt[u] + p.dt_bias[c0 + (ok ? q : 0)]) : 0.f;
        buf[idx] = dt;
        buf[TC * CB + idx] = ok ? dt * to_float(pre_x[u]) : 0.f;
      }
      cur_x[u] = pre_x[u];
      if (MODE != 1) cur_z[u] = pre_z[u];
    }
#pragma unroll
    for (int u = 0; u < BC_PER; ++u) {
      const int idx = tid + u * SS_THREADS, k = idx / (2 * NP), j = idx - k * (2 * NP), arr = j / NP, n = j - arr * NP;
      if (idx < 2 * TC * NP) buf[2 * TC * CB + idx] = k < tc && n < p.N ? to_float(pre_bc[u]) : 0.f;
    }
  };
  fetch(0);
  put(ss_s, 0);
  __syncthreads();
  int which = 0;
  for (int i0 = 0; i0 < n_tok; i0 += TC) {
    float* buf = ss_s + which * BUF;
    const bool more = i0 + TC < n_tok;
    if (more) fetch(i0 + TC);
    float* dt_s = buf + ch;               // [TC][CB]; a token's place takes its y when the step size is used
    const float* dx_s = buf + TC * CB + ch;
    const float* bc_s = buf + 2 * TC * CB + r * NS;  // [TC][B NP | C NP]
#pragma unroll 1
    for (int k0 = 0; k0 < TC; k0 += 4) {
      float y[4];
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        const int k = k0 + kk;
        const float dt = dt_s[k * CB], dx = dx_s[k * CB];
        if (MODE == 1) dt_sum += dt;
        float b[NS], cc[NS];
#pragma unroll
        for (int j = 0; j < NS; j += 4) {
          const float4 bv = *reinterpret_cast<const float4*>(bc_s + k * 2 * NP + j);
          b[j] = bv.x, b[j + 1] = bv.y, b[j + 2] = bv.z, b[j + 3] = bv.w;
          if (MODE != 1) {
            const float4 cv = *reinterpret_cast<const float4*>(bc_s + k * 2 * NP + NP + j);
            cc[j] = cv.x, cc[j + 1] = cv.y, cc[j + 2] = cv.z, cc[j + 3] = cv.w;
          }
        }
        float acc = 0.f;
#pragma unroll
        for (int j = 0; j < NS; ++j) {
          S[j] = fmaf(pow2_for<T>(dt * a2[j]), S[j], dx * b[j]);
          if (MODE != 1) acc = fmaf(S[j], cc[j], acc);
        }
        y[kk] = acc;
      }
      if (MODE != 1) {
        // Two tokens stay with each lane of a pair, then one with each lane of four.
        int token = 0;
        if (L >= 2) {
          const bool up = (r & 1) != 0;
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const float give = up ? y[i] : y[i + 2], keep = up ? y[i + 2] : y[i];
            y[i] = keep + __shfl_xor_sync(0xffffffffu, give, 1);
          }
          token = up ? 2 : 0;
        }
        if (L >= 4) {
          const bool up = (r & 2) != 0;
          const float give = up ? y[0] : y[1], keep = up ? y[1] : y[0];
          y[0] = keep + __shfl_xor_sync(0xffffffffu, give, 2);
          token += up ? 1 : 0;
#pragma unroll
          for (int off = 4; off < L; off <<= 1) y[0] += __shfl_xor_sync(0xffffffffu, y[0], off);
        }
        constexpr int OWN = L >= 4 ? 1 : 4 / L;
        if (L <= 4 || r < 4) {
#pragma unroll
          for (int i = 0; i < OWN; ++i) dt_s[(k0 + token + i) * CB] = y[i];
        }
      }
    }
    if (MODE != 1) {
      __syncthreads();
#pragma unroll
      for (int u = 0; u < CH_PER; ++u) {
        const int idx = tid + u * SS_THREADS, k = idx / CB, q = idx - k * CB;
        if (idx < TC * CB && i0 + k < n_tok && c0 + q < p.inner)
          out[(size_t)(i0 + k) * p.out_stride + q] =
              from_float<T>(fmaf(p.d_skip[c0 + q], to_float(cur_x[u]), buf[idx]) * silu_for<T>(to_float(cur_z[u])));
      }
    }
    if (more) put(ss_s + (which ^ 1) * BUF, i0 + TC);
    __syncthreads();  // the next tokens are in place, and these may be overwritten
    which ^= 1;
  }
  if (MODE == 2) return;
  if (live) {
#pragma unroll
    for (int k = 0; k < NS; ++k) {
      const int n = r * NS + k;
      if (n < p.N) st[n] = S[k];
    }
    if (MODE == 1 && r == 0) p.chunk_dt[place * p.inner + c] = dt_sum;
  }
}

// Per sequence: the states its chunks start from, in order (each in the place of the chunk's own last state), and
// the sequence's new state.
template <typename T>
__global__ void selective_combine_kernel(SelectiveScan p) {
  allow_dependents();
  grid_dependency_wait();
  const int s = blockIdx.y, n_tok = p.q_len[s];
  if (n_tok <= 0) return;
  const size_t total = (size_t)p.inner * p.N, first = (size_t)(p.q_start[s] / p.chunk + s);
  const int chunks = (n_tok + p.chunk - 1) / p.chunk;
  for (size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (size_t)gridDim.x * blockDim.x) {
    const size_t c = e / p.N;
    const float a2 = p.a2[e];
    float* st = p.state + (size_t)p.seq_slots[s] * p.state_stride + e;
    float S = *st;
    for (int k = 0; k < chunks; ++k) {
      float* at = p.chunk_states + (first + k) * total + e;
      const float own = *at;
      *at = S;
      S = fmaf(pow2_for<T>(a2 * p.chunk_dt[(first + k) * p.inner + c]), S, own);
    }
    *st = S;
  }
}

// One token of every sequence: dt = softplus(W_dt low + bias) with `low` the first `rank` columns of the row
// `low | B | C`, then the state's update and the gated result.  L lanes share a channel and its row of W_dt.
template <typename T, int L, int NS>
__global__ void __launch_bounds__(SS_THREADS)
selective_step_kernel(SelectiveScan p, const T* __restrict__ low, const T* __restrict__ w_dt, int rank, int packs) {
  constexpr int CB = SS_THREADS / L, PK = 16 / (int)sizeof(T), AHEAD = 4;
  extern __shared__ __align__(16) float ss_s[];
  float* low_s = ss_s;                      // [rank, padded to 8]
  float* bc_s = low_s + (rank + 7) / 8 * 8; // [2 N]
  allow_dependents();
  const int tid = threadIdx.x, r = tid % L, ch = tid / L;
  const int c = blockIdx.x * CB + ch, s = blockIdx.y;
  const bool live = c < p.inner;
  const int row_c = live ? c : 0;
  float a2[NS];
#pragma unroll
  for (int k = 0; k < NS; ++k) {
    const int n = r * NS + k;
    a2[k] = live && n < p.N ? p.a2[(size_t)c * p.N + n] : 0.f;
  }
  const T* wr = w_dt + (size_t)row_c * rank;
  // Weights do not depend on the kernel before this one.
  uint4 ahead[AHEAD];
  if (packs) {
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
      const int i = (r + u * L) * PK;
      ahead[u] = i < rank ? __ldg(reinterpret_cast<const uint4*>(wr + i)) : make_uint4(0u, 0u, 0u, 0u);
    }
  }
  const float bias = p.dt_bias[row_c], skip = p.d_skip[row_c];
  const int slot = p.seq_slots[s];
  const size_t row = (size_t)p.q_start[s];
  float* st = p.state + (size_t)slot * p.state_stride + (size_t)row_c * p.N;
  if (r == 0) asm volatile("prefetch.global.L2 [%0];" ::"l"(st));
  grid_dependency_wait();
  float S[NS];
#pragma unroll
  for (int k = 0; k < NS; ++k) {
    const int n = r * NS + k;
    S[k] = live && n < p.N ? st[n] : 0.f;
  }
  const float xv = to_float(((const T*)p.x)[row * p.x_stride + row_c]);
  const float zv = to_float(((const T*)p.z)[row * p.z_stride + row_c]);
  const T* lr = low + row * p.bc_stride;
  for (int i = tid; i < (rank + 7) / 8 * 8; i += SS_THREADS) low_s[i] = i < rank ? to_float(lr[i]) : 0.f;
  for (int i = tid; i < 2 * p.N; i += SS_THREADS) bc_s[i] = to_float(lr[rank + i]);
  __syncthreads();
  float acc = 0.f;
  if (packs) {
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
      const int i = (r + u * L) * PK;
      const T* e = reinterpret_cast<const T*>(&ahead[u]);
      if (i < rank) {
#pragma unroll
        for (int q = 0; q < PK; ++q) acc = fmaf(to_float(e[q]), low_s[i + q], acc);
      }
    }
    for (int i = (r + AHEAD * L) * PK; i < rank; i += L * PK) {
      const uint4 raw = __ldg(reinterpret_cast<const uint4*>(wr + i));
      const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
      for (int q = 0; q < PK; ++q) acc = fmaf(to_float(e[q]), low_s[i + q], acc);
    }
  } else {
    for (int i = r; i < rank; i += L) acc = fmaf(to_float(wr[i]), low_s[i], acc);
  }
#pragma unroll
  for (int off = L / 2; off > 0; off >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, off);
  const float dt = softplus_for<T>(acc + bias), dx = dt * xv;
  float y = 0.f;
#pragma unroll
  for (int k = 0; k < NS; ++k) {
    const int n = r * NS + k;
    if (n < p.N) {
      S[k] = fmaf(pow2_for<T>(dt * a2[k]), S[k], dx * bc_s[n]);
      y = fmaf(S[k], bc_s[p.N + n], y);
    }
  }
#pragma unroll
  for (int off = L / 2; off > 0; off >>= 1) y += __shfl_xor_sync(0xffffffffu, y, off);
  if (live) {
#pragma unroll
    for (int k = 0; k < NS; ++k) {
      const int n = r * NS + k;
      if (n < p.N) st[n] = S[k];
    }
    if (r == 0) ((T*)p.out)[row * p.out_stride + c] = from_float<T>(fmaf(skip, xv, y) * silu_for<T>(zv));
  }
}

}  // namespace vx

using namespace vx;

template <typename T, int V>
static void launch_conv_act(const void* x, long long x_stride, int channels, int taps, const float* w_t, const float* bias,
                            float* state, long long state_stride, void* out, long long out_stride, const int* q_start,
                            const int* q_len, const int* seq_slots, int num_seqs, int longest, int act,
                            cudaStream_t stream) {
  // The general form re-reads its inputs, so a tile may be as short; it must still hold what reads the state.
  const int tile = taps <= 4 ? CA_TILE : (taps - 1 <= 32 ? 32 : 1 << 30);
  const int tiles = tile >= longest ? 1 : (longest + tile - 1) / tile;
  const dim3 grid((channels / V + 127) / 128, tiles, num_seqs);
#define VX_CONV_ACT(TAPS)                                                                                                \
  launch_pdl(conv_act_kernel<T, V, TAPS>, grid, dim3(128), 0, stream, (const T*)x, x_stride, channels, taps, w_t, bias, state, \
             state_stride, (T*)out, out_stride, q_start, q_len, seq_slots, tile, act)
  if (taps <= 4) VX_CONV_ACT(4);
  else VX_CONV_ACT(0);
#undef VX_CONV_ACT
}

// x rows [tokens, channels] -> out rows, w_t [taps, channels]; `longest`: no portion has more tokens.
VX_API int vx_conv_act(const void* x, int dtype, long long x_stride, int channels, int taps, const float* w_t,
                       const float* bias, float* state, long long state_stride, void* out, long long out_stride,
                       const int* q_start, const int* q_len, const int* seq_slots, int num_seqs, int longest, int act,
                       cudaStream_t stream) {
  if (num_seqs <= 0 || channels <= 0 || longest <= 0) return 0;
  if (taps < 1 || num_seqs > 65535) return (int)cudaErrorInvalidValue;
  const int pack = dtype == VX_DTYPE_F32 ? 4 : 8;
  const bool vec = channels % pack == 0 && x_stride % pack == 0 && out_stride % pack == 0 &&
                   ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
#define VX_CONV_LAUNCH(T, V)                                                                                           \
  launch_conv_act<T, V>(x, x_stride, channels, taps, w_t, bias, state, state_stride, out, out_stride, q_start, q_len, \
                        seq_slots, num_seqs, longest, act, stream)
  if (dtype == VX_DTYPE_F32) {
    if (vec) VX_CONV_LAUNCH(float, 4);
    else VX_CONV_LAUNCH(float, 1);
  } else {
    if (vec) VX_CONV_LAUNCH(__nv_bfloat16, 8);
    else VX_CONV_LAUNCH(__nv_bfloat16, 1);
  }
#undef VX_CONV_LAUNCH
  return (int)cudaGetLastError();
}

template <typename T, int L, int NS>
static int launch_selective_scan(const SelectiveScan& p, int num_seqs, int num_tokens, cudaStream_t stream) {
  constexpr int CB = SS_THREADS / L, NP = L * NS, TC = NP >= 256 ? 4 : NP >= 128 ? 8 : 16;
  constexpr size_t smem = sizeof(float) * 2 * (2 * TC * CB + 2 * TC * NP);
  static bool configured = false;
  if (smem > 48 * 1024 && !configured) {
    cudaError_t e = cudaFuncSetAttribute(selective_scan_kernel<T, L, NS, 0>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(selective_scan_kernel<T, L, NS, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(selective_scan_kernel<T, L, NS, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const int blocks = (p.inner + CB - 1) / CB;
  if (p.chunk <= 0 || num_tokens <= p.chunk) {
    launch_pdl(selective_scan_kernel<T, L, NS, 0>, dim3(blocks, num_seqs), dim3(SS_THREADS), smem, stream, p);
    return (int)cudaGetLastError();
  }
  const dim3 grid(blocks, num_seqs, (num_tokens + p.chunk - 1) / p.chunk);
  launch_pdl(selective_scan_kernel<T, L, NS, 1>, grid, dim3(SS_THREADS), smem, stream, p);
  int cblocks = (int)(((size_t)p.inner * p.N + 255) / 256);
  if (cblocks > 148 * 8) cblocks = 148 * 8;
  launch_pdl(selective_combine_kernel<T>, dim3(cblocks, num_seqs), dim3(256), 0, stream, p);
  launch_pdl(selective_scan_kernel<T, L, NS, 2>, grid, dim3(SS_THREADS), smem, stream, p);
  return (int)cudaGetLastError();
}

// The most states of a channel the kernels hold.
VX_API int vx_selective_max_state() { return 512; }

// Channels of one block of the scan, for the caller's choice of chunks.
VX_API int vx_selective_block_channels(int N) {
  if (N <= 4) return SS_THREADS;
  if (N <= 8) return SS_THREADS / 2;
  if (N <= 16) return SS_THREADS / 4;
  if (N <= 32) return SS_THREADS / 8;
  if (N <= 64) return SS_THREADS / 16;
  return SS_THREADS / 32;
}

#define VX_SELECTIVE_SIZES(CALL)   \
  if (p.N <= 4) { CALL(1, 4) }     \
  if (p.N <= 8) { CALL(2, 4) }     \
  if (p.N <= 16) { CALL(4, 4) }    \
  if (p.N <= 32) { CALL(8, 4) }    \
  if (p.N <= 64) { CALL(16, 4) }   \
  if (p.N <= 128) { CALL(32, 4) }  \
  if (p.N <= 256) { CALL(32, 8) }  \
  CALL(32, 16)

// chunk 0 (or the two chunk buffers null): every sequence in one block per group of channels; else chunk_states
// holds (num_tokens / chunk + num_seqs + 1) * inner * N floats and chunk_dt as many times inner.
VX_API int vx_selective_scan(const void* x, int dtype, long long x_stride, const float* dt, long long dt_stride,
                             const float* dt_bias, const float* a2, const void* bc, long long bc_stride,
                             const float* d_skip, const void* z, long long z_stride, void* out, long long out_stride,
                             float* state, long long state_stride, int inner, int N, int chunk, float* chunk_states,
                             float* chunk_dt, const int* q_start, const int* q_len, const int* seq_slots, int num_seqs,
                             int num_tokens, cudaStream_t stream) {
  if (num_seqs <= 0 || num_tokens <= 0) return 0;
  if (inner <= 0 || N <= 0 || N > 512 || num_seqs > 65535) return (int)cudaErrorInvalidValue;
  if (chunk_states == nullptr || chunk_dt == nullptr) chunk = 0;
  const SelectiveScan p = {x, x_stride, dt, dt_stride, dt_bias, a2, bc, bc_stride, d_skip, z, z_stride, out, out_stride,
                           state, state_stride, inner, N, chunk, q_start, q_len, seq_slots, chunk_states, chunk_dt};
#define VX_SCAN_CALL(L, NS) VX_BY_DTYPE(dtype, return (launch_selective_scan<T, L, NS>(p, num_seqs, num_tokens, stream)))
  VX_SELECTIVE_SIZES(VX_SCAN_CALL)
#undef VX_SCAN_CALL
}

template <typename T, int L, int NS>
static int launch_selective_step(const SelectiveScan& p, const void* low, const void* w_dt, int rank, int num_seqs,
                                 cudaStream_t stream) {
  constexpr int CB = SS_THREADS / L;
  const size_t smem = sizeof(float) * ((size_t)(rank + 7) / 8 * 8 + 2 * (size_t)p.N);
  if (smem > 46 * 1024) return -1;
  const int packs = rank % (16 / (int)sizeof(T)) == 0 && (reinterpret_cast<uintptr_t>(w_dt) & 15) == 0;
  launch_pdl(selective_step_kernel<T, L, NS>, dim3((p.inner + CB - 1) / CB, num_seqs), dim3(SS_THREADS), smem, stream, p,
             (const T*)low, (const T*)w_dt, rank, packs);
  return (int)cudaGetLastError();
}

// One token of every sequence; `low` rows hold low [rank] | B [N] | C [N]; -1: sizes the kernel does not take.
VX_API int vx_selective_step(const void* x, int dtype, long long x_stride, const void* low, long long low_stride,
                             const void* w_dt, int rank, const float* dt_bias, const float* a2, const float* d_skip,
                             const void* z, long long z_stride, void* out, long long out_stride, float* state,
                             long long state_stride, int inner, int N, const int* q_start, const int* seq_slots,
                             int num_seqs, cudaStream_t stream) {
  if (num_seqs <= 0) return 0;
  if (inner <= 0 || N <= 0 || N > 512 || rank <= 0 || num_seqs > 65535) return (int)cudaErrorInvalidValue;
  const SelectiveScan p = {x, x_stride, nullptr, 0, dt_bias, a2, nullptr, low_stride, d_skip, z, z_stride, out, out_stride,
                           state, state_stride, inner, N, 0, q_start, nullptr, seq_slots, nullptr, nullptr};
#define VX_STEP_CALL(L, NS) VX_BY_DTYPE(dtype, return (launch_selective_step<T, L, NS>(p, low, w_dt, rank, num_seqs, stream)))
  VX_SELECTIVE_SIZES(VX_STEP_CALL)
#undef VX_STEP_CALL
}
