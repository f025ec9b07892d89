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

// Sixteen bytes of a row as floats.
template <typename T, int V>
struct RowVec;
template <>
struct RowVec<float, 4> {
  float4 raw;
  __device__ __forceinline__ void load(const float* p) { raw = *reinterpret_cast<const float4*>(p); }
  __device__ __forceinline__ void get(float (&v)[4]) const { v[0] = raw.x, v[1] = raw.y, v[2] = raw.z, v[3] = raw.w; }
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
};
template <typename T>
struct RowVec<T, 1> {};

// PV neighbouring values of a row.
template <typename T, int PV>
struct PairOf;
template <typename T>
struct PairOf<T, 1> {
  T v;
  __device__ __forceinline__ void load(const T* p) { v = *p; }
  __device__ __forceinline__ float get(int) const { return to_float(v); }
  static __device__ __forceinline__ void store(T* p, const float (&f)[1]) { *p = from_float<T>(f[0]); }
};
template <>
struct PairOf<float, 2> {
  float2 v;
  __device__ __forceinline__ void load(const float* p) { v = *reinterpret_cast<const float2*>(p); }
  __device__ __forceinline__ float get(int e) const { return e == 0 ? v.x : v.y; }
  static __device__ __forceinline__ void store(float* p, const float (&f)[2]) {
    *reinterpret_cast<float2*>(p) = make_float2(f[0], f[1]);
  }
};
template <>
struct PairOf<__nv_bfloat16, 2> {
  uint32_t v;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { v = *reinterpret_cast<const uint32_t*>(p); }
  __device__ __forceinline__ float get(int e) const { return __uint_as_float(e == 0 ? v << 16 : v & 0xffff0000u); }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&f)[2]) {
    *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(f[0], f[1]);
  }
};

// ---------------------------------------------------------------------------------------------
// out_t = act(bias + sum_k w[k] x_(t - taps + 1 + k)) per channel.  state[slot][m][c], m = 0 .. taps - 2, is the
// input taps - 1 - m positions before the portion's first token (zero before the sequence's start).  w_t
// [taps][channels].  A thread takes V neighbouring channels of a tile of CA_TILE tokens; only the first tile of a
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
    PairOf<T, V> raw[CA_TILE];
#pragma unroll
    for (int i = 0; i < CA_TILE; ++i) raw[i].load(xc + (size_t)min(lo + i, hi - 1) * x_stride);
#pragma unroll
    for (int m = 0; m < TAPS - 1; ++m) {
      const int j = lo - (TAPS - 1) + m;  // place of this input in the portion
      if (j >= 0) {
        PairOf<T, V> r;
        r.load(xc + (size_t)j * x_stride);
#pragma unroll
        for (int v = 0; v < V; ++v) win[m][v] = r.get(v);
      } else {
        const int at = taps - 1 + j;
#pragma unroll
        for (int v = 0; v < V; ++v) win[m][v] = at >= 0 ? st[(size_t)at * channels + v] : 0.f;
      }
    }
#pragma unroll
    for (int i = 0; i < CA_TILE; ++i) {
      if (lo + i < hi) {
        float acc[V];
#pragma unroll
        for (int v = 0; v < V; ++v) {
          const float now = raw[i].get(v);
          float a = fmaf(w[TAPS - 1][v], now, b[v]);
#pragma unroll
          for (int k = 0; k < TAPS - 1; ++k) a = fmaf(w[k][v], win[k][v], a);
          acc[v] = act_for<T>(a, act);
#pragma unroll
          for (int k = 0; k + 1 < TAPS - 1; ++k) win[k][v] = win[k + 1][v];
          win[TAPS - 2][v] = now;
        }
        PairOf<T, V>::store(oc + (size_t)(lo + i) * out_stride, acc);
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
      PairOf<T, V>::store(oc + (size_t)i * out_stride, acc);
    }
  }
  if (lo != 0) return;
  // What the portion leaves; ascending m: what is read lies at or behind what has been written.
#pragma unroll 1
  for (int m = 0; m < taps - 1; ++m) {
    const int j = n - (taps - 1) + m;
#pragma unroll
    for (int v = 0; v < V; ++v)
      st[(size_t)m * channels + v] = j >= 0 ? to_float(xc[(size_t)j * x_stride + v]) : st[(size_t)(m + n) * channels + v];
  }
}

// ---------------------------------------------------------------------------------------------
// The scan.  Channels never meet, so a block takes CB channels of one sequence.  Its scan warps do nothing else: L lanes of
// a warp share a channel, each with NS of its states in registers, and four tokens' shares of y meet by shuffles at
// once, each ending in another lane.  Four helper warps, each for every fourth tile of tokens, bring a tile into a shared
// buffer of its own (step sizes through their softplus), ask for the one four tiles on, wait until the tile has
// been scanned and turn its sums into outputs: a tile's way through its warp may take three times as long as
// its scan.  Scan warps and helpers meet at two barriers per buffer.  A token of no step size and no input (behind the end) changes nothing.
//
// Mode 0: a whole sequence in one block, from the slot's state.  Long portions of models with few channels run in
// chunks of `chunk` tokens side by side: every chunk from a zero state, keeping its last state and the sum of
// its step sizes (mode 1; a chunk's whole decay is exp(A sum dt)); the chunks' starting states in order
// (selective_combine_kernel); every chunk again from its starting state, writing y (mode 2).  The chunks of
// sequence s lie at places q_start[s] / chunk + s + c.
constexpr int SS_THREADS = 128;  // of the one-token kernel
constexpr int SS_HELPERS = 32, SS_GROUPS = 4;  // helpers of a tile (a warp), and tiles that are looked after side by side
__host__ __device__ constexpr int ss_scan_threads(int L) { return L == 1 ? 32 : L <= 4 ? 64 : 128; }
__host__ __device__ constexpr int ss_tile(int L, int NP) { return NP >= 256 ? 4 : NP >= 128 || L == 1 ? 8 : 16; }

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
  int* status;
};

template <typename T, int L, int NS, int MODE, bool VEC>
__global__ void __launch_bounds__(ss_scan_threads(L) + SS_GROUPS * SS_HELPERS) selective_scan_kernel(SelectiveScan p) {
  constexpr int SCAN = ss_scan_threads(L), CB = SCAN / L, NP = L * NS, TC = ss_tile(L, NP);
  constexpr int BUF = 2 * TC * CB + 2 * TC * NP;  // dt, dt x, then B | C of every token
  // A helper's places of a tile: CH_PER tokens of PV neighbouring channels, STEP tokens apart.  VEC: channels in
  // pairs, and the B | C rows in packs of sixteen bytes, where sizes and alignment allow it.
  constexpr int PV = VEC ? 2 : 1, LANES = CB / PV, STEP = SS_HELPERS / LANES;
  constexpr int CH_PER = (TC + STEP - 1) / STEP;
  constexpr int BC_PER = 2 * TC * NP / SS_HELPERS;       // values a helper
  static_assert(SS_HELPERS % CB == 0 && 2 * TC * NP % SS_HELPERS == 0, "a helper keeps to its channels");
  extern __shared__ __align__(16) float ss_s[];  // a buffer per group, then as many tiles of y [TC][CB]
  __shared__ __align__(8) unsigned long long bars[2 * SS_GROUPS];  // per buffer: a tile is there; it has been scanned
  float* y_s = ss_s + SS_GROUPS * BUF;
  allow_dependents();
  const int tid = threadIdx.x, c0 = blockIdx.x * CB, s = blockIdx.y;
  const bool scans = tid < SCAN;
  const int r = tid % L, ch = tid / L, c = c0 + ch;  // of a scanning thread
  const bool live = scans && c < p.inner;
  float a2[NS], S[NS];
  if (scans) {
#pragma unroll
    for (int k = 0; k < NS; ++k) {
      const int n = r * NS + k;
      a2[k] = live && n < p.N ? p.a2[(size_t)c * p.N + n] : 0.f;
    }
  }
  const int group = (tid - SCAN) / SS_HELPERS, helper = (tid - SCAN) % SS_HELPERS;  // of a helper
  const int q = scans ? 0 : (helper % LANES) * PV, k0 = scans ? 0 : helper / LANES;
  const bool q_ok = !scans && c0 + q < p.inner;
  float bias[PV], skip[PV];
#pragma unroll
  for (int e = 0; e < PV; ++e) {
    bias[e] = q_ok ? p.dt_bias[c0 + q + e] : 0.f;
    skip[e] = q_ok ? p.d_skip[c0 + q + e] : 0.f;
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
  const int tiles = (n_tok + TC - 1) / TC;
  if (tid == 0) {
    for (int g = 0; g < SS_GROUPS; ++g) {
      mbar_init(smem_u32(&bars[g]), SS_HELPERS);
      mbar_init(smem_u32(&bars[SS_GROUPS + g]), SCAN / 32);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  // Packs of B and C: what lies behind N states of a row is never written again.
  if (VEC && p.N < NP)
    for (int idx = tid; idx < SS_GROUPS * 2 * TC * NP; idx += blockDim.x)
      if ((idx & (NP - 1)) >= p.N) ss_s[(idx / (2 * TC * NP)) * BUF + 2 * TC * CB + idx % (2 * TC * NP)] = 0.f;
  __syncthreads();
  if (scans) {
#pragma unroll
    for (int k = 0; k < NS; ++k) {
      const int n = r * NS + k;
      S[k] = MODE != 1 && live && n < p.N ? st[n] : 0.f;
    }
    float dt_sum = 0.f;
    for (int i = 0; i < tiles; ++i) {
      const int g_of = i % SS_GROUPS;
      const float* buf = ss_s + g_of * BUF;
      mbar_wait(smem_u32(&bars[g_of]), (uint32_t)(i / SS_GROUPS) & 1u, p.status);
      const float* dt_s = buf + ch;
      const float* dx_s = buf + TC * CB + ch;
      const float* bc_s = buf + 2 * TC * CB + r * NS;
      float* y_out = y_s + g_of * TC * CB + ch;
      // Four tokens at a time, in the order in which a warp should issue them: the next four's loads, this four's sums,
      // the next four's decays.  A tile's sums stay in registers until its last token: a store among the loads of
      // later tokens would hold them up (it could be to the same place).
      constexpr int OWN = L >= 4 ? 1 : 4 / L;
      float sums[TC / 4][OWN];
      int token = 0;
      float decay[4][NS], input[4][NS], cc[4][NS];
      auto load = [&](int g, float (&dt)[4], float (&dx)[4], float (&b)[4][NS], float (&c)[4][NS]) {
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
          const int k = g + kk;
          dt[kk] = dt_s[k * CB], dx[kk] = dx_s[k * CB];
#pragma unroll
          for (int j = 0; j < NS; j += 4) {
            const float4 bv = *reinterpret_cast<const float4*>(bc_s + k * 2 * NP + j);
            b[kk][j] = bv.x, b[kk][j + 1] = bv.y, b[kk][j + 2] = bv.z, b[kk][j + 3] = bv.w;
            if (MODE != 1) {
              const float4 cv = *reinterpret_cast<const float4*>(bc_s + k * 2 * NP + NP + j);
              c[kk][j] = cv.x, c[kk][j + 1] = cv.y, c[kk][j + 2] = cv.z, c[kk][j + 3] = cv.w;
            }
          }
        }
      };
      auto weigh = [&](const float (&dt)[4], const float (&dx)[4], const float (&b)[4][NS]) {
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
          if (MODE == 1) dt_sum += dt[kk];
#pragma unroll
          for (int j = 0; j < NS; ++j) {
            decay[kk][j] = pow2_for<T>(dt[kk] * a2[j]);
            input[kk][j] = dx[kk] * b[kk][j];
          }
        }
      };
      {
        float dt[4], dx[4], b[4][NS];
        load(0, dt, dx, b, cc);
        weigh(dt, dx, b);
      }
#pragma unroll
      for (int g = 0; g < TC; g += 4) {
        float dt[4], dx[4], b[4][NS], c_next[4][NS];
        if (g + 4 < TC) load(g + 4, dt, dx, b, c_next);
        float y[4];
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
          float acc = 0.f;
#pragma unroll
          for (int j = 0; j < NS; ++j) {
            S[j] = fmaf(decay[kk][j], S[j], input[kk][j]);
            if (MODE != 1) acc = fmaf(S[j], cc[kk][j], acc);
          }
          y[kk] = acc;
        }
        // Two tokens stay with each lane of a pair, then one with each lane of four.
        float kept[2], given[2];
        if (MODE != 1 && L >= 2) {
          const bool up = (r & 1) != 0;
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            given[e] = __shfl_xor_sync(0xffffffffu, up ? y[e] : y[e + 2], 1);
            kept[e] = up ? y[e + 2] : y[e];
          }
          token = up ? 2 : 0;
        }
        if (g + 4 < TC) {
          weigh(dt, dx, b);
          if (MODE != 1) {
#pragma unroll
            for (int kk = 0; kk < 4; ++kk)
#pragma unroll
              for (int j = 0; j < NS; ++j) cc[kk][j] = c_next[kk][j];
          }
        }
        if (MODE != 1) {
          if (L >= 2) {
#pragma unroll
            for (int e = 0; e < 2; ++e) y[e] = kept[e] + given[e];
          }
          if (L >= 4) {
            const bool up = (r & 2) != 0;
            const float give = up ? y[0] : y[1], keep = up ? y[1] : y[0];
            y[0] = keep + __shfl_xor_sync(0xffffffffu, give, 2);
            token += up ? 1 : 0;
            if constexpr (L > 4) {
#pragma unroll
              for (int off = 4; off < L; off <<= 1) y[0] += __shfl_xor_sync(0xffffffffu, y[0], off);
            }
          }
#pragma unroll
          for (int e = 0; e < OWN; ++e) sums[g / 4][e] = y[e];
        }
      }
      if (MODE != 1 && (L <= 4 || r < 4)) {
#pragma unroll
        for (int g = 0; g < TC; g += 4)
#pragma unroll
          for (int e = 0; e < OWN; ++e) y_out[(g + token + e) * CB] = sums[g / 4][e];
      }
      __syncwarp();
      if ((tid & 31) == 0) mbar_arrive(smem_u32(&bars[SS_GROUPS + g_of]));
    }
    if (MODE != 2 && live) {
#pragma unroll
      for (int k = 0; k < NS; ++k) {
        const int n = r * NS + k;
        if (n < p.N) st[n] = S[k];
      }
      if (MODE == 1 && r == 0) p.chunk_dt[place * p.inner + c] = dt_sum;
    }
    return;
  }
  // Helpers.  Loads go to valid places, used or not: behind conditions they would be waited for one by one.
  const int col = q_ok ? q : 0;
  const T* x = (const T*)p.x + start * p.x_stride + c0 + col;
  const T* z = (const T*)p.z + start * p.z_stride + c0 + col;
  const T* bc = (const T*)p.bc + start * p.bc_stride;
  const float* dtl = p.dt + start * p.dt_stride + c0 + col;
  T* out = (T*)p.out + start * p.out_stride + c0 + col;
  typedef PairOf<T, PV> Pair;
  Pair in_x[CH_PER], in_z[CH_PER], past_x[CH_PER], past_z[CH_PER];  // on their way; of the tile that is scanned
  PairOf<float, PV> in_dt[CH_PER];
  T in_bc[VEC ? 1 : BC_PER];
  // Sixteen-byte packs of a tile's B | C rows: a helper's are at the same places of every tile.
  constexpr int PACK = 16 / (int)sizeof(T), PACK_PER = VEC ? (2 * TC * NP / PACK + SS_HELPERS - 1) / SS_HELPERS : 1;
  RowVec<T, VEC ? PACK : 1> in_packs[PACK_PER];
  int pack_token[PACK_PER], pack_col[PACK_PER], pack_at[PACK_PER];
  if constexpr (VEC) {
    const int per_row = 2 * p.N / PACK, packs = TC * per_row;
#pragma unroll
    for (int u = 0; u < PACK_PER; ++u) {
      const int at = helper + u * SS_HELPERS, k = min(at, packs - 1) / per_row, j = (min(at, packs - 1) - k * per_row) * PACK;
      pack_token[u] = k;
      pack_col[u] = j;
      pack_at[u] = at < packs ? k * 2 * NP + (j < p.N ? j : NP + j - p.N) : -1;
    }
  }
  auto fetch = [&](int i) {
    const int i0 = i * TC;
#pragma unroll
    for (int u = 0; u < CH_PER; ++u) {
      const size_t row = (size_t)min(i0 + k0 + u * STEP, n_tok - 1);
      in_x[u].load(x + row * p.x_stride);
      in_dt[u].load(dtl + row * p.dt_stride);
      if (MODE != 1) in_z[u].load(z + row * p.z_stride);
    }
    if constexpr (VEC) {
#pragma unroll
      for (int u = 0; u < PACK_PER; ++u) {
        in_packs[u].load(bc + (size_t)min(i0 + pack_token[u], n_tok - 1) * p.bc_stride + pack_col[u]);
      }
    } else {
#pragma unroll
      for (int u = 0; u < BC_PER; ++u) {
        const int idx = helper + u * SS_HELPERS, k = idx / (2 * NP), j = idx - k * (2 * NP), arr = j / NP, n = j - arr * NP;
        if (MODE == 1 && NP >= SS_HELPERS && arr == 1) continue;
        in_bc[u] = bc[(size_t)min(i0 + k, n_tok - 1) * p.bc_stride + arr * p.N + min(n, p.N - 1)];
      }
    }
  };
  auto put = [&](int i) {
    const int i0 = i * TC;
    float* buf = ss_s + group * BUF;
#pragma unroll
    for (int u = 0; u < CH_PER; ++u) {
      const int k = k0 + u * STEP;
      const bool ok = q_ok && i0 + k < n_tok;
      if (k < TC) {
        float dt[PV], dx[PV];
#pragma unroll
        for (int e = 0; e < PV; ++e) {
          dt[e] = ok ? softplus_for<T>(in_dt[u].get(e) + bias[e]) : 0.f;
          dx[e] = ok ? dt[e] * in_x[u].get(e) : 0.f;
        }
        PairOf<float, PV>::store(buf + k * CB + q, dt);
        PairOf<float, PV>::store(buf + TC * CB + k * CB + q, dx);
      }
    }
    float* bc_out = buf + 2 * TC * CB;
    if constexpr (VEC) {
#pragma unroll
      for (int u = 0; u < PACK_PER; ++u) {
        if (pack_at[u] >= 0) {
          float v[PACK];
          in_packs[u].get(v);
#pragma unroll
          for (int e = 0; e < PACK; e += 4)
            *reinterpret_cast<float4*>(bc_out + pack_at[u] + e) = make_float4(v[e], v[e + 1], v[e + 2], v[e + 3]);
        }
      }
    } else {
#pragma unroll
      for (int u = 0; u < BC_PER; ++u) {
        const int idx = helper + u * SS_HELPERS, k = idx / (2 * NP), j = idx - k * (2 * NP), n = j & (NP - 1);
        if (MODE == 1 && NP >= SS_HELPERS && j >= NP) continue;
        bc_out[idx] = i0 + k < n_tok && n < p.N ? to_float(in_bc[u]) : 0.f;
      }
    }
  };
  auto finish = [&](int i) {
#pragma unroll
    for (int u = 0; u < CH_PER; ++u) {
      const int k = k0 + u * STEP;
      if (k < TC && q_ok && i * TC + k < n_tok) {
        float y[PV];
#pragma unroll
        for (int e = 0; e < PV; ++e)
          y[e] = fmaf(skip[e], past_x[u].get(e), y_s[group * TC * CB + k * CB + q + e]) * silu_for<T>(past_z[u].get(e));
        Pair::store(out + (size_t)(i * TC + k) * p.out_stride, y);
      }
    }
  };
  // (A token behind the end has dt = dx = 0: what B and C hold there does not matter.)
  const uint32_t there = smem_u32(&bars[group]), scanned = smem_u32(&bars[SS_GROUPS + group]);
  if (group < tiles) fetch(group);
  for (int t = group; t < tiles; t += SS_GROUPS) {
    put(t);
    mbar_arrive(there);
#pragma unroll
    for (int u = 0; u < CH_PER; ++u) {
      past_x[u] = in_x[u];
      if (MODE != 1) past_z[u] = in_z[u];
    }
    if (t + SS_GROUPS < tiles) fetch(t + SS_GROUPS);
    mbar_wait(scanned, (uint32_t)(t / SS_GROUPS) & 1u, p.status);
    if (MODE != 1) finish(t);
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
    float* at = p.chunk_states + first * total + e;
    const float* dt = p.chunk_dt + first * p.inner + c;
    float S = *st;
    for (int k = 0; k < chunks; k += 8) {
      // Eight chunks' values are under way together.
      float own[8], decay[8];
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        const size_t at_k = (size_t)min(k + u, chunks - 1);
        own[u] = at[at_k * total];
        decay[u] = dt[at_k * p.inner];
      }
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        if (k + u < chunks) {
          at[(size_t)(k + u) * total] = S;
          S = fmaf(pow2_for<T>(a2 * decay[u]), S, own[u]);
        }
      }
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
  const bool pairs = channels % 2 == 0 && x_stride % 2 == 0 && out_stride % 2 == 0 &&
                     ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(out)) & 7) == 0;
#define VX_CONV_LAUNCH(T, V)                                                                                           \
  launch_conv_act<T, V>(x, x_stride, channels, taps, w_t, bias, state, state_stride, out, out_stride, q_start, q_len, \
                        seq_slots, num_seqs, longest, act, stream)
  if (dtype == VX_DTYPE_F32) {
    if (pairs) VX_CONV_LAUNCH(float, 2);
    else VX_CONV_LAUNCH(float, 1);
  } else {
    if (pairs) VX_CONV_LAUNCH(__nv_bfloat16, 2);
    else VX_CONV_LAUNCH(__nv_bfloat16, 1);
  }
#undef VX_CONV_LAUNCH
  return (int)cudaGetLastError();
}

template <typename T, int L, int NS, bool VEC>
static int launch_selective_scan(const SelectiveScan& p, int num_seqs, int num_tokens, cudaStream_t stream) {
  constexpr int THREADS = ss_scan_threads(L) + SS_GROUPS * SS_HELPERS, CB = ss_scan_threads(L) / L, NP = L * NS, TC = ss_tile(L, NP);
  constexpr size_t smem = sizeof(float) * SS_GROUPS * (3 * TC * CB + 2 * TC * NP);
  static bool configured = false;
  if (smem > 48 * 1024 && !configured) {
    cudaError_t e = cudaFuncSetAttribute(selective_scan_kernel<T, L, NS, 0, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(selective_scan_kernel<T, L, NS, 1, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(selective_scan_kernel<T, L, NS, 2, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const int blocks = (p.inner + CB - 1) / CB;
  if (p.chunk <= 0 || num_tokens <= p.chunk) {
    launch_pdl(selective_scan_kernel<T, L, NS, 0, VEC>, dim3(blocks, num_seqs), dim3(THREADS), smem, stream, p);
    return (int)cudaGetLastError();
  }
  const dim3 grid(blocks, num_seqs, (num_tokens + p.chunk - 1) / p.chunk);
  launch_pdl(selective_scan_kernel<T, L, NS, 1, VEC>, grid, dim3(THREADS), smem, stream, p);
  int cblocks = (int)(((size_t)p.inner * p.N + 255) / 256);
  if (cblocks > 148 * 8) cblocks = 148 * 8;
  launch_pdl(selective_combine_kernel<T>, dim3(cblocks, num_seqs), dim3(256), 0, stream, p);
  launch_pdl(selective_scan_kernel<T, L, NS, 2, VEC>, grid, dim3(THREADS), smem, stream, p);
  return (int)cudaGetLastError();
}

template <typename T, int L, int NS>
static int choose_selective_scan(const SelectiveScan& p, int num_seqs, int num_tokens, cudaStream_t stream) {
  if constexpr (NS == 4 && L <= 16) {
    // Channels in pairs, B and C in sixteen-byte packs: sizes, pitches and pointers allow it.
    const int pack = 16 / (int)sizeof(T);
    const bool vec = p.N % pack == 0 && p.inner % 2 == 0 && p.x_stride % 2 == 0 && p.z_stride % 2 == 0 && p.out_stride % 2 == 0 &&
                     p.dt_stride % 2 == 0 && p.bc_stride % pack == 0 && (reinterpret_cast<uintptr_t>(p.bc) & 15) == 0 &&
                     ((reinterpret_cast<uintptr_t>(p.x) | reinterpret_cast<uintptr_t>(p.z) | reinterpret_cast<uintptr_t>(p.out) |
                       reinterpret_cast<uintptr_t>(p.dt)) & 7) == 0;
    if (vec) return launch_selective_scan<T, L, NS, true>(p, num_seqs, num_tokens, stream);
  }
  return launch_selective_scan<T, L, NS, false>(p, num_seqs, num_tokens, stream);
}

// The most states of a channel the kernels hold.
VX_API int vx_selective_max_state() { return 512; }

// Channels of one block of the scan, for the caller's choice of chunks.
VX_API int vx_selective_block_channels(int N) {
  const int L = N <= 4 ? 1 : N <= 8 ? 2 : N <= 16 ? 4 : N <= 32 ? 8 : N <= 64 ? 16 : 32;
  return ss_scan_threads(L) / L;
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
                             int num_tokens, int* status, cudaStream_t stream) {
  if (num_seqs <= 0 || num_tokens <= 0) return 0;
  if (inner <= 0 || N <= 0 || N > 512 || num_seqs > 65535) return (int)cudaErrorInvalidValue;
  if (chunk_states == nullptr || chunk_dt == nullptr) chunk = 0;
  const SelectiveScan p = {x, x_stride, dt, dt_stride, dt_bias, a2, bc, bc_stride, d_skip, z, z_stride, out, out_stride,
                           state, state_stride, inner, N, chunk, q_start, q_len, seq_slots, chunk_states, chunk_dt,
                           status};
#define VX_SCAN_CALL(L, NS) VX_BY_DTYPE(dtype, return (choose_selective_scan<T, L, NS>(p, num_seqs, num_tokens, stream)))
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
                           state, state_stride, inner, N, 0, q_start, nullptr, seq_slots, nullptr, nullptr, nullptr};
#define VX_STEP_CALL(L, NS) VX_BY_DTYPE(dtype, return (launch_selective_step<T, L, NS>(p, low, w_dt, rank, num_seqs, stream)))
  VX_SELECTIVE_SIZES(VX_STEP_CALL)
#undef VX_STEP_CALL
}
