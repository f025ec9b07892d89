// The gated delta rule (delta_rule.cuh) for the two ends of a step's length.
//
//   gated_delta_step_kernel       one token of the gated delta rule per sequence in one launch: what
//                                 prepare makes, the state's update, the read-out, its norm and gate
//   gated_delta_chunk_kernel, gated_delta_pass_kernel
//                                 the gated delta rule over long portions in chunks of 32 tokens: what a
//                                 chunk does to any state, made for all chunks side by side, then the
//                                 states in order, as small matrix products
//
// What the recurrence reads and keeps is float32 whatever the storage type of the projections.
#include "common.cuh"
#include "delta_rule.cuh"
#include "recurrent.cuh"

namespace vx {

// One token of every sequence (q_len 1), a block per (sequence, head): convolutions, unit vectors,
// decay and write strength as above, the state's update, the read-out, its RMS norm over the head
// (`norm_eps`, weight norm_w [Dv]) and the gate (gate_act: 1 sigmoid, 2 silu).  The decay's logits and
// the gate's are columns of the step's rows, or (rank_a, rank_g > 0) come out of the second half of a
// low-rank pair here: a_up [heads * Dk, rank_a] and g_up [heads * Dv, rank_g] times columns of the rows.
// RL lanes share a column of S (Dk floats in a row), NCH chunks of four rows each; both sums of a column
// (what k reads out of the decayed state, and what q reads) are made in one pass over the old state:
// S_new^T q = (g S)^T q + change (k . q).
struct GatedDeltaOut {
  const void* gate;
  long long gate_stride;
  const void* a_up;
  const void* g_up;
  int rank_a, rank_g;
  const float* norm_w;
  float norm_eps;
  int gate_act;
  void* out;
  long long out_stride;
};

constexpr int GD_THREADS = 256;

// Three sums over the block at once.
__device__ __forceinline__ void block_sum3(float& a, float& b, float& c, float* scratch /* 32 x 3 floats */) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  a = warp_sum(a);
  b = warp_sum(b);
  c = warp_sum(c);
  if (lane == 0) scratch[3 * warp] = a, scratch[3 * warp + 1] = b, scratch[3 * warp + 2] = c;
  __syncthreads();
  a = b = c = 0.f;
#pragma unroll
  for (int w = 0; w < GD_THREADS / 32; ++w) a += scratch[3 * w], b += scratch[3 * w + 1], c += scratch[3 * w + 2];
}

template <typename T, int FORM, int RL, int NCH, bool VEC>
__global__ void __launch_bounds__(GD_THREADS)
gated_delta_step_kernel(GatedDelta p, GatedDeltaOut o, float* __restrict__ state, long long state_stride,
                        float* __restrict__ ring_out, const int* __restrict__ q_start,
                        const int* __restrict__ seq_slots) {
  extern __shared__ __align__(16) float gd_s[];
  __shared__ float scratch[96];
  constexpr int KD = RL * NCH * 4, WARPS = GD_THREADS / 32;
  const int Dk = p.Dk, Dv = p.Dv, group = p.heads / p.kv_heads;
  float* w_s = gd_s;            // [KD] decay
  float* k_s = w_s + KD;        // [KD] key, convolved and activated
  float* q_s = k_s + KD;        // [KD] query
  float* low_a = q_s + KD;      // [rank_a, padded to 4]
  float* low_g = low_a + (o.rank_a + 3) / 4 * 4;
  float* v_s = low_g + (o.rank_g + 3) / 4 * 4;  // [Dv] values, then the read-out
  float* gate_s = v_s + Dv;     // [Dv]
  allow_dependents();
  const int h = blockIdx.x, seq = blockIdx.y, kh = h / group;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int slot = seq_slots[seq], row = q_start[seq];
  float* S = state + (size_t)slot * state_stride + (size_t)h * Dv * Dk;
  // The state's lines are asked for while the projection before this kernel still runs.
  for (size_t at = (size_t)tid * 32; at < (size_t)Dk * Dv; at += (size_t)GD_THREADS * 32)
    asm volatile("prefetch.global.L2 [%0];" ::"l"(S + at));
  grid_dependency_wait();
  const int pos = p.positions[row];
  // This warp's first columns of the state, on their way while the vectors are made.
  constexpr int COLS = 32 / RL;                // columns of a warp at a time
  constexpr int UN = NCH >= 4 ? 4 : 16 / NCH;  // of them under way together
  const int sub = lane % RL, sub_col = lane / RL;
  float s[UN][NCH * 4];
  auto load_state = [&](int base) {
#pragma unroll
    for (int u = 0; u < UN; ++u) {
      const int col = base + u * WARPS * COLS + sub_col;
      const float* src = S + (size_t)col * Dk;
#pragma unroll
      for (int c = 0; c < NCH; ++c) {
        const int ch = (c * RL + sub) * 4;
        if (VEC) {
          const float4 v = (col < Dv && ch < Dk) ? *reinterpret_cast<const float4*>(src + ch) : make_float4(0.f, 0.f, 0.f, 0.f);
          s[u][4 * c] = v.x; s[u][4 * c + 1] = v.y; s[u][4 * c + 2] = v.z; s[u][4 * c + 3] = v.w;
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) s[u][4 * c + e] = (col < Dv && ch + e < Dk) ? src[ch + e] : 0.f;
        }
      }
    }
  };
  load_state(warp * COLS);
  const int keys = p.kv_heads * Dk, C = 2 * keys + p.heads * Dv;
  const float* ring = p.ring + (size_t)slot * p.ring_stride;
  float* ring_now = ring_out + (size_t)slot * p.ring_stride + (size_t)ring_row(pos, p.taps) * C;
  const T* x_row = (const T*)p.x + (size_t)row * p.x_stride;
  const T* a_row = (const T*)p.a + (size_t)row * p.a_stride;
  const T* gate_row = (const T*)o.gate + (size_t)row * o.gate_stride;
  const bool owns_keys = h % group == 0;
  for (int j = tid; j < o.rank_a; j += GD_THREADS) low_a[j] = to_float(a_row[j]);
  for (int j = tid; j < o.rank_g; j += GD_THREADS) low_g[j] = to_float(gate_row[j]);
  // q, k and v in turns over the threads.
  for (int j = tid; j < 2 * KD + Dv; j += GD_THREADS) {
    const bool is_v = j >= 2 * KD, is_k = !is_v && j >= KD;
    const int ch = is_v ? j - 2 * KD : is_k ? j - KD : j;
    float v = 0.f;
    if (is_v || ch < Dk) {
      const int c = is_v ? 2 * keys + h * Dv + ch : (is_k ? keys : 0) + kh * Dk + ch;
      v = conv_at<T>(p, ring, C, c, row, 0, pos);
      if (p.taps > 1 && (is_v || owns_keys)) ring_now[c] = to_float(x_row[c]);
    }
    (is_v ? v_s : is_k ? k_s : q_s)[ch] = v;
  }
  const float rate = -expf(p.a_log[h]);
  const float beta = sq_sigmoid(to_float(((const T*)p.b)[(size_t)row * p.b_stride + h]));
  float g = 1.f;
  if (FORM == DR_HEAD) g = expf(rate * sq_softplus(to_float(a_row[h]) + p.dt_bias[h]));
  __syncthreads();
  if (FORM == DR_CHANNEL) {
    if (o.rank_a > 0) {
      const bool packs = o.rank_a % (16 / (int)sizeof(T)) == 0;
      rank_product<T, GD_THREADS / 32>((const T*)o.a_up + (size_t)h * Dk * o.rank_a, low_a, o.rank_a, Dk, packs, w_s);
    }
  }
  if (o.rank_g > 0) {
    const bool packs = o.rank_g % (16 / (int)sizeof(T)) == 0;
    rank_product<T, GD_THREADS / 32>((const T*)o.g_up + (size_t)h * Dv * o.rank_g, low_g, o.rank_g, Dv, packs, gate_s);
  } else {
    for (int c = tid; c < Dv; c += GD_THREADS) gate_s[c] = to_float(gate_row[(size_t)h * Dv + c]);
  }
  // The unit vectors' lengths, and k . q, from the vectors as they stand.
  float sq = 0.f, sk = 0.f, kq = 0.f;
  for (int ch = tid; ch < KD; ch += GD_THREADS) {
    const float kv = k_s[ch], qv = q_s[ch];
    sq = fmaf(qv, qv, sq);
    sk = fmaf(kv, kv, sk);
    kq = fmaf(kv, qv, kq);
  }
  block_sum3(sq, sk, kq, scratch);  // (also: the second products' rows are complete)
  const float iq = p.q_scale / sqrtf(sq + p.unit_eps), ik = 1.0f / sqrtf(sk + p.unit_eps);
  kq *= iq * ik;
  // This lane's rows of the vectors.
  float wr[NCH * 4], kr[NCH * 4], qr[NCH * 4];
#pragma unroll
  for (int c = 0; c < NCH; ++c)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int ch = (c * RL + sub) * 4 + e;
      wr[4 * c + e] = g;
      if (FORM == DR_CHANNEL) {
        const float z = ch < Dk ? (o.rank_a > 0 ? w_s[ch] : to_float(a_row[h * Dk + ch])) + p.dt_bias[h * Dk + ch] : 0.f;
        wr[4 * c + e] = expf(rate * sq_softplus(z));
      }
      kr[4 * c + e] = k_s[ch] * ik;
      qr[4 * c + e] = q_s[ch] * iq;
    }
  for (int base = warp * COLS; base < Dv; base += WARPS * COLS * UN) {
    if (base != warp * COLS) load_state(base);
#pragma unroll
    for (int u = 0; u < UN; ++u) {
      const int col = base + u * WARPS * COLS + sub_col;
      // Read before the shuffles, replaced after them: every lane of the column has its value by then.
      const float value = col < Dv ? v_s[col] : 0.f;
      float read = 0.f, out = 0.f;
#pragma unroll
      for (int e = 0; e < NCH * 4; ++e) {
        s[u][e] *= wr[e];
        read = fmaf(s[u][e], kr[e], read);
        out = fmaf(s[u][e], qr[e], out);
      }
#pragma unroll
      for (int off = RL / 2; off > 0; off >>= 1) {
        read += __shfl_xor_sync(0xffffffffu, read, off);
        out += __shfl_xor_sync(0xffffffffu, out, off);
      }
      if (col < Dv) {
        const float change = beta * (value - read);
        float* dst = S + (size_t)col * Dk;
#pragma unroll
        for (int c = 0; c < NCH; ++c) {
          const int ch = (c * RL + sub) * 4;
#pragma unroll
          for (int e = 0; e < 4; ++e) s[u][4 * c + e] = fmaf(kr[4 * c + e], change, s[u][4 * c + e]);
          if (VEC) {
            if (ch < Dk)
              *reinterpret_cast<float4*>(dst + ch) = make_float4(s[u][4 * c], s[u][4 * c + 1], s[u][4 * c + 2], s[u][4 * c + 3]);
          } else {
#pragma unroll
            for (int e = 0; e < 4; ++e)
              if (ch + e < Dk) dst[ch + e] = s[u][4 * c + e];
          }
        }
        if (sub == 0) v_s[col] = fmaf(change, kq, out);
      }
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < Dv; c += GD_THREADS) ss = fmaf(v_s[c], v_s[c], ss);
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)Dv + o.norm_eps);
  T* dst = (T*)o.out + (size_t)row * o.out_stride + (size_t)h * Dv;
  for (int c = tid; c < Dv; c += GD_THREADS) {
    const float z = gate_s[c];
    dst[c] = from_float<T>(v_s[c] * inv * o.norm_w[c] * (o.gate_act == 2 ? sq_silu(z) : sq_sigmoid(z)));
  }
}

// ---------------------------------------------------------------------------------------------
// Long portions of the gated delta rule, in chunks of GC = 32 tokens (key sizes up to 128).  With S_0 the
// state a chunk starts from, P_(s->t) the product of the decays of tokens s + 1 .. t (per state row), and
// u_t the corrected, scaled value that token t writes (S_t = g_t S_(t-1) + k_t u_t^T),
//     S_t = P_(0->t) S_0 + sum_(s <= t) P_(s->t) k_s u_s^T
//     u_t + beta_t sum_(s < t) A_ts u_s = beta_t (v_t - (P_(0->t) k_t)^T S_0),   A_ts = k_t^T P_(s->t) k_s
//     o_t = (P_(0->t) q_t)^T S_0 + sum_(s <= t) B_ts u_s,                        B_ts = q_t^T P_(s->t) k_s
// (the chunkwise form of Yang et al., "Parallelizing Linear Transformers with the Delta Rule over Sequence
// Length", with decays).  The unit lower triangular system has a right side that is affine in S_0, so
//     U = U0 - W S_0;    O = Qt S_0 + B U;    S_GC = P_(0->GC) S_0 + Kh^T U
// with U0 and W its solutions for beta v and beta P k, Qt = P q, Kh_s = P_(s->GC) k_s.
//
// gated_delta_chunk_kernel makes W, Qt, Kh, U0, B and P of every (chunk, head), a block each: nothing in it
// waits for another chunk.  Decays enter as running products, each at most 1, so nothing overflows however
// strong they are.  gated_delta_pass_kernel walks a sequence's chunks in order, a block per (GP_COLS value
// columns, head, sequence): the state's columns never meet.  All of it float32, in a fixed order; a token's
// result depends, within rounding, on where its chunk began.
//
// A chunk's record: [W | Qt | Kh] of [GC][KD] floats each (KD: Dk padded with zeros to a multiple of 32), B
// [GC][GC + 4], P [KD]; then U0 in tiles of [GC][GP_COLS].  Chunk c of sequence s lies at place q_start[s] /
// GC + s + c.
constexpr int GC = 32, GP_COLS = 16, GP_THREADS = 256, GC_BP = GC + 4;
constexpr int GD_CHUNKED_MAX_DK = 128;

__host__ __device__ inline size_t gc_main_floats(int KD) { return (size_t)3 * GC * KD + GC * GC_BP + KD; }
__host__ __device__ inline size_t gc_record_floats(int KD, int Dv) {
  return gc_main_floats(KD) + (size_t)((Dv + GP_COLS - 1) / GP_COLS) * GC * GP_COLS;
}

// Sums 32 values over the warp's lanes, value i ending in lane i.
__device__ __forceinline__ float warp_transpose_sum(float (&v)[32], int lane) {
#pragma unroll
  for (int off = 16; off > 0; off >>= 1) {
    const bool upper = (lane & off) != 0;
#pragma unroll
    for (int i = 0; i < off; ++i) {
      const float give = upper ? v[i] : v[i + off];
      const float keep = upper ? v[i + off] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, off);
    }
  }
  return v[0];
}

// Channel ch's convolution inputs for the portion's tokens i0 .. i0 + 7 (at most four taps; those at or behind
// `end`: 0); pos0 is the position of the portion's first token.
template <typename T>
__device__ __forceinline__ void conv_inputs(const GatedDelta& p, const float* __restrict__ ring, int C, int ch, int start,
                                            int i0, int end, int pos0, float (&v)[11]) {
  const T* x = (const T*)p.x + ch;
  T raw[11];
  // Loads from valid places, used or not: behind conditions they would be waited for one by one.
#pragma unroll
  for (int u = 0; u < 11; ++u) raw[u] = x[(size_t)(start + min(max(i0 - 3 + u, 0), end - 1)) * p.x_stride];
#pragma unroll
  for (int u = 0; u < 11; ++u) v[u] = i0 - 3 + u < end ? to_float(raw[u]) : 0.f;
  if (i0 < 3) {
#pragma unroll
    for (int u = 0; u < 3; ++u) {
      const int i = i0 - 3 + u;
      if (i < 0) v[u] = pos0 + i >= 0 && -i < p.taps ? ring[(size_t)ring_row(pos0 + i, p.taps) * C + ch] : 0.f;
    }
  }
}

// The activated convolution from those inputs.
template <typename T>
__device__ __forceinline__ void conv_outputs(const GatedDelta& p, int C, int ch, int i0, int end, const float (&v)[11],
                                             float (&out)[8]) {
  float w[4];
#pragma unroll
  for (int k = 0; k < 4; ++k) w[k] = 3 - k < p.taps ? p.conv_w[(size_t)(p.taps - 4 + k) * C + ch] : 0.f;
#pragma unroll
  for (int u = 0; u < 8; ++u) {
    float acc = 0.f;
#pragma unroll
    for (int k = 0; k < 4; ++k) acc = fmaf(w[k], v[u + k], acc);
    out[u] = i0 + u < end ? conv_silu<T>(acc) : 0.f;
  }
}

template <typename T, int FORM, int NV>
__global__ void __launch_bounds__(GP_THREADS, 3)
gated_delta_chunk_kernel(GatedDelta p, float* __restrict__ records, const int* __restrict__ q_start,
                         const int* __restrict__ q_len, const int* __restrict__ seq_slots) {
  constexpr int KD = 32 * NV, KP = KD + 4;
  extern __shared__ __align__(16) float gc_s[];
  float* k_s = gc_s;               // [GC][KP] unit keys
  float* q_s = k_s + GC * KP;      // [GC][KP] scaled unit queries
  float* g_s = q_s + GC * KP;      // [GC][KP] decays (DR_CHANNEL), or [GC] (DR_HEAD)
  float* m_s = g_s + (FORM == DR_CHANNEL ? GC * KP : GC);  // [GC][GC_BP] beta_i A_ij
  float* beta_s = m_s + GC * GC_BP;                        // [GC]
  const int tiles = (p.Dv + GP_COLS - 1) / GP_COLS, cols = KD + tiles * GP_COLS;
  float* v_s = beta_s + GC;                                // [GC][tiles * GP_COLS] values
  allow_dependents();
  const int chunk = blockIdx.x, h = blockIdx.y, seq = blockIdx.z;
  grid_dependency_wait();
  const int n_all = q_len[seq], first = chunk * GC;
  if (first >= n_all) return;
  const int n = min(GC, n_all - first), start = q_start[seq];
  const int Dk = p.Dk, Dv = p.Dv, kh = h / (p.heads / p.kv_heads);
  const int keys = p.kv_heads * Dk, C = 2 * keys + p.heads * Dv;
  const float* ring = p.ring + (size_t)seq_slots[seq] * p.ring_stride;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int pos0 = p.positions[start];
  const size_t place = (size_t)(start / GC + seq + chunk);
  float* rec = records + (place * p.heads + h) * gc_record_floats(KD, Dv);
  float *w_out = rec, *q_out = rec + GC * KD, *k_out = q_out + GC * KD, *b_out = k_out + GC * KD,
        *p_out = b_out + GC * GC_BP, *u_out = p_out + KD;
  // A token behind the portion's end writes nothing, reads nothing and decays nothing.  Units of eight tokens
  // of one channel: q, k and v in turns over the threads.
  const int v_cols = tiles * GP_COLS, unit_cols = 2 * KD + v_cols, units = (GC / 8) * unit_cols;
  // (Two units of a thread at a time: the second's loads are under way before the first is worked out.)
  auto place_of = [&](int unit, int& i0, int& ch, int& pitch) -> float* {
    i0 = unit / unit_cols * 8;
    const int c = unit % unit_cols;
    const bool is_v = c >= 2 * KD, is_k = !is_v && c >= KD;
    const int d = is_v ? c - 2 * KD : is_k ? c - KD : c;
    ch = d < (is_v ? Dv : Dk) ? (is_v ? 2 * keys + h * Dv + d : (is_k ? keys : 0) + kh * Dk + d) : -1;
    pitch = is_v ? v_cols : KP;
    return is_v ? v_s + i0 * v_cols + d : (is_k ? k_s : q_s) + i0 * KP + d;
  };
  if (p.taps <= 4) {
    for (int unit = tid; unit < units; unit += 2 * GP_THREADS) {
      float in[2][11], made[8];
      int i0[2], ch[2], pitch[2];
      float* dst[2];
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        ch[q] = -1;
        if (unit + q * GP_THREADS < units) dst[q] = place_of(unit + q * GP_THREADS, i0[q], ch[q], pitch[q]);
        else dst[q] = nullptr;
        if (ch[q] >= 0) conv_inputs<T>(p, ring, C, ch[q], start, first + i0[q], n_all, pos0, in[q]);
      }
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        if (dst[q] == nullptr) continue;
        if (ch[q] >= 0) conv_outputs<T>(p, C, ch[q], first + i0[q], n_all, in[q], made);
#pragma unroll
        for (int u = 0; u < 8; ++u) dst[q][u * pitch[q]] = ch[q] >= 0 ? made[u] : 0.f;
      }
    }
  } else {
#pragma unroll 1
    for (int unit = tid; unit < units; unit += GP_THREADS) {
      int i0, ch, pitch;
      float* dst = place_of(unit, i0, ch, pitch);
#pragma unroll 1
      for (int u = 0; u < 8; ++u) {
        const int at = first + i0 + u;
        dst[u * pitch] = ch >= 0 && at < n_all ? conv_at<T>(p, ring, C, ch, start + at, at, pos0 + at) : 0.f;
      }
    }
  }
  const float rate = -expf(p.a_log[h]);
  if (FORM == DR_CHANNEL) {
    for (int unit = tid; unit < (GC / 8) * KD; unit += GP_THREADS) {
      const int i0 = unit / KD * 8, d = unit % KD;
      T z[8];
      const int at = h * Dk + min(d, Dk - 1);
#pragma unroll
      for (int u = 0; u < 8; ++u)
        z[u] = ((const T*)p.a)[(size_t)(start + first + min(i0 + u, n - 1)) * p.a_stride + at];
      const float bias = p.dt_bias[at];
#pragma unroll
      for (int u = 0; u < 8; ++u)
        g_s[(i0 + u) * KP + d] = i0 + u < n && d < Dk ? expf(rate * sq_softplus(to_float(z[u]) + bias)) : 1.f;
    }
  }
  if (tid < GC) {
    const size_t row = (size_t)(start + first + tid);
    beta_s[tid] = tid < n ? sq_sigmoid(to_float(((const T*)p.b)[row * p.b_stride + h])) : 0.f;
    if (FORM == DR_HEAD)
      g_s[tid] = tid < n ? expf(rate * sq_softplus(to_float(((const T*)p.a)[row * p.a_stride + h]) + p.dt_bias[h])) : 1.f;
  }
  __syncthreads();
  for (int i = warp; i < GC; i += GP_THREADS / 32) {
    float sq = 0.f, sk = 0.f;
#pragma unroll
    for (int e = 0; e < NV; ++e) {
      const float qv = q_s[i * KP + lane + 32 * e], kv = k_s[i * KP + lane + 32 * e];
      sq = fmaf(qv, qv, sq);
      sk = fmaf(kv, kv, sk);
    }
    const float iq = p.q_scale / sqrtf(warp_sum(sq) + p.unit_eps), ik = 1.0f / sqrtf(warp_sum(sk) + p.unit_eps);
#pragma unroll
    for (int e = 0; e < NV; ++e) {
      q_s[i * KP + lane + 32 * e] *= iq;
      k_s[i * KP + lane + 32 * e] *= ik;
    }
  }
  __syncthreads();
  // Column j of A and B: k_j carried forward by the decays, a warp per column; sixteen rows' sums at a time.
  for (int jj = warp; jj < GC; jj += GP_THREADS / 32) {
    const int j = (jj & 8) ? GC - 1 - (jj ^ 8) % GC : jj;  // a warp's four columns: two early ones, two late ones
    float r[NV];
#pragma unroll
    for (int e = 0; e < NV; ++e) r[e] = k_s[j * KP + lane + 32 * e];
    float carried = 1.f;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      float v[32];
      if (half * 16 + 15 < j) {
        // Rows before the column: zeros.
        if (lane < 16) m_s[(half * 16 + lane) * GC_BP + j] = 0.f;
        else b_out[(half * 16 + lane - 16) * GC_BP + j] = 0.f;
        continue;
      }
#pragma unroll
      for (int ii = 0; ii < 16; ++ii) {
        const int i = half * 16 + ii;
        float a = 0.f, b = 0.f;
        if (i >= j) {
          if (i > j) {
            if (FORM == DR_HEAD) carried *= g_s[i];
            else {
#pragma unroll
              for (int e = 0; e < NV; ++e) r[e] *= g_s[i * KP + lane + 32 * e];
            }
          }
#pragma unroll
          for (int e = 0; e < NV; ++e) {
            a = fmaf(k_s[i * KP + lane + 32 * e], r[e], a);
            b = fmaf(q_s[i * KP + lane + 32 * e], r[e], b);
          }
          if (FORM == DR_HEAD) a *= carried, b *= carried;
          if (i == j) a = 0.f;
        }
        v[ii] = a;
        v[16 + ii] = b;
      }
      const float sum = warp_transpose_sum(v, lane);
      const int i = half * 16 + (lane & 15);
      if (lane < 16) m_s[i * GC_BP + j] = beta_s[i] * sum;
      else b_out[i * GC_BP + j] = sum;
    }
  }
  __syncthreads();
  // The triangular system, a thread per right side: the key columns (W), then the value columns (U0).
  for (int col = tid; col < cols; col += GP_THREADS) {
    const bool is_key = col < KD;
    const int c = col - KD;
    if (is_key) {
      float product = 1.f, suffix = 1.f;
#pragma unroll 8
      for (int i = 0; i < GC; ++i) {
        product *= FORM == DR_HEAD ? g_s[i] : g_s[i * KP + col];
        q_out[i * KD + col] = q_s[i * KP + col] * product;
        q_s[i * KP + col] = k_s[i * KP + col] * product;  // the right side, in the place of a query that is done
      }
      p_out[col] = product;
#pragma unroll 8
      for (int i = GC - 1; i >= 0; --i) {
        k_out[i * KD + col] = k_s[i * KP + col] * suffix;
        suffix *= FORM == DR_HEAD ? g_s[i] : g_s[i * KP + col];
      }
    }
    float x[GC];
    const float* rhs = is_key ? q_s + col : v_s + c;
    const int rhs_pitch = is_key ? KP : v_cols;
#pragma unroll
    for (int i = 0; i < GC; ++i) x[i] = beta_s[i] * rhs[i * rhs_pitch];
#pragma unroll
    for (int i = 1; i < GC; ++i) {
      float sum0 = 0.f, sum1 = 0.f, sum2 = 0.f, sum3 = 0.f;
#pragma unroll
      for (int j = 0; j < i; j += 4) {
        // (Entries on and behind the diagonal are zero.)
        const float4 m = *reinterpret_cast<const float4*>(m_s + i * GC_BP + j);
        sum0 = fmaf(m.x, x[j], sum0);
        if (j + 1 < i) sum1 = fmaf(m.y, x[j + 1], sum1);
        if (j + 2 < i) sum2 = fmaf(m.z, x[j + 2], sum2);
        if (j + 3 < i) sum3 = fmaf(m.w, x[j + 3], sum3);
      }
      x[i] -= (sum0 + sum1) + (sum2 + sum3);
    }
    float* dst = is_key ? w_out + col : u_out + (size_t)(c / GP_COLS) * GC * GP_COLS + c % GP_COLS;
    const int pitch = is_key ? KD : GP_COLS;
#pragma unroll
    for (int i = 0; i < GC; ++i) dst[i * pitch] = x[i];
  }
}

// Warps 0-3 make U and carry the state (a thread: four rows of four columns, in registers; a copy in shared
// memory for the products that read it), warps 4-7 make O.  Records come in by bulk copies, two stages.
template <int NV>
__global__ void __launch_bounds__(GP_THREADS)
gated_delta_pass_kernel(const float* __restrict__ records, float* __restrict__ state, long long state_stride,
                        float* __restrict__ out, long long out_stride, int heads, int Dk, int Dv,
                        const int* __restrict__ q_start, const int* __restrict__ q_len,
                        const int* __restrict__ seq_slots, ConvRing ring, int* status) {
  constexpr int KD = 32 * NV, SP = KD + 4;
  constexpr int MAIN = 3 * GC * KD + GC * GC_BP + KD, STAGE = MAIN + GC * GP_COLS;
  extern __shared__ __align__(16) float gp_s[];
  float* S_s = gp_s + 2 * STAGE;             // [GP_COLS][SP]
  float* U_s = S_s + GP_COLS * SP;           // [GC][GP_COLS + 4]
  constexpr int UP = GP_COLS + 4;
  __shared__ __align__(8) unsigned long long bars[2];
  const int tile = blockIdx.x, h = blockIdx.y, seq = blockIdx.z;
  const int n = q_len[seq];
  if (n <= 0) {
    allow_dependents();
    return;
  }
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int start = q_start[seq], slot = seq_slots[seq], chunks = (n + GC - 1) / GC;
  const uint32_t bar0 = smem_u32(&bars[0]), bar1 = smem_u32(&bars[1]);
  if (tid == 0) {
    mbar_init(bar0, 1);
    mbar_init(bar1, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  __syncthreads();
  grid_dependency_wait();
  const size_t record = gc_record_floats(KD, Dv);
  const float* base = records + ((size_t)(start / GC + seq) * heads + h) * record;
  auto issue = [&](int c) {
    const uint32_t bar = (c & 1) ? bar1 : bar0;
    const float* src = base + (size_t)c * heads * record;
    float* dst = gp_s + (c & 1) * STAGE;
    mbar_expect_tx(bar, (uint32_t)STAGE * 4u);
    bulk_copy_g2s(smem_u32(dst), src, (uint32_t)MAIN * 4u, bar);
    bulk_copy_g2s(smem_u32(dst + MAIN), src + MAIN + (size_t)tile * GC * GP_COLS, (uint32_t)(GC * GP_COLS) * 4u, bar);
  };
  if (tid == 0) {
    issue(0);
    if (chunks > 1) issue(1);
  }
  if (ring.x != nullptr && tile == 0) {
    if (ring.dtype == VX_DTYPE_F32) ring_write_last<float>(ring, slot, start, n, h);
    else ring_write_last<__nv_bfloat16>(ring, slot, start, n, h);
  }
  float* st = state + (size_t)slot * state_stride + (size_t)h * Dv * Dk;
  const int k0 = lane * 4, my_cols = (warp & 3) * 4;  // the state's share of a thread of warps 0-3
  const bool carries = warp < 4 && k0 < KD;
  float S[4][4];
#pragma unroll
  for (int c = 0; c < 4; ++c)
#pragma unroll
    for (int e = 0; e < 4; ++e) S[c][e] = 0.f;
  if (carries) {
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const int col = tile * GP_COLS + my_cols + c;
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (col < Dv && k0 + e < Dk) S[c][e] = st[(size_t)col * Dk + k0 + e];
      *reinterpret_cast<float4*>(S_s + (my_cols + c) * SP + k0) = make_float4(S[c][0], S[c][1], S[c][2], S[c][3]);
    }
  }
  __syncthreads();
  // The product [W; Qt] S: eight rows by four columns a thread, the inner size dealt to eight lanes.
  const int kg = lane & 7, c0 = (lane >> 3) * 4;
  for (int chunk = 0; chunk < chunks; ++chunk) {
    const float* buf = gp_s + (chunk & 1) * STAGE;
    mbar_wait((chunk & 1) ? bar1 : bar0, (uint32_t)(chunk >> 1) & 1u, status);
    float acc[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) acc[i] = 0.f;
    const float* rows = buf + (size_t)warp * 8 * KD + 4 * kg;  // W's 32 rows, then Qt's
#pragma unroll
    for (int step = 0; step < NV; ++step) {
      float4 sv[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) sv[c] = *reinterpret_cast<const float4*>(S_s + (c0 + c) * SP + 4 * kg + 32 * step);
#pragma unroll
      for (int r = 0; r < 8; ++r) {
        const float4 wv = *reinterpret_cast<const float4*>(rows + r * KD + 32 * step);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          acc[4 * r + c] = fmaf(wv.x, sv[c].x, acc[4 * r + c]);
          acc[4 * r + c] = fmaf(wv.y, sv[c].y, acc[4 * r + c]);
          acc[4 * r + c] = fmaf(wv.z, sv[c].z, acc[4 * r + c]);
          acc[4 * r + c] = fmaf(wv.w, sv[c].w, acc[4 * r + c]);
        }
      }
    }
    // Over the eight lanes, lane kg ending with row kg of the eight.
#pragma unroll
    for (int off = 4; off > 0; off >>= 1) {
      const bool upper = (kg & off) != 0;
#pragma unroll
      for (int i = 0; i < 4 * off; ++i) {
        const float give = upper ? acc[i] : acc[i + 4 * off];
        const float keep = upper ? acc[i + 4 * off] : acc[i];
        acc[i] = keep + __shfl_xor_sync(0xffffffffu, give, off);
      }
    }
    const int row = (warp & 3) * 8 + kg;
    if (warp < 4) {
      const float4 u0 = *reinterpret_cast<const float4*>(buf + MAIN + row * GP_COLS + c0);
      *reinterpret_cast<float4*>(U_s + row * UP + c0) = make_float4(u0.x - acc[0], u0.y - acc[1], u0.z - acc[2], u0.w - acc[3]);
    }
    __syncthreads();  // U is there, and everybody has read the state
    if (warp < 4) {
      if (carries) {
        const float* kh = buf + 2 * GC * KD + k0;
        const float4 pv = *reinterpret_cast<const float4*>(buf + 3 * GC * KD + GC * GC_BP + k0);
#pragma unroll
        for (int c = 0; c < 4; ++c) S[c][0] *= pv.x, S[c][1] *= pv.y, S[c][2] *= pv.z, S[c][3] *= pv.w;
#pragma unroll 8
        for (int i = 0; i < GC; ++i) {
          const float4 kv = *reinterpret_cast<const float4*>(kh + i * KD);
          const float4 uv = *reinterpret_cast<const float4*>(U_s + i * UP + my_cols);
          const float u[4] = {uv.x, uv.y, uv.z, uv.w};
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            S[c][0] = fmaf(kv.x, u[c], S[c][0]);
            S[c][1] = fmaf(kv.y, u[c], S[c][1]);
            S[c][2] = fmaf(kv.z, u[c], S[c][2]);
            S[c][3] = fmaf(kv.w, u[c], S[c][3]);
          }
        }
#pragma unroll
        for (int c = 0; c < 4; ++c)
          *reinterpret_cast<float4*>(S_s + (my_cols + c) * SP + k0) = make_float4(S[c][0], S[c][1], S[c][2], S[c][3]);
      }
    } else {
      const float* b = buf + 3 * GC * KD + row * GC_BP;
#pragma unroll
      for (int j = 0; j < GC; j += 4) {
        const float4 bv = *reinterpret_cast<const float4*>(b + j);
        const float bj[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float4 uv = *reinterpret_cast<const float4*>(U_s + (j + e) * UP + c0);
          acc[0] = fmaf(bj[e], uv.x, acc[0]);
          acc[1] = fmaf(bj[e], uv.y, acc[1]);
          acc[2] = fmaf(bj[e], uv.z, acc[2]);
          acc[3] = fmaf(bj[e], uv.w, acc[3]);
        }
      }
      const int token = chunk * GC + row;
      if (token < n) {
        float* dst = out + (size_t)(start + token) * out_stride + (size_t)h * Dv + tile * GP_COLS + c0;
#pragma unroll
        for (int c = 0; c < 4; ++c)
          if (tile * GP_COLS + c0 + c < Dv) dst[c] = acc[c];
      }
    }
    __syncthreads();  // the state is the next chunk's, and the stage may be filled again
    if (tid == 0 && chunk + 2 < chunks) issue(chunk + 2);
  }
  allow_dependents();
  if (carries) {
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const int col = tile * GP_COLS + my_cols + c;
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (col < Dv && k0 + e < Dk) st[(size_t)col * Dk + k0 + e] = S[c][e];
    }
  }
}

}  // namespace vx

using namespace vx;

template <typename T, int FORM, int NV>
static int launch_gated_delta_chunks(const GatedDelta& p, float* records, float* state, long long state_stride,
                                     float* out, long long out_stride, const int* q_start, const int* q_len,
                                     const int* seq_slots, int num_seqs, int num_tokens, const ConvRing& ring, int* status,
                                     cudaStream_t stream) {
  constexpr int KD = 32 * NV, KP = KD + 4;
  const size_t v_cols = (size_t)(p.Dv + GP_COLS - 1) / GP_COLS * GP_COLS;
  const size_t smem = sizeof(float) * ((size_t)(FORM == DR_CHANNEL ? 3 : 2) * GC * KP + GC * GC_BP + 2 * GC + GC * v_cols);
  if (smem > 200 * 1024) return -1;
  static size_t configured = 0;
  const size_t pass_smem = sizeof(float) * (2 * (gc_main_floats(KD) + GC * GP_COLS) + GP_COLS * (KD + 4) + GC * (GP_COLS + 4));
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(gated_delta_chunk_kernel<T, FORM, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(gated_delta_pass_kernel<NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)pass_smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  launch_pdl(gated_delta_chunk_kernel<T, FORM, NV>, dim3((num_tokens + GC - 1) / GC, p.heads, num_seqs), dim3(GP_THREADS), smem,
             stream, p, records, q_start, q_len, seq_slots);
  launch_pdl(gated_delta_pass_kernel<NV>, dim3((p.Dv + GP_COLS - 1) / GP_COLS, p.heads, num_seqs), dim3(GP_THREADS), pass_smem,
             stream, (const float*)records, state, state_stride, out, out_stride, p.heads, p.Dk, p.Dv, q_start, q_len,
             seq_slots, ring, status);
  return (int)cudaGetLastError();
}

// Floats of scratch `vx_gated_delta_chunks` wants for a step of up to num_tokens tokens of num_seqs sequences; -1: a
// key size it does not take.
VX_API long long vx_gated_delta_chunk_scratch(int num_tokens, int num_seqs, int heads, int Dk, int Dv) {
  if (Dk > GD_CHUNKED_MAX_DK) return -1;
  const int KD = (Dk + 31) / 32 * 32;
  return ((long long)num_tokens / GC + num_seqs + 1) * heads * (long long)gc_record_floats(KD, Dv);
}

// The gated delta rule over each sequence's tokens in chunks of matrix products; arguments as above.
VX_API int vx_gated_delta_chunks(const void* x, int dtype, long long x_stride, const void* b, long long b_stride,
                                 const void* a, long long a_stride, int per_channel, const float* dt_bias,
                                 const float* a_log, const float* conv_w, int taps, float* ring, long long ring_stride,
                                 float* state, long long state_stride, const int* positions, float unit_eps,
                                 float q_scale, int heads, int kv_heads, int Dk, int Dv, float* records,
                                 long long record_floats, float* out, long long out_stride, const int* q_start,
                                 const int* q_len, const int* seq_slots, int num_seqs, int num_tokens, int* status,
                                 cudaStream_t stream) {
  if (num_seqs <= 0 || num_tokens <= 0) return 0;
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads != 0 || Dk <= 0 || Dv <= 0 || taps < 1) return (int)cudaErrorInvalidValue;
  const long long need = vx_gated_delta_chunk_scratch(num_tokens, num_seqs, heads, Dk, Dv);
  if (need < 0) return -1;
  if (record_floats < need || (reinterpret_cast<uintptr_t>(records) & 15) != 0) return (int)cudaErrorInvalidValue;
  const GatedDelta p = {x, x_stride, b, b_stride, a, a_stride, dt_bias, a_log, conv_w, ring, ring_stride, positions,
                        taps, heads, kv_heads, Dk, Dv, unit_eps, q_scale};
  const ConvRing keep = {taps > 1 ? x : nullptr, x_stride, dtype, ring, ring_stride, positions, taps, kv_heads, Dk, Dv, heads};
#define VX_GD_CHUNKS(FORM, NV)                                                                                       \
  VX_BY_DTYPE(dtype, return (launch_gated_delta_chunks<T, FORM, NV>(p, records, state, state_stride, out, out_stride, \
                                                                    q_start, q_len, seq_slots, num_seqs, num_tokens,  \
                                                                    keep, status, stream)))
#define VX_GD_CHUNKS_FORM(NV)                      \
  if (per_channel) { VX_GD_CHUNKS(DR_CHANNEL, NV) } \
  else { VX_GD_CHUNKS(DR_HEAD, NV) }
  if (Dk <= 32) { VX_GD_CHUNKS_FORM(1) }
  if (Dk <= 64) { VX_GD_CHUNKS_FORM(2) }
  if (Dk <= 96) { VX_GD_CHUNKS_FORM(3) }
  VX_GD_CHUNKS_FORM(4)
#undef VX_GD_CHUNKS_FORM
#undef VX_GD_CHUNKS
}

template <typename T, int FORM>
static int launch_gated_delta_step(const GatedDelta& p, const GatedDeltaOut& o, float* state, long long state_stride,
                                   float* ring, const int* q_start, const int* seq_slots, int num_seqs,
                                   cudaStream_t stream) {
  const dim3 grid(p.heads, num_seqs);
  const bool vec = p.Dk % 4 == 0 && state_stride % 4 == 0 && (reinterpret_cast<uintptr_t>(state) & 15) == 0;
#define VX_GD_LAUNCH(RL, NCH, VEC)                                                                                 \
  do {                                                                                                             \
    const size_t smem = sizeof(float) * (3 * (size_t)(RL * NCH * 4) + 2 * (size_t)p.Dv + o.rank_a + o.rank_g + 8); \
    if (smem > 46 * 1024) return -1;                                                                               \
    launch_pdl(gated_delta_step_kernel<T, FORM, RL, NCH, VEC>, grid, dim3(GD_THREADS), smem, stream, p, o, state,  \
               state_stride, ring, q_start, seq_slots);                                                            \
    return (int)cudaGetLastError();                                                                                \
  } while (0)
#define VX_GD_STEP(RL, NCH) \
  if (p.Dk <= RL * NCH * 4) VX_GD_LAUNCH(RL, NCH, true);
  if (!vec) {
    if (p.Dk <= 128) VX_GD_LAUNCH(32, 1, false);
    if (p.Dk <= 512) VX_GD_LAUNCH(32, 4, false);
    return -1;
  }
  VX_GD_STEP(4, 1)
  VX_GD_STEP(8, 1)
  VX_GD_STEP(16, 1)
  VX_GD_STEP(32, 1)
  VX_GD_STEP(32, 2)
  VX_GD_STEP(32, 4)
#undef VX_GD_STEP
#undef VX_GD_LAUNCH
  return -1;
}

// One token of every sequence; -1: sizes the kernel does not take (nothing launched).
VX_API int vx_gated_delta_step(const void* x, int dtype, long long x_stride, const void* b, long long b_stride,
                               const void* a, long long a_stride, int per_channel, const float* dt_bias,
                               const float* a_log, const float* conv_w, int taps, float* ring, long long ring_stride,
                               float* state, long long state_stride, const int* positions, float unit_eps,
                               float q_scale, int heads, int kv_heads, int Dk, int Dv, const void* gate,
                               long long gate_stride, const void* a_up, int rank_a, const void* g_up, int rank_g,
                               const float* norm_w, float norm_eps, int gate_act, void* out, long long out_stride,
                               const int* q_start, const int* seq_slots, int num_seqs, cudaStream_t stream) {
  if (num_seqs <= 0) return 0;
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads != 0 || Dk <= 0 || Dv <= 0 || taps < 1) return (int)cudaErrorInvalidValue;
  const GatedDelta p = {x, x_stride, b, b_stride, a, a_stride, dt_bias, a_log, conv_w, ring, ring_stride, positions,
                        taps, heads, kv_heads, Dk, Dv, unit_eps, q_scale};
  const GatedDeltaOut o = {gate, gate_stride, a_up, g_up, rank_a, rank_g, norm_w, norm_eps, gate_act, out, out_stride};
  if (per_channel) {
    VX_BY_DTYPE(dtype, return (launch_gated_delta_step<T, DR_CHANNEL>(p, o, state, state_stride, ring, q_start, seq_slots,
                                                                      num_seqs, stream)));
  }
  VX_BY_DTYPE(dtype, return (launch_gated_delta_step<T, DR_HEAD>(p, o, state, state_stride, ring, q_start, seq_slots,
                                                                 num_seqs, stream)));
}
