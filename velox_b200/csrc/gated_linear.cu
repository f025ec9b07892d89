// Gated linear attention: a state of key rows by value columns per head, S <- diag(alpha) S + k v^T, read by S^T q,
// with a decay alpha = sigmoid(z)^(1 / tau) per head and key channel.
//
//   gated_linear_step_kernel   one token of every sequence in one launch: the decays (second half of their low-rank
//                              pair included), the state's update, the read-out, its norm and gate; a cluster
//                              of CTAs shares a head's value columns
//   gated_linear_chunk_kernel, gated_linear_pass_kernel
//                              portions in chunks of 32 tokens: what a chunk's queries, keys and decays come to, all
//                              chunks side by side, then the states in order as small matrix products
//
// Decays and their logarithms, S and every sum over it are float32 whatever the storage type.
#include "common.cuh"
#include "recurrent.cuh"

namespace vx {

// q, k, v are columns of the step's rows (`stride` apart): q and k [heads, Dk], v [heads, Dv].
struct GatedLinear {
  const void *q, *k, *v;
  long long stride;
  const float* a_bias;   // [heads * Dk], joins the decay's logits
  float q_scale, decay_scale;  // decay_scale: log2(e) / tau
  int heads, Dk, Dv;
  const int *q_start, *q_len, *seq_slots;
};

// sigmoid(z)^(1 / tau) = 2^(-softplus(-z) log2(e) / tau)
template <typename T>
__device__ __forceinline__ float gate_decay(float z, float decay_scale) {
  return pow2_for<T>(-softplus_for<T>(-z) * decay_scale);
}

// ---------------------------------------------------------------------------------------------
// One token of every sequence (q_len 1).  A cluster of `gridDim.x / heads` CTAs per (head, sequence), a CTA a slice of
// the value columns; the sums of squares of the slices meet through distributed shared memory.  RL lanes share
// a column of S (Dk floats in a row), NCH chunks of four rows each.
struct GatedLinearOut {
  const void* low;        // [tokens, rank]: the pair's inner values
  long long low_stride;
  const void* a_up;       // [heads * Dk, rank]
  int rank;
  const void* gate;       // [tokens, heads * Dv]
  long long gate_stride;
  const float* norm_w;    // [Dv]
  float norm_eps;
  void* out;
  long long out_stride;
  float* state;           // [slots][heads, Dv, Dk]
  long long state_stride;
};

constexpr int GL_THREADS = 256, GL_MAX_CLUSTER = 8;

template <typename T, int RL, int NCH, bool VEC>
__global__ void __launch_bounds__(GL_THREADS) gated_linear_step_kernel(GatedLinear p, GatedLinearOut o, int cluster) {
  extern __shared__ __align__(16) float gl_s[];
  __shared__ float scratch[32];
  __shared__ float sums[GL_MAX_CLUSTER];
  constexpr int KD = RL * NCH * 4, WARPS = GL_THREADS / 32;
  const int Dk = p.Dk, Dv = p.Dv, slice = (Dv + cluster - 1) / cluster;
  float* w_s = gl_s;                          // [KD] decay
  float* k_s = w_s + KD;                      // [KD]
  float* q_s = k_s + KD;                      // [KD]
  float* low_s = q_s + KD;                    // [rank, padded to 8]
  float* v_s = low_s + (o.rank + 7) / 8 * 8;  // [slice] values, then the read-out
  allow_dependents();
  const int h = blockIdx.x / cluster, part = blockIdx.x - h * cluster, seq = blockIdx.y;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int c_lo = part * slice, cols = max(0, min(Dv, c_lo + slice) - c_lo);
  const int slot = p.seq_slots[seq];
  const size_t row = (size_t)p.q_start[seq];
  float* S = o.state + (size_t)slot * o.state_stride + ((size_t)h * Dv + c_lo) * Dk;
  // The state's and the small matrix's lines are asked for while the projection before this kernel still runs.
  for (size_t at = (size_t)tid * 32; at < (size_t)Dk * cols; at += (size_t)GL_THREADS * 32)
    asm volatile("prefetch.global.L2 [%0];" ::"l"(S + at));
  const T* a_up = (const T*)o.a_up + (size_t)h * Dk * o.rank;
  for (size_t at = (size_t)tid * (128 / sizeof(T)); at < (size_t)Dk * o.rank; at += (size_t)GL_THREADS * (128 / sizeof(T)))
    asm volatile("prefetch.global.L2 [%0];" ::"l"(a_up + at));
  grid_dependency_wait();
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
          const float4 v = (col < cols && ch < Dk) ? *reinterpret_cast<const float4*>(src + ch) : make_float4(0.f, 0.f, 0.f, 0.f);
          s[u][4 * c] = v.x; s[u][4 * c + 1] = v.y; s[u][4 * c + 2] = v.z; s[u][4 * c + 3] = v.w;
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) s[u][4 * c + e] = (col < cols && ch + e < Dk) ? src[ch + e] : 0.f;
        }
      }
    }
  };
  load_state(warp * COLS);
  const T* q = (const T*)p.q + row * p.stride + (size_t)h * Dk;
  const T* k = (const T*)p.k + row * p.stride + (size_t)h * Dk;
  const T* v = (const T*)p.v + row * p.stride + (size_t)h * Dv + c_lo;
  const T* low = (const T*)o.low + row * o.low_stride;
  for (int j = tid; j < KD; j += GL_THREADS) {
    q_s[j] = j < Dk ? to_float(q[j]) * p.q_scale : 0.f;
    k_s[j] = j < Dk ? to_float(k[j]) : 0.f;
  }
  for (int j = tid; j < cols; j += GL_THREADS) v_s[j] = to_float(v[j]);
  for (int j = tid; j < (o.rank + 7) / 8 * 8; j += GL_THREADS) low_s[j] = j < o.rank ? to_float(low[j]) : 0.f;
  __syncthreads();
  const bool packs = o.rank % (16 / (int)sizeof(T)) == 0 && (reinterpret_cast<uintptr_t>(a_up) & 15) == 0;
  rank_product<T, WARPS>(a_up, low_s, o.rank, Dk, packs, w_s);
  __syncthreads();
  for (int j = tid; j < KD; j += GL_THREADS)
    w_s[j] = j < Dk ? gate_decay<T>(w_s[j] + p.a_bias[h * Dk + j], p.decay_scale) : 1.f;
  __syncthreads();
  float wr[NCH * 4], kr[NCH * 4], qr[NCH * 4];
#pragma unroll
  for (int c = 0; c < NCH; ++c)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int ch = (c * RL + sub) * 4 + e;
      wr[4 * c + e] = w_s[ch];
      kr[4 * c + e] = k_s[ch];
      qr[4 * c + e] = q_s[ch];
    }
  for (int base = warp * COLS; base < cols; base += WARPS * COLS * UN) {
    if (base != warp * COLS) load_state(base);
#pragma unroll
    for (int u = 0; u < UN; ++u) {
      const int col = base + u * WARPS * COLS + sub_col;
      // Read before the shuffles, replaced after them: every lane of the column has its value by then.
      const float value = col < cols ? v_s[col] : 0.f;
      float read = 0.f;
#pragma unroll
      for (int e = 0; e < NCH * 4; ++e) {
        s[u][e] = fmaf(wr[e], s[u][e], kr[e] * value);
        read = fmaf(s[u][e], qr[e], read);
      }
#pragma unroll
      for (int off = RL / 2; off > 0; off >>= 1) read += __shfl_xor_sync(0xffffffffu, read, off);
      if (col < cols) {
        float* dst = S + (size_t)col * Dk;
#pragma unroll
        for (int c = 0; c < NCH; ++c) {
          const int ch = (c * RL + sub) * 4;
          if (VEC) {
            if (ch < Dk)
              *reinterpret_cast<float4*>(dst + ch) = make_float4(s[u][4 * c], s[u][4 * c + 1], s[u][4 * c + 2], s[u][4 * c + 3]);
          } else {
#pragma unroll
            for (int e = 0; e < 4; ++e)
              if (ch + e < Dk) dst[ch + e] = s[u][4 * c + e];
          }
        }
        if (sub == 0) v_s[col] = read;
      }
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < cols; c += GL_THREADS) ss = fmaf(v_s[c], v_s[c], ss);
  ss = block_sum(ss, scratch);
  if (cluster > 1) {
    if (tid < cluster) store_peer(peer_address(&sums[part], tid), ss);
    cluster_meet();  // nobody writes into a peer after this
    ss = 0.f;
    for (int i = 0; i < cluster; ++i) ss += sums[i];
  }
  const float inv = 1.0f / sqrtf(ss / (float)Dv + o.norm_eps);
  const T* gate = (const T*)o.gate + row * o.gate_stride + (size_t)h * Dv + c_lo;
  T* dst = (T*)o.out + row * o.out_stride + (size_t)h * Dv + c_lo;
  for (int c = tid; c < cols; c += GL_THREADS)
    dst[c] = from_float<T>(v_s[c] * inv * o.norm_w[c_lo + c] * silu_for<T>(to_float(gate[c])));
}

// ---------------------------------------------------------------------------------------------
// Portions, in chunks of LC = 32 tokens.  With S_0 the state a chunk starts from and P_(s->t) the product of the decays of
// tokens s + 1 .. t (per state row),
//     o_t = (P_(0->t) q_t)^T S_0 + sum_(s <= t) B_ts v_s,      B_ts = q_t^T P_(s->t) k_s
//     S_LC = P_(0->LC) S_0 + sum_s (P_(s->LC) k_s) v_s^T
// (the chunkwise form of Yang et al., "Gated Linear Attention Transformers with Hardware-Efficient Training").
// gated_linear_chunk_kernel makes Qt = P q, Kh = P k, B and P of every (chunk, head), a block each.  Decays
// enter as running products, each at most 1, so nothing overflows however strong they are.
// gated_linear_pass_kernel walks a sequence's chunks in order, a block per (LP_COLS value columns, head, sequence):
// the state's columns never meet.  All of it float32, in a fixed order; a token's result depends, within
// rounding, on where its chunk began.
//
// A chunk's record: Qt and Kh, [LC][KD] floats each (KD: Dk padded with zeros to a multiple of 32), B [LC][LC + 4],
// P [KD].  Chunk c of sequence s lies at place q_start[s] / LC + s + c.
constexpr int LC = 32, LP_COLS = 16, LP_THREADS = 256, LC_BP = LC + 4;

__host__ __device__ inline size_t gl_record_floats(int KD) { return (size_t)2 * LC * KD + LC * LC_BP + KD; }

// Sums 32 values over the warp's lanes, value i ending in lane i.
__device__ __forceinline__ float lanes_transpose_sum(float (&v)[32], int lane) {
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

template <typename T, int NV>
__global__ void __launch_bounds__(LP_THREADS)
gated_linear_chunk_kernel(GatedLinear p, const float* __restrict__ z, long long z_stride, float* __restrict__ records) {
  constexpr int KD = 32 * NV, KP = KD + 4;
  extern __shared__ __align__(16) float gl_s[];
  float* k_s = gl_s;           // [LC][KP]
  float* q_s = k_s + LC * KP;  // [LC][KP]
  float* g_s = q_s + LC * KP;  // [LC][KP] decays
  allow_dependents();
  const int chunk = blockIdx.x, h = blockIdx.y, seq = blockIdx.z;
  grid_dependency_wait();
  const int n_all = p.q_len[seq], first = chunk * LC;
  if (first >= n_all) return;
  const int n = min(LC, n_all - first), start = p.q_start[seq], Dk = p.Dk;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const size_t row0 = (size_t)(start + first);
  const T* q = (const T*)p.q + row0 * p.stride + (size_t)h * Dk;
  const T* k = (const T*)p.k + row0 * p.stride + (size_t)h * Dk;
  const float* zr = z + row0 * z_stride + (size_t)h * Dk;
  // A token behind the portion's end writes nothing, reads nothing and decays nothing.  Units of eight tokens of one
  // channel; loads from valid places, used or not: behind conditions they would be waited for one by one.
  for (int unit = tid; unit < (LC / 8) * KD; unit += LP_THREADS) {
    const int i0 = unit / KD * 8, d = unit % KD, at = min(d, Dk - 1);
    T qv[8], kv[8];
    float zv[8];
#pragma unroll
    for (int u = 0; u < 8; ++u) {
      const size_t r = (size_t)min(i0 + u, n - 1);
      qv[u] = q[r * p.stride + at];
      kv[u] = k[r * p.stride + at];
      zv[u] = zr[r * z_stride + at];
    }
    const float bias = p.a_bias[h * Dk + at];
#pragma unroll
    for (int u = 0; u < 8; ++u) {
      const bool ok = i0 + u < n && d < Dk;
      q_s[(i0 + u) * KP + d] = ok ? to_float(qv[u]) * p.q_scale : 0.f;
      k_s[(i0 + u) * KP + d] = ok ? to_float(kv[u]) : 0.f;
      g_s[(i0 + u) * KP + d] = ok ? gate_decay<T>(zv[u] + bias, p.decay_scale) : 1.f;
    }
  }
  __syncthreads();
  float* rec = records + ((size_t)(start / LC + seq + chunk) * p.heads + h) * gl_record_floats(KD);
  float *q_out = rec, *k_out = rec + LC * KD, *b_out = k_out + LC * KD, *p_out = b_out + LC * LC_BP;
  // Column j of B: k_j carried forward by the decays, a warp per column.
  for (int jj = warp; jj < LC; jj += LP_THREADS / 32) {
    const int j = (jj & 8) ? LC - 1 - (jj ^ 8) % LC : jj;  // a warp's four columns: two early ones, two late ones
    float r[NV], v[32];
#pragma unroll
    for (int e = 0; e < NV; ++e) r[e] = k_s[j * KP + lane + 32 * e];
#pragma unroll
    for (int i = 0; i < LC; ++i) {
      float b = 0.f;
      if (i >= j) {
        if (i > j) {
#pragma unroll
          for (int e = 0; e < NV; ++e) r[e] *= g_s[i * KP + lane + 32 * e];
        }
#pragma unroll
        for (int e = 0; e < NV; ++e) b = fmaf(q_s[i * KP + lane + 32 * e], r[e], b);
      }
      v[i] = b;
    }
    b_out[lane * LC_BP + j] = lanes_transpose_sum(v, lane);
  }
  // Queries from the chunk's start, keys to its end, a thread per channel.
  for (int d = tid; d < KD; d += LP_THREADS) {
    float product = 1.f, suffix = 1.f;
#pragma unroll 8
    for (int i = 0; i < LC; ++i) {
      product *= g_s[i * KP + d];
      q_out[i * KD + d] = q_s[i * KP + d] * product;
    }
    p_out[d] = product;
#pragma unroll 8
    for (int i = LC - 1; i >= 0; --i) {
      k_out[i * KD + d] = k_s[i * KP + d] * suffix;
      suffix *= g_s[i * KP + d];
    }
  }
}

// W rows of the state at a time, as a thread holds them and as they lie in shared memory.
template <int W>
__device__ __forceinline__ void load_rows(const float* p, float (&v)[W]) {
  if constexpr (W == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x, v[1] = f.y, v[2] = f.z, v[3] = f.w;
  } else if constexpr (W == 2) {
    const float2 f = *reinterpret_cast<const float2*>(p);
    v[0] = f.x, v[1] = f.y;
  } else {
    v[0] = *p;
  }
}
template <int W>
__device__ __forceinline__ void store_rows(float* p, const float (&v)[W]) {
  if constexpr (W == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else if constexpr (W == 2) *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
  else *p = v[0];
}

// Warps 0-3 carry the state (a thread: NV rows of four columns, in registers; a copy in shared memory for the
// products that read it), warps 4-7 make o from the state as it was.  Records come in by
// bulk copies, STAGES of them under way; the values' tile comes through registers.
template <typename T, int NV, int STAGES>
__global__ void __launch_bounds__(LP_THREADS)
gated_linear_pass_kernel(GatedLinear p, const float* __restrict__ records, float* __restrict__ state,
                         long long state_stride, float* __restrict__ out, long long out_stride, int* status) {
  constexpr int KD = 32 * NV, SP = KD + 4, VP = LP_COLS + 4;
  constexpr int W = NV % 4 == 0 ? 4 : NV % 2 == 0 ? 2 : 1, NJ = NV / W;  // rows lane * W + 32 W j of a lane
  constexpr int REC = 2 * LC * KD + LC * LC_BP + KD;
  extern __shared__ __align__(16) float gl_s[];
  float* S_s = gl_s + STAGES * REC;       // [LP_COLS][SP]
  float* V_s = S_s + LP_COLS * SP;        // [2][LC][VP]
  __shared__ __align__(8) unsigned long long bars[2];
  const int tile = blockIdx.x, h = blockIdx.y, seq = blockIdx.z;
  const int n = p.q_len[seq];
  if (n <= 0) {
    allow_dependents();
    return;
  }
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int start = p.q_start[seq], slot = p.seq_slots[seq], chunks = (n + LC - 1) / LC;
  const int Dk = p.Dk, Dv = p.Dv;
  const uint32_t bar0 = smem_u32(&bars[0]), bar1 = smem_u32(&bars[1]);
  if (tid == 0) {
    mbar_init(bar0, 1);
    mbar_init(bar1, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  __syncthreads();
  grid_dependency_wait();
  const size_t record = gl_record_floats(KD);
  const float* base = records + ((size_t)(start / LC + seq) * p.heads + h) * record;
  auto issue = [&](int c) {
    const uint32_t bar = STAGES == 2 && (c & 1) ? bar1 : bar0;
    mbar_expect_tx(bar, (uint32_t)REC * 4u);
    bulk_copy_g2s(smem_u32(gl_s + (c % STAGES) * REC), base + (size_t)c * p.heads * record, (uint32_t)REC * 4u, bar);
  };
  if (tid == 0) {
    issue(0);
    if (STAGES == 2 && chunks > 1) issue(1);
  }
  const T* values = (const T*)p.v + (size_t)start * p.stride + (size_t)h * Dv + tile * LP_COLS;
  const int v_col = tid % LP_COLS, v_row = tid / LP_COLS;  // and v_row + 16
  const bool v_ok = tile * LP_COLS + v_col < Dv;
  T v0, v1;  // as stored: they are looked at only when the chunk before is done
  auto fetch_values = [&](int c) {
    const int i0 = c * LC + v_row, col = v_ok ? v_col : 0;
    v0 = values[(size_t)min(i0, n - 1) * p.stride + col];
    v1 = values[(size_t)min(i0 + LC / 2, n - 1) * p.stride + col];
  };
  auto put_values = [&](int c) {
    const int i0 = c * LC + v_row;
    float* dst = V_s + (c & 1) * LC * VP + v_row * VP + v_col;
    dst[0] = v_ok && i0 < n ? to_float(v0) : 0.f;
    dst[LC / 2 * VP] = v_ok && i0 + LC / 2 < n ? to_float(v1) : 0.f;
  };
  fetch_values(0);
  put_values(0);
  float* st = state + (size_t)slot * state_stride + (size_t)h * Dv * Dk;
  const int my_cols = (warp & 3) * 4;
  float S[NJ][4][W];
  if (warp < 4) {
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int k0 = lane * W + 32 * W * j;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int col = tile * LP_COLS + my_cols + c;
#pragma unroll
        for (int e = 0; e < W; ++e) S[j][c][e] = col < Dv && k0 + e < Dk ? st[(size_t)col * Dk + k0 + e] : 0.f;
        store_rows<W>(S_s + (my_cols + c) * SP + k0, S[j][c]);
      }
    }
  }
  __syncthreads();
  // o: eight rows by four columns a thread, the inner size dealt to eight lanes.
  const int kg = lane & 7, c0 = (lane >> 3) * 4;
  for (int chunk = 0; chunk < chunks; ++chunk) {
    const float* buf = gl_s + (chunk % STAGES) * REC;
    const float* v_s = V_s + (chunk & 1) * LC * VP;
    mbar_wait(STAGES == 2 && (chunk & 1) ? bar1 : bar0, (uint32_t)(chunk / STAGES) & 1u, status);
    if (chunk + 1 < chunks) fetch_values(chunk + 1);
    if (warp < 4) {
      const float* kh = buf + LC * KD;
      const float* pv = buf + 2 * LC * KD + LC * LC_BP;
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        float decay[W];
        load_rows<W>(pv + lane * W + 32 * W * j, decay);
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
          for (int e = 0; e < W; ++e) S[j][c][e] *= decay[e];
      }
#pragma unroll 4
      for (int i = 0; i < LC; ++i) {
        float v[4];
        load_rows<4>(v_s + i * VP + my_cols, v);
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
          float kv[W];
          load_rows<W>(kh + i * KD + lane * W + 32 * W * j, kv);
#pragma unroll
          for (int c = 0; c < 4; ++c)
#pragma unroll
            for (int e = 0; e < W; ++e) S[j][c][e] = fmaf(kv[e], v[c], S[j][c][e]);
        }
      }
    } else {
      float acc[32];
#pragma unroll
      for (int i = 0; i < 32; ++i) acc[i] = 0.f;
      const float* rows = buf + (size_t)(warp - 4) * 8 * KD + 4 * kg;
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
      {
        // The chunk's own share, B times the values: four of its 32 tokens a lane, in the same sums.
        const float* b = buf + 2 * LC * KD + (size_t)(warp - 4) * 8 * LC_BP + 4 * kg;
        float vv[4][4];
#pragma unroll
        for (int e = 0; e < 4; ++e) load_rows<4>(v_s + (4 * kg + e) * VP + c0, vv[e]);
#pragma unroll
        for (int r = 0; r < 8; ++r) {
          float bv[4];
          load_rows<4>(b + r * LC_BP, bv);
#pragma unroll
          for (int e = 0; e < 4; ++e)
#pragma unroll
            for (int c = 0; c < 4; ++c) acc[4 * r + c] = fmaf(bv[e], vv[e][c], acc[4 * r + c]);
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
      const int row = (warp - 4) * 8 + kg;
      const int token = chunk * LC + row;
      if (token < n) {
        float* dst = out + (size_t)(start + token) * out_stride + (size_t)h * Dv + tile * LP_COLS + c0;
#pragma unroll
        for (int c = 0; c < 4; ++c)
          if (tile * LP_COLS + c0 + c < Dv) dst[c] = acc[c];
      }
    }
    __syncthreads();  // everybody has read the state and the stage
    if (tid == 0 && chunk + STAGES < chunks) issue(chunk + STAGES);
    if (chunk + 1 < chunks) put_values(chunk + 1);
    if (warp < 4) {
#pragma unroll
      for (int j = 0; j < NJ; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) store_rows<W>(S_s + (my_cols + c) * SP + lane * W + 32 * W * j, S[j][c]);
    }
    __syncthreads();
  }
  allow_dependents();
  if (warp < 4) {
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int k0 = lane * W + 32 * W * j;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int col = tile * LP_COLS + my_cols + c;
#pragma unroll
        for (int e = 0; e < W; ++e)
          if (col < Dv && k0 + e < Dk) st[(size_t)col * Dk + k0 + e] = S[j][c][e];
      }
    }
  }
}

}  // namespace vx

using namespace vx;

template <typename T, int NV>
static int launch_gated_linear_chunks(const GatedLinear& p, const float* z, long long z_stride, float* records,
                                      float* state, long long state_stride, float* out, long long out_stride,
                                      int num_seqs, int longest, int* status, cudaStream_t stream) {
  constexpr int KD = 32 * NV, STAGES = NV <= 8 ? 2 : 1;
  const size_t smem = sizeof(float) * 3 * LC * (KD + 4);
  const size_t pass_smem = sizeof(float) * (STAGES * gl_record_floats(KD) + LP_COLS * (KD + 4) + 2 * LC * (LP_COLS + 4));
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(gated_linear_chunk_kernel<T, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(gated_linear_pass_kernel<T, NV, STAGES>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)pass_smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  launch_pdl(gated_linear_chunk_kernel<T, NV>, dim3((longest + LC - 1) / LC, p.heads, num_seqs), dim3(LP_THREADS), smem,
             stream, p, z, z_stride, records);
  launch_pdl(gated_linear_pass_kernel<T, NV, STAGES>, dim3((p.Dv + LP_COLS - 1) / LP_COLS, p.heads, num_seqs),
             dim3(LP_THREADS), pass_smem, stream, p, (const float*)records, state, state_stride, out, out_stride, status);
  return (int)cudaGetLastError();
}

// Floats of scratch `vx_gated_linear_chunks` wants; -1: a key size it does not take.
VX_API long long vx_gated_linear_scratch(int num_tokens, int num_seqs, int heads, int Dk) {
  if (Dk <= 0 || Dk > 512) return -1;
  const int NV = (Dk + 31) / 32, KD = 32 * (NV <= 4 ? NV : NV <= 6 ? 6 : NV <= 8 ? 8 : NV <= 12 ? 12 : 16);
  return ((long long)num_tokens / LC + num_seqs + 1) * heads * (long long)gl_record_floats(KD);
}

// q, k, v: columns of rows `stride` apart; z float32 [tokens, heads * Dk] (logits without their bias); state [slots][heads,
// Dv, Dk]; out float32 [tokens, heads * Dv]; `longest`: no portion has more tokens.
VX_API int vx_gated_linear_chunks(const void* q, const void* k, const void* v, int dtype, long long stride, const float* z,
                                  long long z_stride, const float* a_bias, float q_scale, float decay_scale, int heads,
                                  int Dk, int Dv, float* records, long long record_floats, float* state,
                                  long long state_stride, float* out, long long out_stride, const int* q_start,
                                  const int* q_len, const int* seq_slots, int num_seqs, int num_tokens, int longest,
                                  int* status, cudaStream_t stream) {
  if (num_seqs <= 0 || num_tokens <= 0 || longest <= 0) return 0;
  if (heads <= 0 || heads > 65535 || num_seqs > 65535 || Dk <= 0 || Dk > 512 || Dv <= 0) return (int)cudaErrorInvalidValue;
  if (record_floats < vx_gated_linear_scratch(num_tokens, num_seqs, heads, Dk) || (reinterpret_cast<uintptr_t>(records) & 15) != 0)
    return (int)cudaErrorInvalidValue;
  const GatedLinear p = {q, k, v, stride, a_bias, q_scale, decay_scale, heads, Dk, Dv, q_start, q_len, seq_slots};
#define VX_GL_CHUNKS(NV)                                                                                                 \
  VX_BY_DTYPE(dtype, return (launch_gated_linear_chunks<T, NV>(p, z, z_stride, records, state, state_stride, out, out_stride, \
                                                               num_seqs, longest, status, stream)))
  if (Dk <= 32) { VX_GL_CHUNKS(1) }
  if (Dk <= 64) { VX_GL_CHUNKS(2) }
  if (Dk <= 96) { VX_GL_CHUNKS(3) }
  if (Dk <= 128) { VX_GL_CHUNKS(4) }
  if (Dk <= 192) { VX_GL_CHUNKS(6) }
  if (Dk <= 256) { VX_GL_CHUNKS(8) }
  if (Dk <= 384) { VX_GL_CHUNKS(12) }
  VX_GL_CHUNKS(16)
#undef VX_GL_CHUNKS
}

template <typename T, int RL, int NCH, bool VEC>
static int launch_gated_linear_step(const GatedLinear& p, const GatedLinearOut& o, int num_seqs, cudaStream_t stream) {
  // CTAs of a cluster: enough to give every SM work, slices of at least a pass of the block's warps.
  int cluster = 1;
  while (cluster < GL_MAX_CLUSTER && p.heads * num_seqs * cluster * 2 <= 2 * 148 && p.Dv / (cluster * 2) >= 8 * (32 / RL))
    cluster *= 2;
  const size_t smem = sizeof(float) * (3 * (size_t)(RL * NCH * 4) + (o.rank + 7) / 8 * 8 + (p.Dv + cluster - 1) / cluster);
  if (smem > 46 * 1024) return -1;
  return (int)launch_pdl_cluster(gated_linear_step_kernel<T, RL, NCH, VEC>, dim3(p.heads * cluster, num_seqs),
                                 dim3(GL_THREADS), smem, cluster, stream, p, o, cluster);
}

template <typename T>
static int choose_gated_linear_step(const GatedLinear& p, const GatedLinearOut& o, int num_seqs, cudaStream_t stream) {
  const bool vec = p.Dk % 4 == 0 && o.state_stride % 4 == 0 && (reinterpret_cast<uintptr_t>(o.state) & 15) == 0;
  if (!vec) {
    if (p.Dk <= 128) return launch_gated_linear_step<T, 32, 1, false>(p, o, num_seqs, stream);
    return launch_gated_linear_step<T, 32, 4, false>(p, o, num_seqs, stream);
  }
  if (p.Dk <= 16) return launch_gated_linear_step<T, 4, 1, true>(p, o, num_seqs, stream);
  if (p.Dk <= 32) return launch_gated_linear_step<T, 8, 1, true>(p, o, num_seqs, stream);
  if (p.Dk <= 64) return launch_gated_linear_step<T, 16, 1, true>(p, o, num_seqs, stream);
  if (p.Dk <= 128) return launch_gated_linear_step<T, 32, 1, true>(p, o, num_seqs, stream);
  if (p.Dk <= 256) return launch_gated_linear_step<T, 32, 2, true>(p, o, num_seqs, stream);
  return launch_gated_linear_step<T, 32, 4, true>(p, o, num_seqs, stream);
}

// One token of every sequence; `low` rows hold the decay pair's inner values, a_up [heads * Dk, rank].  -1: sizes the
// kernel does not take.
VX_API int vx_gated_linear_step(const void* q, const void* k, const void* v, int dtype, long long stride, const void* low,
                                long long low_stride, const void* a_up, int rank, const float* a_bias, float q_scale,
                                float decay_scale, int heads, int Dk, int Dv, const void* gate, long long gate_stride,
                                const float* norm_w, float norm_eps, void* out, long long out_stride, float* state,
                                long long state_stride, const int* q_start, const int* seq_slots, int num_seqs,
                                cudaStream_t stream) {
  if (num_seqs <= 0) return 0;
  if (heads <= 0 || num_seqs > 65535 || Dk <= 0 || Dk > 512 || Dv <= 0 || rank <= 0) return (int)cudaErrorInvalidValue;
  const GatedLinear p = {q, k, v, stride, a_bias, q_scale, decay_scale, heads, Dk, Dv, q_start, nullptr, seq_slots};
  const GatedLinearOut o = {low, low_stride, a_up, rank, gate, gate_stride, norm_w, norm_eps, out, out_stride, state, state_stride};
  VX_BY_DTYPE(dtype, return (choose_gated_linear_step<T>(p, o, num_seqs, stream)));
}
