// Kernels of recurrences whose state per head is a matrix that decays by a factor per key channel, or per head, and
// takes in one outer product a token: the delta rule, and linear attention with gated decays.
//
//   delta_prep   a fused projection's q, k and v behind a causal convolution over time per channel and a SiLU, q and k
//                unit vectors per head (q also scaled), beta's sigmoid, and the low-rank rows of decays and output
//                gates in the engine's type
//   delta_scan   per head S <- diag(g) S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q over the batch's new tokens
//                (without beta: u = v, plain linear attention), with g = exp(-rate softplus(sign (z + bias))) from a
//                product's columns z, one a key channel or one a head; the state is read from and left in the request's
//                slot.  Single tokens and short portions walk token by token with the state in registers; longer ones go
//                eight tokens at a time (`delta_local`, `delta_blocks`), the same sums in another order.
//   low_rank     z = A r for the rows r that columns of a fused projection hold: the second half of a low-rank product,
//                in float32 from the projection on
//
// Everything that enters the recurrence, and the state, is float32.  A product may come as a stack of K-split partial
// sums, which are added on the fly.
#include "common.cuh"

namespace delta {

// log(1 + e^z) without overflow; for small e^z it keeps the digits of e^z
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// ------------------------------------------------------------------------------------------------ delta_prep
constexpr int TILE = 8;       // tokens a warp takes together in a prompt: a projected value is read once for all taps
constexpr int REST = 128;     // beta and low-rank columns a warp takes
constexpr int MAX_TAPS = 32;

struct PrepArgs {
  const float* fused;     // [partials][N][total]: q (G D) | k (G D) | v (H Dv) | .. | beta (H) at beta_at | .. | low at low_at
  long long stride;
  int partials, total;
  const float* taps;      // [channels][T], the last one the current token's
  float* state;           // [slots][T - 1][channels]: the last projected values, the newest last
  const int* q_start;
  const int* state_slot;  // -1: no state (zeros are read, nothing is kept)
  const int* seq_of_token;
  float* mixed;           // [N][channels]: q (unit, scaled) | k (unit) | v
  float* beta;            // [N][H]
  void* low;              // [N][low_width] in the activation type
  int n, heads, kv_heads, dim, vdim, channels, taps_count, beta_at, low_at, low_width, num_slots;
  float unit_eps, q_scale;
  int keep;               // 1: a batch of single tokens, whose states this kernel updates itself
};

// SiLU in the activation type's accuracy: a bfloat16 engine takes the hardware exponential and reciprocal
template <typename TO> __device__ __forceinline__ float silu_for(float z);
template <> __device__ __forceinline__ float silu_for<float>(float z) { return z / (1.0f + expf(-z)); }
template <> __device__ __forceinline__ float silu_for<__nv_bfloat16>(float z) { return __fdividef(z, 1.0f + __expf(-z)); }

template <int VEC>
__device__ __forceinline__ void load_projected(const PrepArgs& a, bool stacked, int token, int c, float (&v)[VEC]) {
  const float* at = a.fused + static_cast<size_t>(token) * a.total + c;
  if constexpr (VEC == 4) {
    if (stacked) sum_partials4(at, a.stride, a.partials, v);
    else load4<float>(at, v);
  } else {
    v[0] = stacked ? sum_partials(at, a.stride, a.partials) : at[0];
  }
}

// The projected value `back` tokens before a sequence's first new one: from its slot, or zero.
template <int VEC>
__device__ __forceinline__ void load_held(const PrepArgs& a, int slot, int taps, int back, int c, float (&v)[VEC]) {
#pragma unroll
  for (int e = 0; e < VEC; ++e) v[e] = 0.f;
  if (slot < 0 || slot >= a.num_slots) return;
  const float* at = a.state + (static_cast<size_t>(slot) * (taps - 1) + (taps - 1 - back)) * a.channels + c;
#pragma unroll
  for (int e = 0; e < VEC; ++e) v[e] = at[e];
}

// T: the number of taps (1 to 4; 0: any number, whose values are read again per tap).  VEC channels a thread, `Tile`
// tokens a warp: 1 where tokens are few (the product may then be a stack of partial sums), else TILE, whose values are
// read together and walked with the taps' window in registers.  A warp takes one head (of q, k or v).
template <typename TO, int T, int VEC, int Tile>
__global__ void __launch_bounds__(128) delta_prep_kernel(const PrepArgs a) {
  let_dependents_start();
  constexpr bool STACKED = Tile == 1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int unit = blockIdx.y * 4 + warp;
  const int first = blockIdx.x * Tile, here = min(Tile, a.n - first);
  const int units = 2 * a.kv_heads + a.heads;
  const int seq_of = lane < here ? a.seq_of_token[first + lane] : -1;   // the step's metadata: no kernel writes it
  wait_for_previous();
  if (unit >= units) {   // beta and the low-rank rows
    const int begin = (unit - units) * REST, end = min(a.heads + a.low_width, begin + REST);
    for (int t = 0; t < here; ++t) {
      const float* row = a.fused + static_cast<size_t>(first + t) * a.total;
#pragma unroll
      for (int i = 0; i < REST / 32; ++i) {
        const int c = begin + lane + 32 * i;
        if (c >= end) continue;
        const float* at = row + (c < a.heads ? a.beta_at + c : a.low_at + c - a.heads);
        const float z = STACKED ? sum_partials(at, a.stride, a.partials) : at[0];
        if (c < a.heads) a.beta[static_cast<size_t>(first + t) * a.heads + c] = 1.0f / (1.0f + expf(-z));
        else static_cast<TO*>(a.low)[static_cast<size_t>(first + t) * a.low_width + c - a.heads] = from_float<TO>(z);
      }
    }
    return;
  }
  const bool normed = unit < 2 * a.kv_heads;
  const int size = normed ? a.dim : a.vdim;
  const int channel0 = normed ? unit * a.dim : 2 * a.kv_heads * a.dim + (unit - 2 * a.kv_heads) * a.vdim;
  const int taps = T > 0 ? T : a.taps_count;
  const int groups = size / VEC;
  const int seq0 = __shfl_sync(0xffffffffu, seq_of, 0);
  const int index0 = first - a.q_start[seq0];   // where the tile's first token stands in its sequence's portion
  float squares[Tile], y[Tile][VEC];
#pragma unroll
  for (int t = 0; t < Tile; ++t) squares[t] = 0.f;
  const bool single = groups <= 32;   // a head's channels are one round of the warp: they stay in registers
  for (int g0 = 0; g0 < groups; g0 += 32) {
    const int g = g0 + lane;
    const bool active = g < groups;
    const int c = channel0 + (active ? g : 0) * VEC;
    float x[Tile][VEC];
#pragma unroll
    for (int t = 0; t < Tile; ++t) load_projected<VEC>(a, STACKED, first + min(t, here - 1), c, x[t]);
    float w[T > 0 ? T : 1][VEC], window[T > 1 ? T - 1 : 1][VEC];   // window[i]: i + 1 tokens back
    if constexpr (T > 0) {
#pragma unroll
      for (int e = 0; e < VEC; ++e)
#pragma unroll
        for (int j = 0; j < T; ++j) w[j][e] = a.taps[static_cast<size_t>(c + e) * T + j];
      const int slot = a.state_slot[seq0];
#pragma unroll
      for (int i = 0; i < T - 1; ++i) {
        if (i + 1 <= index0) load_projected<VEC>(a, STACKED, first - i - 1, c, window[i]);
        else load_held<VEC>(a, slot, taps, i + 1 - index0, c, window[i]);
      }
    }
    int seq = seq0;
#pragma unroll
    for (int t = 0; t < Tile; ++t) {
      if (t < here) {
        const int now = Tile > 1 ? __shfl_sync(0xffffffffu, seq_of, t) : seq0;
        float acc[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
        if constexpr (T > 0) {
          if (Tile > 1 && now != seq) {   // another sequence begins here: its window comes from its slot
            const int slot = a.state_slot[now];
#pragma unroll
            for (int i = 0; i < T - 1; ++i) load_held<VEC>(a, slot, taps, i + 1, c, window[i]);
          }
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
#pragma unroll
            for (int j = 0; j < T - 1; ++j) acc[e] = __fmaf_rn(w[j][e], window[T - 2 - j][e], acc[e]);
            acc[e] = __fmaf_rn(w[T - 1][e], x[t][e], acc[e]);
#pragma unroll
            for (int i = T - 2; i > 0; --i) window[i][e] = window[i - 1][e];
            if (T > 1) window[0][e] = x[t][e];
          }
        } else {
          const int index = first + t - a.q_start[now], slot = a.state_slot[now];
          for (int j = 0; j < taps; ++j) {
            const int lag = taps - 1 - j;
            float u[VEC];
            if (lag <= index) load_projected<VEC>(a, STACKED, first + t - lag, c, u);
            else load_held<VEC>(a, slot, taps, lag - index, c, u);
#pragma unroll
            for (int e = 0; e < VEC; ++e) acc[e] = __fmaf_rn(a.taps[static_cast<size_t>(c + e) * taps + j], u[e], acc[e]);
          }
        }
        seq = now;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          y[t][e] = silu_for<TO>(acc[e]);
          if (active) squares[t] = __fmaf_rn(y[t][e], y[t][e], squares[t]);
        }
        if (!(single && normed) && active) {
          float* dst = a.mixed + static_cast<size_t>(first + t) * a.channels + c;
          if constexpr (VEC == 4) store4<float>(dst, y[t]);
          else dst[0] = y[t][0];
        }
        if (Tile == 1 && a.keep && active && taps > 1) {   // a sequence's one token: its state moves up by one
          const int slot = a.state_slot[seq0];
          if (slot >= 0 && slot < a.num_slots) {
            float* state = a.state + static_cast<size_t>(slot) * (taps - 1) * a.channels + c;
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
              for (int i = 0; i + 1 < taps - 1; ++i)
                state[static_cast<size_t>(i) * a.channels + e] = state[static_cast<size_t>(i + 1) * a.channels + e];
              state[static_cast<size_t>(taps - 2) * a.channels + e] = x[t][e];
            }
          }
        }
      }
    }
  }
  if (!normed) return;
  float gain[Tile];
#pragma unroll
  for (int t = 0; t < Tile; ++t) {
    gain[t] = 1.0f / sqrtf(warp_sum(squares[t]) + a.unit_eps);
    if (unit < a.kv_heads) gain[t] *= a.q_scale;
  }
  for (int g = lane; g < groups; g += 32) {
#pragma unroll
    for (int t = 0; t < Tile; ++t) {
      if (t >= here) continue;
      float* dst = a.mixed + static_cast<size_t>(first + t) * a.channels + channel0 + g * VEC;
      float v[VEC];
      if (single) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] = y[t][e];
      } else if constexpr (VEC == 4) {   // what this very thread stored
        load4<float>(dst, v);
      } else {
        v[0] = dst[0];
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] *= gain[t];
      if constexpr (VEC == 4) store4<float>(dst, v);
      else dst[0] = v[0];
    }
  }
}

// ------------------------------------------------------------------------------------------------ delta_scan
constexpr int STAGED = 8;   // tokens staged at a time: their loads are in flight together

struct ScanArgs {
  const float* mixed;     // [mixed_partials][N][pitch]: q (G D) | k (G D) | v (H Dv) | ..
  long long mixed_stride;
  int mixed_partials, pitch;
  const float* beta;      // [N][H]; null: no delta rule, every token adds k v^T
  const float* gates;     // [partials][N][gate_width]: z of head h, channel d at column gate_at + h D + d, or gate_at + h
  long long stride;
  int partials, gate_width, gate_at;
  const float* rate;      // [H]
  const float* bias;      // [H D], or [H]; null: none
  float sign, q_scale;
  float* state;           // [slots][H][head_stride]: row d, column j of S at d * Dv + j
  const int* q_start;
  const int* state_slot;
  float* out;             // [N][H Dv]
  int heads, kv_heads, dim, vdim, head_stride, num_slots;
  int lanes, cols;        // lanes of a warp that share a thread's columns; columns of a CTA
  int skip_from;          // > 0: sequences that bring at least so many tokens are served elsewhere
  int early_state;        // 1: no kernel still running writes the states: they are read before the wait
};

__device__ __forceinline__ float decay_of(const ScanArgs& a, float rate, float z, float bias) {
  return expf(-rate * softplus(a.sign * (z + bias)));
}

// One CTA owns `cols` value columns of one head's state for one sequence and walks its tokens in order with the state in
// registers: a thread holds R rows of C neighbouring columns, `lanes` neighbouring lanes (a power of two covering the
// head's rows) share those columns and add up by shuffles; no barrier falls inside the walk.  Tokens are staged STAGED
// at a time: q, k and the decays of the head (a lane's rows side by side, its run padded by four floats so that the
// lanes' 16-byte loads fall into different banks), the CTA's columns of v, and beta.  DELTA: the delta rule, else every
// token adds k v^T; HEAD: one decay a head instead of one a key channel.
template <int R, int C, bool DELTA, bool HEAD>
__global__ void __launch_bounds__(128, 4) delta_walk_kernel(const ScanArgs a) {
  extern __shared__ __align__(16) float delta_shared[];
  let_dependents_start();
  if (!a.early_state) wait_for_previous();
  const int D = a.dim, lanes = a.lanes, cols = a.cols;
  constexpr int PITCH = R + 4;
  const int padded = lanes * PITCH;
  float* q = delta_shared;              // [STAGED][padded]
  float* k = q + STAGED * padded;
  float* f = k + STAGED * padded;       // decays
  float* v = f + STAGED * padded;       // [STAGED][cols]
  float* b = v + STAGED * cols;         // [STAGED]; one decay a head: those at f[0 .. STAGED)
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int g = lane % lanes;
  const int j = (warp * (32 / lanes) + lane / lanes) * C;
  const int head = blockIdx.y, seq = blockIdx.z, col0 = blockIdx.x * cols;
  const int cols_here = min(cols, a.vdim - col0);
  const int first = a.q_start[seq], length = a.q_start[seq + 1] - first;
  if (a.skip_from > 0 && length >= a.skip_from) {
    if (a.early_state) wait_for_previous();   // every CTA waits before it leaves
    return;
  }
  const int slot = a.state_slot[seq];
  const size_t out_width = static_cast<size_t>(a.heads) * a.vdim;
  if (slot < 0 || slot >= a.num_slots) {   // a padding row: zeros out, nothing kept
    if (a.early_state) wait_for_previous();
    if (g == 0)
      for (int t = 0; t < length; ++t)
#pragma unroll
        for (int c = 0; c < C; ++c)
          if (j + c < cols_here) a.out[static_cast<size_t>(first + t) * out_width + head * a.vdim + col0 + j + c] = 0.f;
    return;
  }
  float* state = a.state + (static_cast<size_t>(slot) * a.heads + head) * a.head_stride;
  const bool wide = C == 4 && (a.vdim & 3) == 0;   // four columns a 16-byte access
  float S[C][R];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int d = g * R + r;
    const float* at = state + static_cast<size_t>(d) * a.vdim + col0 + j;
    if constexpr (C == 4) {
      if (wide) {
        float four[4] = {0.f, 0.f, 0.f, 0.f};
        if (d < D && j < cols_here) load4<float>(at, four);
#pragma unroll
        for (int c = 0; c < C; ++c) S[c][r] = four[c];
        continue;
      }
    }
#pragma unroll
    for (int c = 0; c < C; ++c) S[c][r] = d < D && j + c < cols_here ? at[c] : 0.f;
  }
  if (a.early_state) wait_for_previous();
  // rows past the head's own are zero in q, k and the decays: the state's rows there stay zero
  const int extra = lanes * R - D;
  for (int i = threadIdx.x; i < STAGED * extra; i += blockDim.x) {
    const int t = i / extra, d = D + i % extra;
    const int at = t * padded + (d / R) * PITCH + d % R;
    q[at] = 0.f;
    k[at] = 0.f;
    if (!HEAD) f[at] = 0.f;
  }
  const int group = head / (a.heads / a.kv_heads);
  const int q_col = group * D, k_col = (a.kv_heads + group) * D, v_col = 2 * a.kv_heads * D + head * a.vdim + col0;
  const float rate = a.rate[head];
  for (int t0 = 0; t0 < length; t0 += STAGED) {
    const int here = min(STAGED, length - t0);
    __syncthreads();   // the tokens staged before are used up
    for (int i = threadIdx.x; i < here * D; i += blockDim.x) {
      const int t = i / D, d = i - t * D;
      const float* row = a.mixed + static_cast<size_t>(first + t0 + t) * a.pitch;
      const int at = t * padded + (d / R) * PITCH + d % R;
      q[at] = a.q_scale * sum_partials(row + q_col + d, a.mixed_stride, a.mixed_partials);
      k[at] = sum_partials(row + k_col + d, a.mixed_stride, a.mixed_partials);
      if (!HEAD) {
        const float z = sum_partials(a.gates + static_cast<size_t>(first + t0 + t) * a.gate_width + a.gate_at + head * D + d, a.stride, a.partials);
        f[at] = decay_of(a, rate, z, a.bias != nullptr ? a.bias[head * D + d] : 0.f);
      }
    }
    for (int i = threadIdx.x; i < here * cols; i += blockDim.x) {
      const int t = i / cols, c = i - t * cols;
      v[i] = c < cols_here ? sum_partials(a.mixed + static_cast<size_t>(first + t0 + t) * a.pitch + v_col + c, a.mixed_stride, a.mixed_partials) : 0.f;
    }
    if (DELTA && threadIdx.x < here) b[threadIdx.x] = a.beta[static_cast<size_t>(first + t0 + threadIdx.x) * a.heads + head];
    if (HEAD && threadIdx.x >= 16 && threadIdx.x - 16 < here) {   // (a CTA has at least a warp)
      const int t = threadIdx.x - 16;
      const float z = sum_partials(a.gates + static_cast<size_t>(first + t0 + t) * a.gate_width + a.gate_at + head, a.stride, a.partials);
      f[t] = decay_of(a, rate, z, a.bias != nullptr ? a.bias[head] : 0.f);
    }
    __syncthreads();
    for (int t = 0; t < here; ++t) {
      const float4* f4 = reinterpret_cast<const float4*>(f + t * padded + g * PITCH);
      const float4* k4 = reinterpret_cast<const float4*>(k + t * padded + g * PITCH);
      const float4* q4 = reinterpret_cast<const float4*>(q + t * padded + g * PITCH);
      float kk[R], sum[C];
#pragma unroll
      for (int r = 0; r < R; r += 4) {
        const float4 x = k4[r >> 2];
        kk[r] = x.x; kk[r + 1] = x.y; kk[r + 2] = x.z; kk[r + 3] = x.w;
      }
#pragma unroll
      for (int c = 0; c < C; ++c) sum[c] = 0.f;
#pragma unroll
      for (int r = 0; r < R; r += 4) {
        const float4 x = HEAD ? make_float4(f[t], f[t], f[t], f[t]) : f4[r >> 2];
        const float keep[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
          for (int c = 0; c < C; ++c) {
            S[c][r + e] *= keep[e];
            if (DELTA) sum[c] = __fmaf_rn(S[c][r + e], kk[r + e], sum[c]);
          }
      }
      if (DELTA) {
        for (int offset = lanes >> 1; offset > 0; offset >>= 1)
#pragma unroll
          for (int c = 0; c < C; ++c) sum[c] += __shfl_xor_sync(0xffffffffu, sum[c], offset);
      }
      const float share = DELTA ? b[t] : 1.f;
#pragma unroll
      for (int c = 0; c < C; ++c) sum[c] = share * (v[t * cols + j + c] - sum[c]);   // u
      float read[C];
#pragma unroll
      for (int c = 0; c < C; ++c) read[c] = 0.f;
#pragma unroll
      for (int r = 0; r < R; r += 4) {
        const float4 x = q4[r >> 2];
        const float qq[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
          for (int c = 0; c < C; ++c) {
            S[c][r + e] = __fmaf_rn(kk[r + e], sum[c], S[c][r + e]);
            read[c] = __fmaf_rn(S[c][r + e], qq[e], read[c]);
          }
      }
      for (int offset = lanes >> 1; offset > 0; offset >>= 1)
#pragma unroll
        for (int c = 0; c < C; ++c) read[c] += __shfl_xor_sync(0xffffffffu, read[c], offset);
      if (g == 0) {
        float* dst = a.out + static_cast<size_t>(first + t0 + t) * out_width + head * a.vdim + col0 + j;
#pragma unroll
        for (int c = 0; c < C; ++c)
          if (j + c < cols_here) dst[c] = read[c];
      }
    }
  }
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int d = g * R + r;
    if (d >= D) continue;
    float* at = state + static_cast<size_t>(d) * a.vdim + col0 + j;
    if constexpr (C == 4) {
      if (wide) {
        const float four[4] = {S[0][r], S[1][r], S[2][r], S[3][r]};
        if (j < cols_here) store4<float>(at, four);
        continue;
      }
    }
#pragma unroll
    for (int c = 0; c < C; ++c)
      if (j + c < cols_here) at[c] = S[c][r];
  }
}

// ------------------------------------------------------------------------------------------------ blocks of tokens
// Longer portions go BLOCK tokens at a time.  With tokens 1 .. B of a block, P_t = g_1 ... g_t and F_t = g_(t+1) ... g_B
// (per key channel, products of decays, never a quotient), S the state before the block and
//
//   A[t][s]  = sum_d k_t k_s g_(s+1) ... g_t  (s < t)        a_t = S^T (P_t k_t)
//   Aq[t][s] = the same with q_t              (s <= t)       c_t = S^T (P_t q_t)
//
// the rule's u_t = beta_t (v_t - a_t - sum_(s<t) A[t][s] u_s) is U = T (V - a) with T = (I + diag(beta) A)^-1 diag(beta),
// lower triangular, and with d_s = v_s - a_s
//
//   o_t = c_t + sum_(s<=t) M[t][s] d_s,  M = Aq T          S <- P_B S + sum_s K_s d_s^T,  K_s = sum_(t>=s) T[t][s] F_t k_t
//
// `delta_local` forms P_t k_t, P_t q_t, K_s, P_B and M of every block and value head by itself; `delta_blocks` walks a
// sequence's blocks with the state in registers: one reduction over the rows, one barrier and one update per BLOCK
// tokens instead of per token, three multiply-adds a state element and token.  Without the delta rule u_t = v_t: a_t is
// not needed, T is the identity, M = Aq and K_s = F_s k_s.
constexpr int BLOCK = 8;

struct BlockArgs {
  ScanArgs s;
  float* records;   // [blocks][head_count][record]: P_t k_t [B][Dp] (delta rule) | P_t q_t [B][Dp] | K_s [B][Dp] | P_B [Dp] | M [B][B]
  int record, padded_dim;   // padded_dim: rows rounded up to what the lanes hold, zeros behind the head's own
  int num_seqs, from;       // sequences that bring at least `from` tokens run here
  int blocks;               // of the whole batch
  int head0, head_count;    // the heads this launch serves
  // Where the walks are few, a sequence is cut into runs of `run_blocks` blocks that walk side by side (0: it is not): first
  // every run but the last by itself, for what it makes of a zero state (A) and of any state (the delta rule: a matrix F,
  // S -> F S + A; without it a decay per row), then the states are carried from run to run, then every run walks again
  // from the state it starts from and gives its outputs.
  int run_blocks, value_slices;
  float* run_states;        // [runs][head_count][D][run_ld]: A, later the state a run starts from (vdim rounded up to four) | F [Dp]
  float* run_decays;        // [runs][head_count][Dp], without the delta rule
  int run_ld, run_values;   // run_values: the column where F begins
};

__host__ __device__ constexpr int record_floats(int padded_dim, bool delta) { return ((delta ? 3 : 2) * BLOCK + 1) * padded_dim + BLOCK * BLOCK; }

// Blocks of sequence `seq`; a warp sums them over the sequences before one.
__device__ __forceinline__ int blocks_of(const BlockArgs& a, int seq) {
  const int length = a.s.q_start[seq + 1] - a.s.q_start[seq];
  return length >= a.from ? (length + BLOCK - 1) / BLOCK : 0;
}

__device__ __forceinline__ int runs_of(const BlockArgs& a, int seq) { return (blocks_of(a, seq) + a.run_blocks - 1) / a.run_blocks; }

struct RunPlace { int seq, run, base; };   // base: the first block of the sequence among the batch's

// The sequence and the run within it of run `index` of the batch; lanes count 32 sequences at a time.
__device__ __forceinline__ RunPlace place_of_run(const BlockArgs& a, int index, int lane) {
  int runs_before = 0, blocks_before = 0;
  for (int base = 0; base < a.num_seqs; base += 32) {
    const int blocks = base + lane < a.num_seqs ? blocks_of(a, base + lane) : 0;
    const int runs = (blocks + a.run_blocks - 1) / a.run_blocks;
    int runs_sum = runs, blocks_sum = blocks;
#pragma unroll
    for (int offset = 1; offset < 32; offset <<= 1) {
      const int other_runs = __shfl_up_sync(0xffffffffu, runs_sum, offset), other_blocks = __shfl_up_sync(0xffffffffu, blocks_sum, offset);
      if (lane >= offset) { runs_sum += other_runs; blocks_sum += other_blocks; }
    }
    const unsigned hit = __ballot_sync(0xffffffffu, runs > 0 && index < runs_before + runs_sum);
    if (hit) {
      const int owner = __ffs(hit) - 1;
      return {base + owner, index - runs_before - __shfl_sync(0xffffffffu, runs_sum - runs, owner),
              blocks_before + __shfl_sync(0xffffffffu, blocks_sum - blocks, owner)};
    }
    runs_before += __shfl_sync(0xffffffffu, runs_sum, 31);
    blocks_before += __shfl_sync(0xffffffffu, blocks_sum, 31);
  }
  return {-1, 0, 0};
}

// The sums of COUNT values over 2 * OFFSET lanes, transposed: every step halves the values a lane holds, so that lane g of
// L ends with the sums of values g * n .. g * n + n - 1, n = COUNT / L; where the lanes outnumber the values, lanes that
// differ in the lowest bits end with the same one.
template <int COUNT, int OFFSET>
struct FoldLanes {
  static __device__ __forceinline__ void run(float* v, int lane) {
    if constexpr (OFFSET > 0) {
      if constexpr (COUNT > 1) {
        constexpr int HALF = COUNT / 2;
        const bool upper = lane & OFFSET;
#pragma unroll
        for (int i = 0; i < HALF; ++i) {
          const float send = upper ? v[i] : v[i + HALF], keep = upper ? v[i + HALF] : v[i];
          v[i] = keep + __shfl_xor_sync(0xffffffffu, send, OFFSET);
        }
        FoldLanes<HALF, OFFSET / 2>::run(v, lane);
      } else {
        v[0] += __shfl_xor_sync(0xffffffffu, v[0], OFFSET);
        FoldLanes<1, OFFSET / 2>::run(v, lane);
      }
    }
  }
};

// grid (blocks, heads / 4): a warp a block and value head.
template <bool DELTA, bool HEAD>
__global__ void __launch_bounds__(128) delta_local_kernel(const BlockArgs a) {
  __shared__ float shared_w[4][BLOCK * BLOCK], shared_t[4][BLOCK * BLOCK];
  wait_for_previous();   // the walk may start only when this kernel is nearly done: see the end
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int block = blockIdx.x, local_head = blockIdx.y * 4 + warp;
  if (local_head >= a.head_count) return;
  const int head = a.head0 + local_head;
  // the block's sequence: lanes count 32 sequences at a time
  int before = 0, seq = -1, within = 0;
  for (int base = 0; base < a.num_seqs && seq < 0; base += 32) {
    const int mine = base + lane < a.num_seqs ? blocks_of(a, base + lane) : 0;
    int total = mine;
#pragma unroll
    for (int offset = 1; offset < 32; offset <<= 1) {
      const int other = __shfl_up_sync(0xffffffffu, total, offset);
      if (lane >= offset) total += other;
    }
    const unsigned hit = __ballot_sync(0xffffffffu, block < before + total && mine > 0);
    if (hit) {
      const int owner = __ffs(hit) - 1;
      seq = base + owner;
      within = block - before - __shfl_sync(0xffffffffu, total - mine, owner);
    }
    before += __shfl_sync(0xffffffffu, total, 31);
  }
  if (seq < 0) return;
  const ScanArgs& s = a.s;
  const int first = s.q_start[seq] + within * BLOCK, here = min(BLOCK, s.q_start[seq + 1] - first);
  const int D = s.dim, Dp = a.padded_dim;
  const int group = head / (s.heads / s.kv_heads);
  const int q_col = group * D, k_col = (s.kv_heads + group) * D;
  const float rate = s.rate[head];
  float* record = a.records + (static_cast<size_t>(block) * a.head_count + local_head) * a.record;
  float* pk = record;
  float* pq = record + (DELTA ? BLOCK * Dp : 0);
  float* kk = pq + BLOCK * Dp;
  float* whole = kk + BLOCK * Dp;
  float pair[BLOCK * BLOCK];   // [t][s], s < t: A (delta rule);  [s][t], s <= t: Aq
#pragma unroll
  for (int i = 0; i < BLOCK * BLOCK; ++i) pair[i] = 0.f;
  float head_decay = 1.f;   // lane t holds token t's
  if (HEAD && lane < here) {
    const float z = sum_partials(s.gates + static_cast<size_t>(first + lane) * s.gate_width + s.gate_at + head, s.stride, s.partials);
    head_decay = decay_of(s, rate, z, s.bias != nullptr ? s.bias[head] : 0.f);
  }
  const float q_scale = s.q_scale;
  for (int d = lane; (HEAD ? d - lane : d) < Dp; d += 32) {   // (one decay a head: every lane takes part in the shuffles)
    float g[BLOCK], k[BLOCK], q[BLOCK];
    const bool row = d < D, kept = !HEAD || d < Dp;
    const float shift = !HEAD && row && s.bias != nullptr ? s.bias[head * D + d] : 0.f;
#pragma unroll
    for (int t = 0; t < BLOCK; ++t) {
      const bool real = row && t < here;
      const float* at = s.mixed + static_cast<size_t>(first + (t < here ? t : 0)) * s.pitch;
      k[t] = real ? at[k_col + d] : 0.f;
      q[t] = real ? q_scale * at[q_col + d] : 0.f;
      if (!HEAD) g[t] = real ? s.gates[static_cast<size_t>(first + t) * s.gate_width + s.gate_at + head * D + d] : 0.f;
    }
    if (!HEAD && s.partials > 1) {
#pragma unroll
      for (int t = 0; t < BLOCK; ++t)
        if (row && t < here) g[t] = sum_partials(s.gates + static_cast<size_t>(first + t) * s.gate_width + s.gate_at + head * D + d, s.stride, s.partials);
    }
#pragma unroll
    for (int t = 0; t < BLOCK; ++t) g[t] = HEAD ? __shfl_sync(0xffffffffu, head_decay, t) : (row && t < here ? decay_of(s, rate, g[t], shift) : (row ? 1.f : 0.f));
#pragma unroll
    for (int from = 0; from < BLOCK; ++from) {
      float w = k[from];
      pair[from * BLOCK + from] = __fmaf_rn(w, q[from], pair[from * BLOCK + from]);
#pragma unroll
      for (int t = from + 1; t < BLOCK; ++t) {
        w *= g[t];
        if (DELTA) pair[t * BLOCK + from] = __fmaf_rn(w, k[t], pair[t * BLOCK + from]);
        pair[from * BLOCK + t] = __fmaf_rn(w, q[t], pair[from * BLOCK + t]);
      }
      if (kept) kk[from * Dp + d] = w;   // F k: the key as it stands at the block's end
    }
    float p = 1.f;
#pragma unroll
    for (int t = 0; t < BLOCK; ++t) {
      p *= g[t];
      if (DELTA && kept) pk[t * Dp + d] = p * k[t];
      if (kept) pq[t * Dp + d] = p * q[t];
    }
    if (kept) whole[d] = p;
  }
  FoldLanes<BLOCK * BLOCK, 16>::run(pair, lane);
  float* w = shared_w[warp];
  float* solved = shared_t[warp];
  w[2 * lane] = pair[0];
  w[2 * lane + 1] = pair[1];
  __syncwarp();
  float* m = whole + Dp;
  if (!DELTA) {   // M is Aq as it stands, K_s the decayed keys
#pragma unroll
    for (int i = lane; i < BLOCK * BLOCK; i += 32) {
      const int t = i / BLOCK, c = i % BLOCK;
      m[i] = c <= t ? w[c * BLOCK + t] : 0.f;
    }
    let_dependents_start();
    return;
  }
  if (lane < BLOCK) {   // column `lane` of T by forward substitution
    float column[BLOCK];
#pragma unroll
    for (int t = 0; t < BLOCK; ++t) {
      float v = t == lane ? 1.f : 0.f;
#pragma unroll
      for (int r = 0; r < t; ++r) v = __fmaf_rn(-w[t * BLOCK + r], column[r], v);   // column[r] is 0 above the diagonal
      const float beta = t < here ? s.beta[static_cast<size_t>(first + t) * s.heads + head] : 0.f;
      column[t] = beta * v;
      solved[t * BLOCK + lane] = column[t];
    }
  }
  __syncwarp();
#pragma unroll
  for (int i = lane; i < BLOCK * BLOCK; i += 32) {
    const int t = i / BLOCK, c = i % BLOCK;
    float v = 0.f;
    for (int r = c; r <= t; ++r) v = __fmaf_rn(w[r * BLOCK + t], solved[r * BLOCK + c], v);
    m[i] = v;
  }
  for (int d = lane; d < Dp; d += 32) {   // what this very thread stored, through T
    float end[BLOCK];
#pragma unroll
    for (int t = 0; t < BLOCK; ++t) end[t] = kk[t * Dp + d];
#pragma unroll
    for (int c = 0; c < BLOCK; ++c) {
      float v = 0.f;
#pragma unroll
      for (int t = c; t < BLOCK; ++t) v = __fmaf_rn(solved[t * BLOCK + c], end[t], v);
      kk[c * Dp + d] = v;
    }
  }
  // (a CTA that leaves counts as having let its dependents start.)  A walk launched while these CTAs still fill the
  // device would be packed onto the few SMs that free up first, several of its long-running CTAs to an SM.
  let_dependents_start();
}

// Two float32 multiply-adds in one instruction.
__device__ __forceinline__ unsigned long long fma2(unsigned long long a, unsigned long long b, unsigned long long c) {
  unsigned long long d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ unsigned long long mul2(unsigned long long a, unsigned long long b) {
  unsigned long long d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ unsigned long long pack2(float lo, float hi) {
  unsigned long long d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ float2 unpack2(unsigned long long v) {
  float2 f;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(v));
  return f;
}
__device__ __forceinline__ void copy16(void* shared, const void* global) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<unsigned>(__cvta_generic_to_shared(shared))), "l"(global) : "memory");
}
__device__ __forceinline__ void copy4(void* shared, const void* global) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(static_cast<unsigned>(__cvta_generic_to_shared(shared))), "l"(global) : "memory");
}

constexpr int STAGES = 3;

// grid (slices, heads, sequences): a CTA owns `cols` value columns of one head's state for one sequence.  A thread holds
// rows 4 g .. 4 g + 3 (with CHUNKS 2 also the same LANES * 4 further on) of four neighbouring columns; LANES lanes, a
// team, cover the head's rows.  Register c of a lane is column c ^ turn of the team's four, `turn` the lane's top two bits:
// adding up over those lanes then needs no selection, every step keeps the first half of the columns and sends the other.
// Whole: blockIdx.z is a sequence.  In runs it is a run of the batch: Gather walks a run for its A and, in the CTAs behind the
// value columns', its F (from the identity with values of zero) and reads nothing out; FromStart walks it from its own state.
enum class Walk { Whole, Gather, FromStart };
template <int LANES, int CHUNKS, bool DELTA, Walk WALK>
__global__ void __launch_bounds__(CHUNKS == 2 ? 128 : 256) delta_blocks_kernel(const BlockArgs a) {
  extern __shared__ __align__(16) float blocks_shared[];
  constexpr bool OUT = WALK != Walk::Gather, RUNS = WALK != Walk::Whole;
  constexpr int C = 4, PAIRS = 2 * CHUNKS, N = BLOCK * C;
  constexpr int COLUMN_LANES = LANES >= C ? C : LANES;   // lanes the columns are shared out over, then the tokens
  constexpr int TOKEN_LANES = LANES / COLUMN_LANES;
  constexpr int OWN_COLUMNS = C / COLUMN_LANES, OWN_TOKENS = BLOCK / TOKEN_LANES;
  constexpr int Dp = 4 * LANES * CHUNKS, RECORD = record_floats(Dp, DELTA), PITCH = LANES * CHUNKS;
  constexpr int Q_ROW = DELTA ? BLOCK : 0, K_ROW = Q_ROW + BLOCK;   // where a record's P q and K begin, in rows
  const ScanArgs& s = a.s;
  let_dependents_start();
  wait_for_previous();
  const int local_head = blockIdx.y, head = a.head0 + local_head, cols = s.cols;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane % LANES, team = lane / LANES;
  int seq = blockIdx.z, base = 0;   // base: the first block of this walk
  bool last = true;
  int first, length;
  if constexpr (RUNS) {
    const RunPlace place = place_of_run(a, blockIdx.z, lane);
    if (place.seq < 0) return;
    seq = place.seq;
    const int begin = place.run * a.run_blocks;
    base = place.base + begin;
    first = s.q_start[seq] + begin * BLOCK;
    const int left = s.q_start[seq + 1] - first;
    last = left <= a.run_blocks * BLOCK;
    length = last ? left : a.run_blocks * BLOCK;
    if (!OUT && last) return;   // no run starts from what the last one makes
  } else {
    first = s.q_start[seq];
    length = s.q_start[seq + 1] - first;
    if (length < a.from) return;   // the token-by-token walk serves it
  }
  const bool whole_map = !OUT && static_cast<int>(blockIdx.x) >= a.value_slices;   // this CTA's columns are F's
  const int col0 = (whole_map ? blockIdx.x - a.value_slices : blockIdx.x) * cols;
  const int j = (warp * (32 / LANES) + team) * C;   // the first of the team's columns among the CTA's
  const int turn = COLUMN_LANES == 4 ? g / TOKEN_LANES : (COLUMN_LANES == 2 ? 2 * g : 0);
  const int cols_here = min(cols, (whole_map ? Dp : s.vdim) - col0);
  const int values_here = whole_map ? 0 : cols_here;   // columns whose values are read; the others' are zero
  const int slot = s.state_slot[seq];
  const size_t out_width = static_cast<size_t>(s.heads) * s.vdim;
  float* out = s.out + static_cast<size_t>(first) * out_width + head * s.vdim + col0;
  if (slot < 0 || slot >= s.num_slots) {
    if (OUT)
      for (int t = 0; t < length; ++t)
        for (int c = threadIdx.x; c < cols_here; c += blockDim.x) out[t * out_width + c] = 0.f;
    return;
  }
  if constexpr (!RUNS) {
    for (int other = lane; other < seq; other += 32) base += blocks_of(a, other);
#pragma unroll
    for (int offset = 16; offset > 0; offset >>= 1) base += __shfl_xor_sync(0xffffffffu, base, offset);
  }
  const int blocks = (length + BLOCK - 1) / BLOCK;
  const int stage_floats = RECORD + BLOCK * cols;
  float* team_values = blocks_shared + STAGES * stage_floats + (warp * (32 / LANES) + team) * 2 * N;   // d, then c, of this team's columns
  const int v_col = 2 * s.kv_heads * s.dim + head * s.vdim + col0;
  const bool wide_v = ((v_col | s.pitch | s.vdim) & 3) == 0 && (reinterpret_cast<uintptr_t>(s.mixed) & 15) == 0;
  // a thread's 16-byte piece of the CTA's columns of v, the same in every block (narrow heads have more pieces than threads)
  const int pieces = BLOCK * cols / 4, piece_t = static_cast<int>(threadIdx.x) / (cols / 4), piece_c = (static_cast<int>(threadIdx.x) - piece_t * (cols / 4)) * 4;
  const bool one_piece = wide_v && pieces <= static_cast<int>(blockDim.x);
  const float* next_record = a.records + (static_cast<size_t>(base) * a.head_count + local_head) * RECORD + threadIdx.x * 4;
  const size_t record_step = static_cast<size_t>(a.head_count) * RECORD;
  int fill = 0;   // the stage that is filled next
  const auto stage = [&](int block) {   // asks for a block's record and the CTA's columns of v
    if (block < blocks) {
      float* at = blocks_shared + fill * stage_floats;
#pragma unroll 4
      for (int i = threadIdx.x * 4, k = 0; i < RECORD; i += blockDim.x * 4, k += blockDim.x * 4) copy16(at + i, next_record + k);
      next_record += record_step;
      float* v = at + RECORD;
      const int here = min(BLOCK, length - block * BLOCK);
      const float* from = s.mixed + static_cast<size_t>(first + block * BLOCK) * s.pitch + v_col;
      if (one_piece) {
        if (static_cast<int>(threadIdx.x) < pieces) {
          if (piece_t < here && piece_c < values_here) copy16(v + piece_t * cols + piece_c, from + static_cast<size_t>(piece_t) * s.pitch + piece_c);
          else *reinterpret_cast<float4*>(v + piece_t * cols + piece_c) = make_float4(0.f, 0.f, 0.f, 0.f);
        }
      } else {
        for (int i = threadIdx.x; i < BLOCK * cols; i += blockDim.x) {
          const int t = i / cols, c = i - t * cols;
          if (t < here && c < values_here) copy4(v + i, from + static_cast<size_t>(t) * s.pitch + c);
          else v[i] = 0.f;
        }
      }
    }
    fill = fill + 1 == STAGES ? 0 : fill + 1;
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int i = 0; i < STAGES - 1; ++i) stage(i);
  float* state = s.state + (static_cast<size_t>(slot) * s.heads + head) * s.head_stride;
  const size_t run_at = (static_cast<size_t>(blockIdx.z) * a.head_count + local_head) * s.dim * a.run_ld + (whole_map ? a.run_values : 0) + col0;
  unsigned long long S[C][PAIRS];
#pragma unroll
  for (int p = 0; p < PAIRS; ++p)
#pragma unroll
    for (int c = 0; c < C; ++c) {
      const int d = (p / 2) * 4 * LANES + 4 * g + (p & 1) * 2, column = j + (c ^ turn);
      const bool mine = column < cols_here;
      if constexpr (OUT) {
        const float* at = RUNS ? a.run_states + run_at + static_cast<size_t>(d) * a.run_ld + column
                               : state + static_cast<size_t>(d) * s.vdim + col0 + column;
        S[c][p] = pack2(mine && d < s.dim ? at[0] : 0.f, mine && d + 1 < s.dim ? at[RUNS ? a.run_ld : s.vdim] : 0.f);
      } else {
        S[c][p] = pack2(whole_map && d < s.dim && d == col0 + column ? 1.f : 0.f, whole_map && d + 1 < s.dim && d + 1 == col0 + column ? 1.f : 0.f);
      }
    }
  constexpr int DECAYS = !OUT && !DELTA ? (Dp + 31) / 32 : 1;   // a thread's share of the rows' decays, at one warp a CTA
  float run_decay[DECAYS];
#pragma unroll
  for (int k = 0; k < DECAYS; ++k) run_decay[k] = 1.f;
  int taken = 0;   // the stage of the block at hand
  for (int block = 0; block < blocks; ++block) {
    asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");
    __syncthreads();   // the block's record is there, and everyone is done with the stage that is filled next
    stage(block + STAGES - 1);
    const float* at = blocks_shared + taken * stage_floats;
    taken = taken + 1 == STAGES ? 0 : taken + 1;
    const ulonglong2* rows = reinterpret_cast<const ulonglong2*>(at) + g;   // row r: + r * PITCH; chunk: + LANES
    const float* v = at + RECORD;
    float sum[2][N];   // a_t, then c_t, of this thread's rows: [column][token]
#pragma unroll
    for (int which = DELTA ? 0 : 1; which < (OUT ? 2 : 1); ++which) {
#pragma unroll
      for (int t = 0; t < BLOCK; ++t) {
        unsigned long long acc[C];
#pragma unroll
        for (int chunk = 0; chunk < CHUNKS; ++chunk) {
          const ulonglong2 x = rows[((which == 0 ? 0 : Q_ROW) + t) * PITCH + chunk * LANES];
#pragma unroll
          for (int c = 0; c < C; ++c) {
            acc[c] = chunk == 0 ? mul2(S[c][0], x.x) : fma2(S[c][2 * chunk], x.x, acc[c]);
            acc[c] = fma2(S[c][2 * chunk + 1], x.y, acc[c]);
          }
        }
#pragma unroll
        for (int c = 0; c < C; ++c) {
          const float2 f = unpack2(acc[c]);
          sum[which][c * BLOCK + t] = f.x + f.y;
        }
      }
    }
#pragma unroll
    for (int half = N / 2, offset = LANES / 2; half >= OWN_COLUMNS * BLOCK && offset > 0; half /= 2, offset /= 2)
#pragma unroll
      for (int i = 0; i < half; ++i)
#pragma unroll
        for (int which = DELTA ? 0 : 1; which < (OUT ? 2 : 1); ++which) sum[which][i] += __shfl_xor_sync(0xffffffffu, sum[which][i + half], offset);
    // this lane holds its columns' sums, shared with TOKEN_LANES - 1 others: d_t = v_t - a_t of its own tokens
#pragma unroll
    for (int i = 0; i < OWN_COLUMNS; ++i) {
      if constexpr (DELTA) FoldLanes<BLOCK, TOKEN_LANES / 2>::run(sum[0] + i * BLOCK, lane);
      if constexpr (OUT) FoldLanes<BLOCK, TOKEN_LANES / 2>::run(sum[1] + i * BLOCK, lane);
      const int c = turn + i;
#pragma unroll
      for (int k = 0; k < OWN_TOKENS; ++k) {
        const int t = g % TOKEN_LANES * OWN_TOKENS + k;
        team_values[c * BLOCK + t] = v[t * cols + j + c] - (DELTA ? sum[0][i * BLOCK + k] : 0.f);
        if (OUT) team_values[N + c * BLOCK + t] = sum[1][i * BLOCK + k];
      }
    }
    __syncwarp();
    const float* decay = at + (K_ROW + BLOCK) * Dp;
    if (!OUT && !DELTA && blockIdx.x == 0) {
#pragma unroll
      for (int k = 0; k < DECAYS; ++k)
        if (static_cast<int>(threadIdx.x + k * blockDim.x) < Dp) run_decay[k] *= decay[threadIdx.x + k * blockDim.x];
    }
#pragma unroll
    for (int chunk = 0; chunk < CHUNKS; ++chunk) {
      const ulonglong2 x = *(reinterpret_cast<const ulonglong2*>(decay) + g + chunk * LANES);
#pragma unroll
      for (int c = 0; c < C; ++c) {
        S[c][2 * chunk] = mul2(S[c][2 * chunk], x.x);
        S[c][2 * chunk + 1] = mul2(S[c][2 * chunk + 1], x.y);
      }
    }
    float d[C][BLOCK];
#pragma unroll
    for (int c = 0; c < C; ++c)
#pragma unroll
      for (int t = 0; t < BLOCK; t += 4) {
        const float4 four = *reinterpret_cast<const float4*>(team_values + (c ^ turn) * BLOCK + t);
        d[c][t] = four.x; d[c][t + 1] = four.y; d[c][t + 2] = four.z; d[c][t + 3] = four.w;
      }
#pragma unroll
    for (int t = 0; t < BLOCK; ++t) {
      unsigned long long dd[C];
#pragma unroll
      for (int c = 0; c < C; ++c) dd[c] = pack2(d[c][t], d[c][t]);
#pragma unroll
      for (int chunk = 0; chunk < CHUNKS; ++chunk) {
        const ulonglong2 x = rows[(K_ROW + t) * PITCH + chunk * LANES];
#pragma unroll
        for (int c = 0; c < C; ++c) {
          S[c][2 * chunk] = fma2(x.x, dd[c], S[c][2 * chunk]);
          S[c][2 * chunk + 1] = fma2(x.y, dd[c], S[c][2 * chunk + 1]);
        }
      }
    }
    const float* m = decay + Dp;
    const int here = min(BLOCK, length - block * BLOCK);
#pragma unroll
    for (int i = 0; i < (OUT ? (N + LANES - 1) / LANES : 0); ++i) {
      const int at_value = g + i * LANES, t = at_value / C, c = at_value % C;
      if (at_value < N && t < here && j + c < cols_here) {
        float o = team_values[N + c * BLOCK + t];
#pragma unroll
        for (int r = 0; r < BLOCK; r += 4) {
          const float4 row = *reinterpret_cast<const float4*>(m + t * BLOCK + r);
          const float4 four = *reinterpret_cast<const float4*>(team_values + c * BLOCK + r);
          o = __fmaf_rn(row.x, four.x, o);
          o = __fmaf_rn(row.y, four.y, o);
          o = __fmaf_rn(row.z, four.z, o);
          o = __fmaf_rn(row.w, four.w, o);
        }
        out[static_cast<size_t>(block * BLOCK + t) * out_width + j + c] = o;
      }
    }
    __syncwarp();   // the team's values are used up before the next block overwrites them
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  if (RUNS && OUT && !last) return;   // the run behind this one starts from what the carry made
#pragma unroll
  for (int p = 0; p < PAIRS; ++p)
#pragma unroll
    for (int c = 0; c < C; ++c) {
      const int d = (p / 2) * 4 * LANES + 4 * g + (p & 1) * 2, column = j + (c ^ turn);
      float* at = OUT ? state + static_cast<size_t>(d) * s.vdim + col0 + column
                      : a.run_states + run_at + static_cast<size_t>(d) * a.run_ld + column;
      const float2 two = unpack2(S[c][p]);
      if (column < cols_here) {
        if (d < s.dim) at[0] = two.x;
        if (d + 1 < s.dim) at[OUT ? s.vdim : a.run_ld] = two.y;
      }
    }
  if (!OUT && !DELTA && blockIdx.x == 0) {
#pragma unroll
    for (int k = 0; k < DECAYS; ++k)
      if (static_cast<int>(threadIdx.x + k * blockDim.x) < Dp)
        a.run_decays[(static_cast<size_t>(blockIdx.z) * a.head_count + local_head) * Dp + threadIdx.x + k * blockDim.x] = run_decay[k];
  }
}

// ------------------------------------------------------------------------------------------------ states from run to run
// grid (columns / CARRY_COLS, heads, sequences): S <- F S + A over a sequence's runs, each left the state it starts from
// where its A was.  A warp takes every eighth row of F, whose columns its lanes hold the state's rows for (EC groups of 128);
// the products meet by shuffles, the new state in shared memory.  STAGED: the next run's F and A are brought into shared
// memory (`padded_dim` columns and the CTA's own a row) while the present run's are multiplied; heads of more than 128 rows
// read them where they lie.
constexpr int CARRY_COLS = 8;
__host__ __device__ constexpr int carry_pitch(int padded_dim) { return padded_dim + CARRY_COLS; }
__host__ __device__ constexpr int carry_rows(int padded_dim) { return padded_dim + 4; }   // a state column's pitch: the columns fall into different banks

template <int EC, bool STAGED>
__global__ void __launch_bounds__(256) delta_carry_kernel(const BlockArgs a) {
  extern __shared__ __align__(16) float carry_shared[];   // two states of [CARRY_COLS][rows], then (STAGED) two runs' [D][F | A]
  const ScanArgs& s = a.s;
  let_dependents_start();
  wait_for_previous();
  const int local_head = blockIdx.y, head = a.head0 + local_head, seq = blockIdx.z, col0 = blockIdx.x * CARRY_COLS;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, D = s.dim, slot = s.state_slot[seq];
  const int runs = runs_of(a, seq), cols_here = min(CARRY_COLS, s.vdim - col0);
  if (runs == 0 || slot < 0 || slot >= s.num_slots) return;
  int first_run = 0;
  for (int other = lane; other < seq; other += 32) first_run += runs_of(a, other);
#pragma unroll
  for (int offset = 16; offset > 0; offset >>= 1) first_run += __shfl_xor_sync(0xffffffffu, first_run, offset);
  const float* state = s.state + (static_cast<size_t>(slot) * s.heads + head) * s.head_stride + col0;
  const int rows = carry_rows(a.padded_dim);
  float* now = carry_shared;
  float* next = carry_shared + rows * CARRY_COLS;
  for (int i = threadIdx.x; i < rows * CARRY_COLS; i += blockDim.x) {
    const int d = i / CARRY_COLS, c = i % CARRY_COLS;
    now[c * rows + d] = c < cols_here && d < D ? state[static_cast<size_t>(d) * s.vdim + c] : 0.f;
    next[c * rows + d] = 0.f;
  }
  const int own_col = lane / 4;   // where a row's eight sums end: four lanes hold the same one
  const bool keeper = lane % 4 == 0 && own_col < cols_here;
  const int pitch = carry_pitch(a.padded_dim), stage_floats = D * pitch;
  float* stages = carry_shared + 2 * rows * CARRY_COLS;
  const bool wide_a = cols_here == CARRY_COLS;   // (columns of A beyond the head's own values are not there)
  const auto stage = [&](int run) {   // asks for a run's F and this CTA's columns of A
    if (run + 1 < runs) {
      const float* held = a.run_states + (static_cast<size_t>(first_run + run) * a.head_count + local_head) * D * a.run_ld;
      float* at = stages + (run & 1) * stage_floats;
      const int pieces = a.padded_dim / 4;
      for (int i = threadIdx.x; i < D * pieces; i += blockDim.x) {
        const int d = i / pieces, p = (i - d * pieces) * 4;
        copy16(at + d * pitch + p, held + static_cast<size_t>(d) * a.run_ld + a.run_values + p);
      }
      for (int i = threadIdx.x; i < D * 2; i += blockDim.x) {
        const int d = i >> 1, p = (i & 1) * 4;
        float* to = at + d * pitch + a.padded_dim + p;
        const float* from = held + static_cast<size_t>(d) * a.run_ld + col0 + p;
        if (wide_a) {
          copy16(to, from);
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            if (p + e < cols_here) copy4(to + e, from + e);
            else to[e] = 0.f;
          }
        }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (STAGED) stage(0);
  for (int run = 0; run < runs; ++run) {
    float* held = a.run_states + (static_cast<size_t>(first_run + run) * a.head_count + local_head) * D * a.run_ld;
    if (STAGED) asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();   // `now` is complete, the run's F and A are there, and everyone is done with the stage filled next
    if (STAGED) stage(run + 1);
    if (run + 1 == runs) {
      for (int i = threadIdx.x; i < D * CARRY_COLS; i += blockDim.x) {
        const int d = i / CARRY_COLS, c = i % CARRY_COLS;
        if (c < cols_here) held[static_cast<size_t>(d) * a.run_ld + col0 + c] = now[c * rows + d];
      }
      return;
    }
    float S[EC][4][CARRY_COLS];
#pragma unroll
    for (int ec = 0; ec < EC; ++ec)
#pragma unroll
      for (int c = 0; c < CARRY_COLS; ++c) {
        float four[4] = {0.f, 0.f, 0.f, 0.f};
        if (ec * 128 + lane * 4 < a.padded_dim) load4<float>(now + c * rows + ec * 128 + lane * 4, four);
#pragma unroll
        for (int i = 0; i < 4; ++i) S[ec][i][c] = four[i];
      }
#pragma unroll 4
    for (int d = warp; d < D; d += 8) {
      const float* row = STAGED ? stages + (run & 1) * stage_floats + d * pitch : held + static_cast<size_t>(d) * a.run_ld + a.run_values;
      float* mine = held + static_cast<size_t>(d) * a.run_ld + col0 + own_col;
      const float added = keeper ? (STAGED ? row[a.padded_dim + own_col] : *mine) : 0.f;
      float sum[CARRY_COLS];
#pragma unroll
      for (int c = 0; c < CARRY_COLS; ++c) sum[c] = 0.f;
#pragma unroll
      for (int ec = 0; ec < EC; ++ec) {
        float f[4] = {0.f, 0.f, 0.f, 0.f};
        if (ec * 128 + lane * 4 < D) load4<float>(row + ec * 128 + lane * 4, f);
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int c = 0; c < CARRY_COLS; ++c) sum[c] = __fmaf_rn(f[i], S[ec][i][c], sum[c]);
      }
      FoldLanes<CARRY_COLS, 16>::run(sum, lane);
      if (keeper) {
        next[own_col * rows + d] = sum[0] + added;
        *mine = now[own_col * rows + d];
      }
    }
    float* swap = now;
    now = next;
    next = swap;
  }
}

// The same without the delta rule, where a run only multiplies every row of the state: a thread an element of it.
__global__ void __launch_bounds__(256) gated_carry_kernel(const BlockArgs a, int padded_dim) {
  const ScanArgs& s = a.s;
  let_dependents_start();
  wait_for_previous();
  const int local_head = blockIdx.y, head = a.head0 + local_head, seq = blockIdx.z, lane = threadIdx.x & 31, slot = s.state_slot[seq];
  const int runs = runs_of(a, seq);
  if (runs == 0 || slot < 0 || slot >= s.num_slots) return;
  int first_run = 0;
  for (int other = lane; other < seq; other += 32) first_run += runs_of(a, other);
#pragma unroll
  for (int offset = 16; offset > 0; offset >>= 1) first_run += __shfl_xor_sync(0xffffffffu, first_run, offset);
  const int index = blockIdx.x * blockDim.x + threadIdx.x;
  if (index >= s.dim * s.vdim) return;
  const int d = index / s.vdim, c = index - d * s.vdim;
  float S = s.state[(static_cast<size_t>(slot) * s.heads + head) * s.head_stride + index];
  const size_t step = static_cast<size_t>(a.head_count) * s.dim * a.run_ld, decay_step = static_cast<size_t>(a.head_count) * padded_dim;
  float* held = a.run_states + (static_cast<size_t>(first_run) * a.head_count + local_head) * s.dim * a.run_ld + static_cast<size_t>(d) * a.run_ld + c;
  const float* decay = a.run_decays + (static_cast<size_t>(first_run) * a.head_count + local_head) * padded_dim + d;
  constexpr int AHEAD = 4;
  for (int run = 0; run < runs; run += AHEAD) {
    float added[AHEAD], keep[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
      if (run + i + 1 < runs) {
        added[i] = held[(run + i) * step];
        keep[i] = decay[(run + i) * decay_step];
      }
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
      if (run + i < runs) {
        held[(run + i) * step] = S;
        if (run + i + 1 < runs) S = __fmaf_rn(keep[i], S, added[i]);
      }
  }
}

// ------------------------------------------------------------------------------------------------ low_rank
// z[n][c] = sum_r A[c][r] * x[n][r], x the `rank` columns of a fused projection from `at` on (a stack of partial sums is
// added up), A [C][padded] in the activation type with zeros behind its rank (16-byte rows).  A thread takes one column of
// TOK tokens, whose low-rank rows lie in shared memory.
constexpr int LOW_THREADS = 128;

template <typename T, int TOK>
__global__ void __launch_bounds__(LOW_THREADS) low_rank_kernel(const float* __restrict__ fused, int partials, long long stride, int total,
                                                               int at, const T* __restrict__ A, int padded, int rank,
                                                               float* __restrict__ z, int n, int columns) {
  extern __shared__ __align__(16) float low_shared[];   // [TOK][padded]
  let_dependents_start();
  wait_for_previous();
  const int first = blockIdx.y * TOK, here = min(TOK, n - first);
  for (int i = threadIdx.x; i < TOK * padded; i += LOW_THREADS) {
    const int t = i / padded, r = i - t * padded;
    low_shared[i] = t < here && r < rank ? sum_partials(fused + static_cast<size_t>(first + t) * total + at + r, stride, partials) : 0.f;
  }
  __syncthreads();
  const int c = blockIdx.x * LOW_THREADS + threadIdx.x;
  if (c >= columns) return;
  const T* row = A + static_cast<size_t>(c) * padded;
  float acc[TOK];
#pragma unroll
  for (int t = 0; t < TOK; ++t) acc[t] = 0.f;
  for (int r = 0; r < padded; r += 8) {
    float w[8];
    {
      float lo[4], hi[4];
      load4<T>(row + r, lo);
      load4<T>(row + r + 4, hi);
#pragma unroll
      for (int e = 0; e < 4; ++e) { w[e] = lo[e]; w[4 + e] = hi[e]; }
    }
#pragma unroll
    for (int t = 0; t < TOK; ++t) {
      const float4 x0 = *reinterpret_cast<const float4*>(low_shared + t * padded + r);
      const float4 x1 = *reinterpret_cast<const float4*>(low_shared + t * padded + r + 4);
      acc[t] = __fmaf_rn(w[0], x0.x, acc[t]); acc[t] = __fmaf_rn(w[1], x0.y, acc[t]);
      acc[t] = __fmaf_rn(w[2], x0.z, acc[t]); acc[t] = __fmaf_rn(w[3], x0.w, acc[t]);
      acc[t] = __fmaf_rn(w[4], x1.x, acc[t]); acc[t] = __fmaf_rn(w[5], x1.y, acc[t]);
      acc[t] = __fmaf_rn(w[6], x1.z, acc[t]); acc[t] = __fmaf_rn(w[7], x1.w, acc[t]);
    }
  }
#pragma unroll
  for (int t = 0; t < TOK; ++t)
    if (t < here) z[static_cast<size_t>(first + t) * columns + c] = acc[t];
}

template <typename T>
static void launch_low_rank(const float* fused, int partials, long long stride, int total, int at, const void* A, int padded, int rank,
                            float* z, int n, int columns, cudaStream_t stream) {
  const unsigned blocks = static_cast<unsigned>((columns + LOW_THREADS - 1) / LOW_THREADS);
  const T* a = static_cast<const T*>(A);
  if (n <= 64) {   // few tokens: one each, so that they fill the device
    launch_dependent(low_rank_kernel<T, 1>, dim3(blocks, n), LOW_THREADS, padded * sizeof(float), stream, fused, partials, stride,
                     total, at, a, padded, rank, z, n, columns);
  } else {
    launch_dependent(low_rank_kernel<T, 8>, dim3(blocks, (n + 7) / 8), LOW_THREADS, 8 * padded * sizeof(float), stream, fused, partials,
                     stride, total, at, a, padded, rank, z, n, columns);
  }
}

}  // namespace delta

// =========================================================================================== launchers
using namespace delta;

extern "C" int shrike_short_conv_keep(const float* fused, int partials, long long stride, int total, float* state,
                                      const int* q_start, const int* state_slot, int channels, int taps_count, int num_seqs,
                                      int num_slots, cudaStream_t stream);

// `longest`: the most new tokens a sequence of the batch brings (0: not known).  A batch of up to 64 single tokens has its
// convolution states moved up by the kernel itself, otherwise a second launch updates them.
SHRIKE_API int shrike_delta_prep(const float* fused, int partials, long long stride, int total, const float* taps, float* state,
                                 const int* q_start, const int* state_slot, const int* seq_of_token, float* mixed, float* beta,
                                 void* low, int dtype, int n, int heads, int kv_heads, int dim, int vdim, int taps_count,
                                 int beta_at, int low_at, int low_width, int num_seqs, int num_slots, float unit_eps, float q_scale,
                                 int longest, cudaStream_t stream) {
  if (n <= 0) return SHRIKE_OK;
  if (heads < 1 || kv_heads < 1 || heads % kv_heads || dim < 1 || vdim < 1 || taps_count < 1 || taps_count > MAX_TAPS || partials < 1)
    return SHRIKE_BAD_ARGUMENT;
  const int channels = 2 * kv_heads * dim + heads * vdim;
  if (beta_at < channels || beta_at + heads > total || low_at < 0 || low_at + low_width > total) return SHRIKE_BAD_ARGUMENT;
  PrepArgs a = {fused, stride, partials, total, taps, state, q_start, state_slot, seq_of_token, mixed, beta, low,
                n, heads, kv_heads, dim, vdim, channels, taps_count, beta_at, low_at, low_width, num_slots, unit_eps, q_scale,
                longest == 1 ? 1 : 0};
  const bool vec = dim % 4 == 0 && vdim % 4 == 0 && total % 4 == 0 && stride % 4 == 0 &&
                   (reinterpret_cast<uintptr_t>(fused) | reinterpret_cast<uintptr_t>(mixed)) % 16 == 0;
  const bool few = n <= 64 || partials > 1;   // a warp a token and head; otherwise TILE tokens a warp
  const int units = 2 * kv_heads + heads + (heads + low_width + REST - 1) / REST;
  const int tile = few ? 1 : TILE;
  const dim3 grid(static_cast<unsigned>((n + tile - 1) / tile), static_cast<unsigned>((units + 3) / 4));
  if (grid.y > 65535) return SHRIKE_BAD_ARGUMENT;
  if (longest == 1 && !few) a.keep = 0;
#define SHRIKE_PREP(TO, T, V)                                                                     \
  do {                                                                                            \
    if (few) launch_dependent(delta_prep_kernel<TO, T, V, 1>, grid, 128, 0, stream, a);           \
    else launch_dependent(delta_prep_kernel<TO, T, V, TILE>, grid, 128, 0, stream, a);            \
  } while (0)
#define SHRIKE_PREP_TAPS(TO, V)                      \
  do {                                               \
    if (taps_count == 1) SHRIKE_PREP(TO, 1, V);      \
    else if (taps_count == 2) SHRIKE_PREP(TO, 2, V); \
    else if (taps_count == 3) SHRIKE_PREP(TO, 3, V); \
    else if (taps_count == 4) SHRIKE_PREP(TO, 4, V); \
    else SHRIKE_PREP(TO, 0, V);                      \
  } while (0)
  if (dtype == SHRIKE_F32) { if (vec) SHRIKE_PREP_TAPS(float, 4); else SHRIKE_PREP_TAPS(float, 1); }
  else if (dtype == SHRIKE_BF16) { if (vec) SHRIKE_PREP_TAPS(__nv_bfloat16, 4); else SHRIKE_PREP_TAPS(__nv_bfloat16, 1); }
  else return SHRIKE_BAD_ARGUMENT;
#undef SHRIKE_PREP_TAPS
#undef SHRIKE_PREP
  const int status = shrike_launch_status();
  if (status != SHRIKE_OK || taps_count == 1 || a.keep) return status;
  // only after every token has read the old states
  return shrike_short_conv_keep(fused, partials, stride, total, state, q_start, state_slot, channels, taps_count, num_seqs,
                                num_slots, stream);
}

// How a walk is laid out for heads of dim x vdim: R rows of C columns a thread, the lanes that share those columns.
struct DeltaShape { int rows, each, lanes, cols, threads; size_t smem; };
static inline bool delta_shape(int dim, int vdim, DeltaShape* shape) {
  const int rows = dim <= 256 ? 8 : 32, each = dim <= 256 ? 4 : 1;
  int lanes = 1;
  while (lanes * rows < dim) lanes *= 2;
  if (lanes > 32) return false;
  const int per_warp = 32 / lanes * each;
  const int warps = max(1, min(4, (vdim + per_warp - 1) / per_warp));
  shape->rows = rows; shape->each = each; shape->lanes = lanes; shape->cols = per_warp * warps; shape->threads = warps * 32;
  shape->smem = (static_cast<size_t>(3) * STAGED * lanes * (rows + 4) + static_cast<size_t>(STAGED) * shape->cols + STAGED) * sizeof(float);
  return shape->smem <= static_cast<size_t>(shrike_device().max_smem);
}

// Scratch floats of one head of one block of BLOCK tokens; 0: heads of this size walk token by token.
SHRIKE_API int shrike_delta_scan_record(int dim, int delta) {
  DeltaShape shape;
  if (dim > 256 || !delta_shape(dim, 4, &shape)) return 0;
  return record_floats(shape.lanes * shape.rows, delta != 0);
}
SHRIKE_API int shrike_delta_scan_block() { return BLOCK; }

// How many blocks a run has where a batch of `seqs` sequences in blocks (`blocks` in all, `longest` the most of one), `heads` heads at a
// time, is to be cut into runs; 0: it is not.  A run is walked twice (the delta rule: dim / vdim times more), so runs pay where the
// walks alone would leave most of the SMs idle.
SHRIKE_API int shrike_delta_scan_run_blocks(int blocks, int longest, int seqs, int heads, int dim, int vdim, int delta) {
  DeltaShape shape;
  if (dim > 256 || seqs < 1 || longest < 48 || !delta_shape(dim, vdim, &shape)) return 0;
  const long long sms = shrike_device().sm_count, each = static_cast<long long>((vdim + 31) / 32) * heads;   // each: CTAs of one run
  const long long wanted = 2 * sms / each;   // runs that fill the device
  if (wanted < 3 * static_cast<long long>(seqs) || (delta && sms / each < 4 * static_cast<long long>(seqs))) return 0;
  const int run = static_cast<int>((blocks + wanted - 1) / wanted), least = delta ? 32 : 16;
  return run < least ? least : run;
}

// Scratch floats of one head of one run.
SHRIKE_API long long shrike_delta_scan_run_floats(int dim, int vdim, int delta) {
  DeltaShape shape;
  if (!delta_shape(dim, vdim, &shape)) return 0;
  const long long padded = shape.lanes * shape.rows, values = (vdim + 3) / 4 * 4;
  return static_cast<long long>(dim) * (values + (delta ? padded : 0)) + padded;
}

// `mixed` (`mixed_partials` slices `mixed_stride` apart, rows of `pitch`): q | k | v; only a walk takes more than one slice.
// `beta` null: no delta rule.  `gate_each`: 1, one decay a head, or dim, one a key channel (`bias`, where there is one, has
// heads * gate_each numbers); the decays' columns begin at `gate_at`.
// Sequences that bring at least `from` tokens (0: none) run in blocks, for which the caller holds `records`
// (blocks x head_count x shrike_delta_scan_record floats, `blocks` = the sum of ceil(length / BLOCK) over them); heads are
// then served `head_count` at a time.  `early_state` 1: the caller knows that whatever kernel wrote the states has finished
// (an earlier step, not merely an earlier launch), so that the walk may read them while the kernel before it runs.  `shorter`: whether the batch has sequences below `from`.
// `run_blocks` > 0: sequences are cut into runs of so many blocks, `runs` in all (the sum of ceil(blocks / run_blocks)), for which the
// caller holds `run_scratch` (runs x head_count x shrike_delta_scan_run_floats).
SHRIKE_API int shrike_delta_scan(const float* mixed, int mixed_partials, long long mixed_stride, int pitch, const float* beta,
                                 const float* gates, int partials, long long stride, int gate_width, int gate_at, int gate_each,
                                 const float* rate, const float* bias, float sign, float q_scale, float* state, const int* q_start,
                                 const int* state_slot, float* out, int num_seqs, int heads, int kv_heads, int dim, int vdim,
                                 int head_stride, int num_slots, int from, int shorter, float* records, int blocks,
                                 int head_count, int early_state, int run_blocks, int runs, float* run_scratch, cudaStream_t stream) {
  if (num_seqs <= 0) return SHRIKE_OK;
  if (heads < 1 || heads > 65535 || num_seqs > 65535 || kv_heads < 1 || heads % kv_heads || dim < 1 || vdim < 1 || partials < 1 ||
      mixed_partials < 1 || head_stride < dim * vdim || (gate_each != 1 && gate_each != dim) || gate_at < 0 ||
      gate_width < gate_at + heads * gate_each || pitch < 2 * kv_heads * dim + heads * vdim)
    return SHRIKE_BAD_ARGUMENT;
  const bool delta_rule = beta != nullptr, per_head = gate_each == 1 && dim > 1;
  if (per_head && !delta_rule) return SHRIKE_BAD_ARGUMENT;   // no design has asked for that pairing
  if (head_stride % 4 || reinterpret_cast<uintptr_t>(state) % 16) return SHRIKE_BAD_ARGUMENT;
  DeltaShape shape;
  if (!delta_shape(dim, vdim, &shape)) return SHRIKE_BAD_ARGUMENT;   // heads of more than 1,024 rows
  ScanArgs a = {mixed, mixed_stride, mixed_partials, pitch, beta, gates, stride, partials, gate_width, gate_at, rate, bias, sign, q_scale,
                state, q_start, state_slot, out, heads, kv_heads, dim, vdim, head_stride, num_slots, shape.lanes, shape.cols, 0, early_state};
  const bool in_blocks = from > 0 && records != nullptr && blocks > 0 && head_count > 0 && shape.rows == 8;
  if (in_blocks && mixed_partials > 1) return SHRIKE_BAD_ARGUMENT;
  const unsigned slices = static_cast<unsigned>((vdim + shape.cols - 1) / shape.cols);
  if (!in_blocks || shorter) {
    a.skip_from = in_blocks ? from : 0;
    void (*kernel)(ScanArgs);
    if (!delta_rule) kernel = shape.rows == 8 ? delta_walk_kernel<8, 4, false, false> : delta_walk_kernel<32, 1, false, false>;
    else if (per_head) kernel = shape.rows == 8 ? delta_walk_kernel<8, 4, true, true> : delta_walk_kernel<32, 1, true, true>;
    else kernel = shape.rows == 8 ? delta_walk_kernel<8, 4, true, false> : delta_walk_kernel<32, 1, true, false>;
    if (shape.smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(shape.smem));
    launch_dependent(kernel, dim3(slices, heads, num_seqs), static_cast<unsigned>(shape.threads), shape.smem, stream, a);
  }
  if (in_blocks) {
    BlockArgs b = {};
    b.s = a;
    b.records = records;
    b.padded_dim = shape.lanes * shape.rows;
    b.record = record_floats(b.padded_dim, delta_rule);
    b.num_seqs = num_seqs; b.from = from; b.blocks = blocks;
    // Four rows a thread where the walks are few (twice the warps hide each other's waits), eight where there are enough
    // of them (half the adding up over lanes); a head of more than 128 rows takes eight.
    const int sms = shrike_device().sm_count;
    const bool in_runs = run_blocks > 0 && runs > 0 && run_scratch != nullptr;
    if (in_runs && (runs > 65535 || vdim < 1)) return SHRIKE_BAD_ARGUMENT;
    const long long walks = in_runs ? runs : num_seqs;
    const long long quarters = static_cast<long long>((vdim + 31) / 32) * min(head_count, heads) * num_seqs;   // CTAs of 32 columns
    const int chunks = b.padded_dim > 128 || (quarters > 2 * sms && !in_runs) ? 2 : 1;
    const int lanes = b.padded_dim / (4 * chunks);
    const int per_warp = 32 / lanes * 4;
    int warps = max(1, min(chunks == 2 ? 4 : 8, (vdim + per_warp - 1) / per_warp));
    // few heads: narrower CTAs, as many as there are SMs for
    while (warps > 2 && warps % 2 == 0 && !in_runs &&
           static_cast<long long>((vdim + per_warp * warps - 1) / (per_warp * warps)) * min(head_count, heads) * num_seqs * 2 <= sms)
      warps /= 2;
    b.s.cols = per_warp * warps;
    const unsigned block_slices = static_cast<unsigned>((vdim + b.s.cols - 1) / b.s.cols);
    void (*kernel)(BlockArgs) = nullptr;
    void (*gather)(BlockArgs) = nullptr;   // the runs' first walk
#define SHRIKE_DELTA_BLOCKS_OF(L, WALK)                                                                  \
  (delta_rule ? (chunks == 2 ? delta_blocks_kernel<L, 2, true, WALK> : delta_blocks_kernel<L, 1, true, WALK>) \
              : (chunks == 2 ? delta_blocks_kernel<L, 2, false, WALK> : delta_blocks_kernel<L, 1, false, WALK>))
#define SHRIKE_DELTA_BLOCKS(L)                                                                                    \
  kernel = in_runs ? SHRIKE_DELTA_BLOCKS_OF(L, Walk::FromStart) : SHRIKE_DELTA_BLOCKS_OF(L, Walk::Whole), \
  gather = SHRIKE_DELTA_BLOCKS_OF(L, Walk::Gather)
    switch (lanes) {
      case 1: SHRIKE_DELTA_BLOCKS(1); break;
      case 2: SHRIKE_DELTA_BLOCKS(2); break;
      case 4: SHRIKE_DELTA_BLOCKS(4); break;
      case 8: SHRIKE_DELTA_BLOCKS(8); break;
      case 16: SHRIKE_DELTA_BLOCKS(16); break;
      default: SHRIKE_DELTA_BLOCKS(32); break;
    }
#undef SHRIKE_DELTA_BLOCKS
#undef SHRIKE_DELTA_BLOCKS_OF
    const int teams = warps * 32 / lanes;
    size_t smem = (static_cast<size_t>(STAGES) * (b.record + BLOCK * b.s.cols) + static_cast<size_t>(teams) * 2 * BLOCK * 4) * sizeof(float);
    const size_t most = static_cast<size_t>(shrike_device().max_smem);
    if (smem > most) return SHRIKE_BAD_ARGUMENT;
    // The walk's CTAs are few and run long: each asks for so much shared memory that they spread evenly over the SMs
    // instead of being packed where there is room first.
    const auto spread = [&](long long ctas) {
      const long long per_sm = (ctas + sms - 1) / sms;
      const size_t fair = most / static_cast<size_t>(per_sm) - 2048;
      return per_sm <= 8 && fair > smem ? fair : smem;
    };
    const size_t kernel_smem = spread(static_cast<long long>(block_slices) * min(head_count, heads) * walks);
    if (kernel_smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(kernel_smem));
    unsigned gather_slices = block_slices;
    size_t gather_smem = smem;
    if (in_runs) {
      b.run_blocks = run_blocks;
      b.value_slices = static_cast<int>(block_slices);
      b.run_values = (vdim + 3) / 4 * 4;
      b.run_ld = b.run_values + (delta_rule ? b.padded_dim : 0);
      b.run_states = run_scratch;
      b.run_decays = run_scratch + static_cast<size_t>(runs) * min(head_count, heads) * dim * b.run_ld;
      if (delta_rule) gather_slices += static_cast<unsigned>((b.padded_dim + b.s.cols - 1) / b.s.cols);
      gather_smem = spread(static_cast<long long>(gather_slices) * min(head_count, heads) * runs);
      if (gather_smem > 48 * 1024) cudaFuncSetAttribute(gather, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(gather_smem));
    }
    for (int head0 = 0; head0 < heads; head0 += head_count) {
      b.head0 = head0;
      b.head_count = min(head_count, heads - head0);
      void (*local)(BlockArgs) = !delta_rule ? delta_local_kernel<false, false>
                                             : (per_head ? delta_local_kernel<true, true> : delta_local_kernel<true, false>);
      launch_dependent(local, dim3(static_cast<unsigned>(blocks), static_cast<unsigned>((b.head_count + 3) / 4)), 128, 0, stream, b);
      if (in_runs) {
        launch_dependent(gather, dim3(gather_slices, b.head_count, runs), static_cast<unsigned>(warps * 32), gather_smem, stream, b);
        if (delta_rule) {
          const dim3 grid(static_cast<unsigned>((vdim + CARRY_COLS - 1) / CARRY_COLS), b.head_count, num_seqs);
          size_t held = static_cast<size_t>(2) * carry_rows(b.padded_dim) * CARRY_COLS * sizeof(float);
          if (dim <= 128) {
            held += static_cast<size_t>(2) * dim * carry_pitch(b.padded_dim) * sizeof(float);
            if (held > 48 * 1024) cudaFuncSetAttribute(delta_carry_kernel<1, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(held));
            launch_dependent(delta_carry_kernel<1, true>, grid, 256, held, stream, b);
          } else {
            launch_dependent(delta_carry_kernel<2, false>, grid, 256, held, stream, b);
          }
        } else {
          launch_dependent(gated_carry_kernel, dim3(static_cast<unsigned>((dim * vdim + 255) / 256), b.head_count, num_seqs), 256, 0, stream, b, b.padded_dim);
        }
      }
      launch_dependent(kernel, dim3(block_slices, b.head_count, static_cast<unsigned>(walks)), static_cast<unsigned>(warps * 32), kernel_smem, stream, b);
    }
  }
  return shrike_launch_status();
}

// z [N][columns] = the rows of A [columns][padded] (activation type, zeros from `rank` on, `padded` a multiple of 8, rows on
// 16-byte borders) times the `rank` columns of `fused` from `at` on.
SHRIKE_API int shrike_low_rank(const float* fused, int partials, long long stride, int total, int at, const void* A, int dtype,
                               int padded, int rank, float* z, int n, int columns, cudaStream_t stream) {
  if (n <= 0) return SHRIKE_OK;
  if (partials < 1 || columns < 1 || rank < 1 || padded < rank || padded % 8 || padded > 1024 || at < 0 || at + rank > total ||
      reinterpret_cast<uintptr_t>(A) % 16 || n > 8 * 65535)
    return SHRIKE_BAD_ARGUMENT;
  if (dtype == SHRIKE_F32) launch_low_rank<float>(fused, partials, stride, total, at, A, padded, rank, z, n, columns, stream);
  else if (dtype == SHRIKE_BF16) launch_low_rank<__nv_bfloat16>(fused, partials, stride, total, at, A, padded, rank, z, n, columns, stream);
  else return SHRIKE_BAD_ARGUMENT;
  return shrike_launch_status();
}
