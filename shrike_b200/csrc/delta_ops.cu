// Kernels of the delta rule whose state decays per key channel.
//
//   delta_prep   a fused projection's q, k and v behind a causal convolution over time per channel and a SiLU, q and k
//                unit vectors per head (q also scaled), beta's sigmoid, and the low-rank rows of decays and output
//                gates in the engine's type
//   delta_scan   per head S <- diag(g) S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q over the batch's new tokens,
//                with g = exp(-rate softplus(z + bias)) from a second product's columns z; the state is read from and
//                left in the request's slot.  The walk goes token by token with the state in registers.
//
// Everything that enters the recurrence, and the state, is float32.  A product may come as a stack of K-split partial
// sums, which are added on the fly.
#include "common.cuh"

namespace delta {

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }

// log(1 + e^z) without overflow; for small e^z it keeps the digits of e^z
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// ------------------------------------------------------------------------------------------------ delta_prep
constexpr int TILE = 8;       // tokens a warp takes together: a projected value is read once for all taps
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

// T: the number of taps (1 to 4; 0: any number, values read again per tap).  VEC channels a thread.
// A warp takes a head (of q, k or v) and TILE tokens; the tokens' values and the T - 1 before them are read first.
template <typename TO, int T, int VEC>
__global__ void __launch_bounds__(128) delta_prep_kernel(const PrepArgs a) {
  let_dependents_start();
  wait_for_previous();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int unit = blockIdx.y * 4 + warp;
  const int first = blockIdx.x * TILE, here = min(TILE, a.n - first);
  const int units = 2 * a.kv_heads + a.heads;
  if (unit > units) return;
  if (unit == units) {   // beta and the low-rank rows, column by column
    for (int t = 0; t < here; ++t) {
      const float* row = a.fused + static_cast<size_t>(first + t) * a.total;
      for (int c = lane; c < a.heads; c += 32)
        a.beta[static_cast<size_t>(first + t) * a.heads + c] = 1.0f / (1.0f + expf(-sum_partials(row + a.beta_at + c, a.stride, a.partials)));
      TO* low = static_cast<TO*>(a.low) + static_cast<size_t>(first + t) * a.low_width;
      for (int c = lane; c < a.low_width; c += 32) low[c] = from_float<TO>(sum_partials(row + a.low_at + c, a.stride, a.partials));
    }
    return;
  }
  const bool normed = unit < 2 * a.kv_heads;
  const int size = normed ? a.dim : a.vdim;
  const int channel0 = normed ? unit * a.dim : 2 * a.kv_heads * a.dim + (unit - 2 * a.kv_heads) * a.vdim;
  const int taps = T > 0 ? T : a.taps_count;
  constexpr int HALO = T > 1 ? T - 1 : 0;
  float squares[TILE];
#pragma unroll
  for (int t = 0; t < TILE; ++t) squares[t] = 0.f;
  // where each token stands in its sequence, and its sequence's slot
  int index[TILE], slot[TILE];
#pragma unroll
  for (int t = 0; t < TILE; ++t) {
    index[t] = 0;
    slot[t] = -1;
    if (t < here) {
      const int seq = a.seq_of_token[first + t];
      index[t] = first + t - a.q_start[seq];
      const int s = a.state_slot[seq];
      slot[t] = s >= 0 && s < a.num_slots ? s : -1;
    }
  }
  const int groups = size / VEC;
  for (int g = lane; g < groups; g += 32) {
    const int c = channel0 + g * VEC;
    const auto projected = [&](int token, float (&v)[VEC]) {
      const float* at = a.fused + static_cast<size_t>(token) * a.total + c;
      if constexpr (VEC == 4) sum_partials4(at, a.stride, a.partials, v);
      else v[0] = sum_partials(at, a.stride, a.partials);
    };
    float x[TILE + HALO][VEC];
    if constexpr (T > 0) {
#pragma unroll
      for (int i = 0; i < TILE + HALO; ++i) {
        const int token = first + i - HALO;
        if (token >= 0 && i - HALO < here) projected(token, x[i]);
        else {
#pragma unroll
          for (int e = 0; e < VEC; ++e) x[i][e] = 0.f;
        }
      }
    }
    float w[T > 0 ? T : 1][VEC];
    if constexpr (T > 0) {
#pragma unroll
      for (int j = 0; j < T; ++j)
#pragma unroll
        for (int e = 0; e < VEC; ++e) w[j][e] = a.taps[static_cast<size_t>(c + e) * T + j];
    }
#pragma unroll
    for (int t = 0; t < TILE; ++t) {
      if (t >= here) continue;
      float acc[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
      const auto held = [&](int back, int e) {   // the projected value `back` tokens before the sequence's first new one
        return slot[t] >= 0 ? a.state[(static_cast<size_t>(slot[t]) * (taps - 1) + (taps - 1 - back)) * a.channels + c + e] : 0.f;
      };
      if constexpr (T > 0) {
#pragma unroll
        for (int j = 0; j < T; ++j) {
          const int lag = T - 1 - j;
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            const float u = lag <= index[t] ? x[t + j][e] : held(lag - index[t], e);   // x[t + HALO - lag] is x[t + j]
            acc[e] = __fmaf_rn(w[j][e], u, acc[e]);
          }
        }
      } else {
        for (int j = 0; j < taps; ++j) {
          const int lag = taps - 1 - j;
          float u[VEC];
          if (lag <= index[t]) projected(first + t - lag, u);
          else {
#pragma unroll
            for (int e = 0; e < VEC; ++e) u[e] = held(lag - index[t], e);
          }
#pragma unroll
          for (int e = 0; e < VEC; ++e) acc[e] = __fmaf_rn(a.taps[static_cast<size_t>(c + e) * taps + j], u[e], acc[e]);
        }
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        acc[e] = silu(acc[e]);
        squares[t] = __fmaf_rn(acc[e], acc[e], squares[t]);
      }
      float* dst = a.mixed + static_cast<size_t>(first + t) * a.channels + c;
      if constexpr (VEC == 4) store4<float>(dst, acc);
      else dst[0] = acc[0];
      if (a.keep && slot[t] >= 0 && taps > 1) {   // a sequence's one token: its state moves up by one
        float* state = a.state + static_cast<size_t>(slot[t]) * (taps - 1) * a.channels + c;
        float newest[VEC];
        projected(first + t, newest);
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          for (int i = 0; i + 1 < taps - 1; ++i) state[static_cast<size_t>(i) * a.channels + e] = state[static_cast<size_t>(i + 1) * a.channels + e];
          state[static_cast<size_t>(taps - 2) * a.channels + e] = newest[e];
        }
      }
    }
  }
  if (!normed) return;
  float gain[TILE];
#pragma unroll
  for (int t = 0; t < TILE; ++t) {
    gain[t] = 1.0f / sqrtf(warp_sum(squares[t]) + a.unit_eps);
    if (unit < a.kv_heads) gain[t] *= a.q_scale;
  }
  for (int g = lane; g < groups; g += 32) {   // what this very thread stored
#pragma unroll
    for (int t = 0; t < TILE; ++t) {
      if (t >= here) continue;
      float* dst = a.mixed + static_cast<size_t>(first + t) * a.channels + channel0 + g * VEC;
      float v[VEC];
      if constexpr (VEC == 4) load4<float>(dst, v);
      else v[0] = dst[0];
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
  const float* mixed;     // [N][channels]: q (G D) | k (G D) | v (H Dv)
  const float* beta;      // [N][H]
  const float* gates;     // [partials][N][gate_width]: z of head h, channel d at column h D + d
  long long stride;
  int partials, gate_width;
  const float* rate;      // [H]
  const float* bias;      // [H D]
  float* state;           // [slots][H][head_stride]: row d, column j of S at d * Dv + j
  const int* q_start;
  const int* state_slot;
  float* out;             // [N][H Dv]
  int heads, kv_heads, dim, vdim, channels, head_stride, num_slots;
  int lanes, cols;        // lanes of a warp that share a thread's columns; columns of a CTA
};

// One CTA owns `cols` value columns of one head's state for one sequence and walks its tokens in order with the state in
// registers: a thread holds R rows of C neighbouring columns, `lanes` neighbouring lanes (a power of two covering the
// head's rows) share those columns and add up by shuffles; no barrier falls inside the walk.  Tokens are staged STAGED
// at a time: q, k and the decays of the head (a lane's rows side by side, its run padded by four floats so that the
// lanes' 16-byte loads fall into different banks), the CTA's columns of v, and beta.
template <int R, int C>
__global__ void __launch_bounds__(128, 4) delta_walk_kernel(const ScanArgs a) {
  extern __shared__ __align__(16) float delta_shared[];
  let_dependents_start();
  wait_for_previous();
  const int D = a.dim, lanes = a.lanes, cols = a.cols;
  constexpr int PITCH = R + 4;
  const int padded = lanes * PITCH;
  float* q = delta_shared;              // [STAGED][padded]
  float* k = q + STAGED * padded;
  float* f = k + STAGED * padded;       // decays
  float* v = f + STAGED * padded;       // [STAGED][cols]
  float* b = v + STAGED * cols;         // [STAGED]
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int g = lane % lanes;
  const int j = (warp * (32 / lanes) + lane / lanes) * C;
  const int head = blockIdx.y, seq = blockIdx.z, col0 = blockIdx.x * cols;
  const int cols_here = min(cols, a.vdim - col0);
  const int first = a.q_start[seq], length = a.q_start[seq + 1] - first;
  const int slot = a.state_slot[seq];
  const size_t out_width = static_cast<size_t>(a.heads) * a.vdim;
  if (slot < 0 || slot >= a.num_slots) {   // a padding row: zeros out, nothing kept
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
  // rows past the head's own are zero in q, k and the decays: the state's rows there stay zero
  const int extra = lanes * R - D;
  for (int i = threadIdx.x; i < STAGED * extra; i += blockDim.x) {
    const int t = i / extra, d = D + i % extra;
    const int at = t * padded + (d / R) * PITCH + d % R;
    q[at] = 0.f;
    k[at] = 0.f;
    f[at] = 0.f;
  }
  const int group = head / (a.heads / a.kv_heads);
  const int q_col = group * D, k_col = (a.kv_heads + group) * D, v_col = 2 * a.kv_heads * D + head * a.vdim + col0;
  const float rate = a.rate[head];
  for (int t0 = 0; t0 < length; t0 += STAGED) {
    const int here = min(STAGED, length - t0);
    __syncthreads();   // the tokens staged before are used up
    for (int i = threadIdx.x; i < here * D; i += blockDim.x) {
      const int t = i / D, d = i - t * D;
      const float* row = a.mixed + static_cast<size_t>(first + t0 + t) * a.channels;
      const float z = sum_partials(a.gates + static_cast<size_t>(first + t0 + t) * a.gate_width + head * D + d, a.stride, a.partials);
      const int at = t * padded + (d / R) * PITCH + d % R;
      q[at] = row[q_col + d];
      k[at] = row[k_col + d];
      f[at] = expf(-rate * softplus(z + a.bias[head * D + d]));
    }
    for (int i = threadIdx.x; i < here * cols; i += blockDim.x) {
      const int t = i / cols, c = i - t * cols;
      v[i] = c < cols_here ? a.mixed[static_cast<size_t>(first + t0 + t) * a.channels + v_col + c] : 0.f;
    }
    if (threadIdx.x < here) b[threadIdx.x] = a.beta[static_cast<size_t>(first + t0 + threadIdx.x) * a.heads + head];
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
        const float4 x = f4[r >> 2];
        const float keep[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
          for (int c = 0; c < C; ++c) {
            S[c][r + e] *= keep[e];
            sum[c] = __fmaf_rn(S[c][r + e], kk[r + e], sum[c]);
          }
      }
      for (int offset = lanes >> 1; offset > 0; offset >>= 1)
#pragma unroll
        for (int c = 0; c < C; ++c) sum[c] += __shfl_xor_sync(0xffffffffu, sum[c], offset);
      const float share = b[t];
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

}  // namespace delta

// =========================================================================================== launchers
using namespace delta;

// `longest`: the most new tokens a sequence of the batch brings; 1: the kernel also moves every sequence's convolution
// state up by its token, otherwise the caller updates the states afterwards (shrike_short_conv_keep).
SHRIKE_API int shrike_delta_prep(const float* fused, int partials, long long stride, int total, const float* taps, float* state,
                                 const int* q_start, const int* state_slot, const int* seq_of_token, float* mixed, float* beta,
                                 void* low, int dtype, int n, int heads, int kv_heads, int dim, int vdim, int taps_count,
                                 int beta_at, int low_at, int low_width, int num_slots, float unit_eps, float q_scale,
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
  const int units = 2 * kv_heads + heads + 1;
  const dim3 grid(static_cast<unsigned>((n + TILE - 1) / TILE), static_cast<unsigned>((units + 3) / 4));
  if (grid.y > 65535) return SHRIKE_BAD_ARGUMENT;
#define SHRIKE_PREP(TO, T, V) launch_dependent(delta_prep_kernel<TO, T, V>, grid, 128, 0, stream, a)
#define SHRIKE_PREP_TAPS(TO, V)                   \
  do {                                            \
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
  return shrike_launch_status();
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

SHRIKE_API int shrike_delta_scan(const float* mixed, const float* beta, const float* gates, int partials, long long stride,
                                 int gate_width, const float* rate, const float* bias, float* state, const int* q_start,
                                 const int* state_slot, float* out, int num_seqs, int heads, int kv_heads, int dim, int vdim,
                                 int head_stride, int num_slots, cudaStream_t stream) {
  if (num_seqs <= 0) return SHRIKE_OK;
  if (heads < 1 || heads > 65535 || num_seqs > 65535 || kv_heads < 1 || heads % kv_heads || dim < 1 || vdim < 1 || partials < 1 ||
      head_stride < dim * vdim || gate_width < heads * dim)
    return SHRIKE_BAD_ARGUMENT;
  if (head_stride % 4 || reinterpret_cast<uintptr_t>(state) % 16) return SHRIKE_BAD_ARGUMENT;
  DeltaShape shape;
  if (!delta_shape(dim, vdim, &shape)) return SHRIKE_BAD_ARGUMENT;   // heads of more than 1,024 rows
  ScanArgs a = {mixed, beta, gates, stride, partials, gate_width, rate, bias, state, q_start, state_slot, out,
                heads, kv_heads, dim, vdim, 2 * kv_heads * dim + heads * vdim, head_stride, num_slots, shape.lanes, shape.cols};
  void (*kernel)(ScanArgs) = shape.rows == 8 ? delta_walk_kernel<8, 4> : delta_walk_kernel<32, 1>;
  if (shape.smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(shape.smem));
  const dim3 grid(static_cast<unsigned>((vdim + shape.cols - 1) / shape.cols), heads, num_seqs);
  launch_dependent(kernel, grid, static_cast<unsigned>(shape.threads), shape.smem, stream, a);
  return shrike_launch_status();
}
