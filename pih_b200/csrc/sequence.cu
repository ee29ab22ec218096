// Kernels of mixers that carry a state from token to token, and of a residual stream kept in 32-bit.
//
//   embedding_stream      table rows (bf16 or fp32) times one number -> a 32-bit stream
//   rmsnorm_stream        h (fp32) += scale * (delta + bias) (+ the token's embedding and a vector: a loop's next pass);
//                         out = h / sqrt(mean(h^2) + eps) * w, w a vector or ONE number
//   stream_norm_norm      h (fp32) += rms(y + bias) * w1, or with a pair of outputs h += rms(rms(y + bias) * wl + rms(y2 + bias2) *
//                         wr) * w1; out = rms(h) * w2: a norm behind a sub-layer, the sum and the next norm in one pass
//   causal_conv           short causal convolution per channel over each request's rows, the last taps-1 inputs
//                         carried in the request's state slot
//   delta_prepare         unit-norm q and k per head, decay (one a head, or one a head and key channel) and write
//                         strength per head (32-bit)
//   delta_recurrence      gated delta rule: S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q
//   gated_rmsnorm         per-head RMS norm of the read-out (divided by a number a head first), times a weight, times silu(gate)
//                         or sigmoid(gate)
//   gated_part_rmsnorm    y * silu(gate), then an RMS norm in equal parts of the row with a weight a column
//   rglru_gates, _chain   real-gated linear recurrent unit: S <- a S + sqrt(1 - a^2) (i u), out = S * gelu(y)
//
// A step's rows are packed: request r owns rows cu_q[r] .. cu_q[r+1]-1 in the order of their positions, and
// state_slots[r] is its slot in the state tensor (fp32, ``state_stride`` numbers a slot).  Kernels that carry state
// are driven by requests, so rows of padding (no request) are never touched and requests of padding (no rows, slot -1)
// do nothing.  Everything that enters a recurrence is 32-bit: states, decays, gates, unit norms; only the inputs that
// come from projections and convolutions have the storage type T.  A request's result depends on its own rows and
// state alone, in an order of operations fixed by the row: cutting a prompt or batching it changes no bit.
#include "common.cuh"

namespace pih {

constexpr int kMaxTaps = 16;

__device__ __forceinline__ float gelu_tanh_f(float z) {
  return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

template <typename T>
__global__ void embedding_stream_kernel(const T* __restrict__ table, const int* __restrict__ ids, float* __restrict__ out,
                                        int hidden, int vocab, float scale, uint32_t* err) {
  wait_for_prior_kernels();
  launch_dependents();
  const int row = blockIdx.x;
  int id = ids[row];
  const bool bad = id < 0 || id >= vocab;
  if (bad) {
    if (threadIdx.x == 0) publish_error(err, kTokenOutOfVocabulary);
    id = 0;
  }
  for (int c = threadIdx.x; c < hidden; c += blockDim.x)
    out[static_cast<long long>(row) * hidden + c] = bad ? 0.0f : to_float<T>(table[static_cast<long long>(id) * hidden + c]) * scale;
}

// What is added to a row of the stream before it is normed: scale * (delta + bias), then, where a loop's next pass
// begins, table_scale * table[ids[row]] (the token's embedding once more) and a vector.  Null pointers: absent.
template <typename TD>
struct StreamAdd {
  const TD* delta;
  float scale;
  const float* bias;
  const TD* table;
  const int* ids;
  int vocab;
  float table_scale;
  const float* vec;
};

// ``n`` (V) neighbouring columns as one 16-byte load where V is 4
template <int V>
__device__ __forceinline__ void load_floats(float (&v)[V], const float* src) {
  if constexpr (V == 4) {
    const float4 f = *reinterpret_cast<const float4*>(src);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = src[i];
  }
}
template <int V>
__device__ __forceinline__ void load_floats(float (&v)[V], const __nv_bfloat16* src) {
  if constexpr (V == 4) {
    const uint2 w = *reinterpret_cast<const uint2*>(src);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.y));
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = __bfloat162float(src[i]);
  }
}
template <int V>
__device__ __forceinline__ void store_floats(float* dst, const float (&v)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
  else
#pragma unroll
    for (int i = 0; i < V; ++i) dst[i] = v[i];
}
template <int V>
__device__ __forceinline__ void store_floats(__nv_bfloat16* dst, const float (&v)[V]) {
  if constexpr (V == 4) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) dst[i] = __float2bfloat16_rn(v[i]);
  }
}

// The new values of columns c .. c + V - 1 of a row (32-bit sums).
template <typename TD, int V>
__device__ __forceinline__ void stream_sum(float (&v)[V], const float* hr, const TD* dr, const TD* er, const StreamAdd<TD>& add,
                                           int c) {
  load_floats<V>(v, hr + c);
  if (dr != nullptr) {
    float d[V];
    load_floats<V>(d, dr + c);
    if (add.bias != nullptr) {
      float b[V];
      load_floats<V>(b, add.bias + c);
#pragma unroll
      for (int i = 0; i < V; ++i) d[i] += b[i];
    }
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = fmaf(add.scale, d[i], v[i]);
  }
  if (er != nullptr) {
    float e[V];
    load_floats<V>(e, er + c);
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = fmaf(add.table_scale, e[i], v[i]);
  }
  if (add.vec != nullptr) {
    float e[V];
    load_floats<V>(e, add.vec + c);
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] += e[i];
  }
}

// One block a row.  Without ``rows`` the row's new sum is stored back and normed; with ``rows`` (a gather of the rows whose
// logits are wanted) nothing is stored: the sum is formed for the norm alone.  V columns a thread at a time; the first
// kHeld pieces of a thread stay in registers between the sum of squares and the writing, later ones are formed (or read)
// again.
template <typename TD, typename TO, int V>
__global__ void __launch_bounds__(512)
rmsnorm_stream_kernel(float* __restrict__ h, const StreamAdd<TD> add, const float* __restrict__ weight, int weight_len,
                      TO* __restrict__ out, const int* __restrict__ rows, int width, float eps) {
  constexpr int kHeld = 4;
  __shared__ float scratch[33];
  wait_for_prior_kernels();
  launch_dependents();
  const int row = rows != nullptr ? rows[blockIdx.x] : blockIdx.x;
  float* hr = h + static_cast<long long>(row) * width;
  const TD* dr = add.delta != nullptr ? add.delta + static_cast<long long>(row) * width : nullptr;
  const TD* er = nullptr;
  if (add.table != nullptr) {
    const int id = add.ids[row];                               // (a bad id was reported by the embedding)
    er = add.table + static_cast<long long>(id >= 0 && id < add.vocab ? id : 0) * width;
  }
  const bool changes = dr != nullptr || er != nullptr || add.vec != nullptr;
  const int step = static_cast<int>(blockDim.x) * V, c0 = static_cast<int>(threadIdx.x) * V;
  float held[kHeld][V];
  float ss = 0.0f;
#pragma unroll
  for (int u = 0; u < kHeld; ++u) {
    const int c = c0 + u * step;
    if (c < width) {
      stream_sum<TD, V>(held[u], hr, dr, er, add, c);
      if (changes && rows == nullptr) store_floats<V>(hr + c, held[u]);
#pragma unroll
      for (int i = 0; i < V; ++i) ss = fmaf(held[u][i], held[u][i], ss);
    }
  }
  for (int c = c0 + kHeld * step; c < width; c += step) {
    float v[V];
    stream_sum<TD, V>(v, hr, dr, er, add, c);
    if (changes && rows == nullptr) store_floats<V>(hr + c, v);
#pragma unroll
    for (int i = 0; i < V; ++i) ss = fmaf(v[i], v[i], ss);
  }
  ss = block_sum(ss, scratch);
  const float scale = 1.0f / sqrtf(ss / static_cast<float>(width) + eps);
  TO* o = out + static_cast<long long>(blockIdx.x) * width;
  auto write = [&](float (&v)[V], int c) {
    float w[V];
    if (weight_len == 1) {
#pragma unroll
      for (int i = 0; i < V; ++i) w[i] = weight[0];
    } else {
      load_floats<V>(w, weight + c);
    }
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = v[i] * scale * w[i];
    store_floats<V>(o + c, v);
  };
#pragma unroll
  for (int u = 0; u < kHeld; ++u) {
    const int c = c0 + u * step;
    if (c < width) write(held[u], c);
  }
  for (int c = c0 + kHeld * step; c < width; c += step) {
    float v[V];
    if (rows == nullptr) load_floats<V>(v, hr + c);            // (the thread's own store)
    else stream_sum<TD, V>(v, hr, dr, er, add, c);
    write(v, c);
  }
}

// Two sums over a block of up to 1024 threads at once, in an order that depends on blockDim only.
__device__ __forceinline__ float2 block_sum_pair(float2 v, float2* scratch /* 33 */) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
  v.x = warp_sum(v.x);
  v.y = warp_sum(v.y);
  __syncthreads();
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  if (warp == 0) {
    float2 t = lane < warps ? scratch[lane] : make_float2(0.0f, 0.0f);
    t.x = warp_sum(t.x);
    t.y = warp_sum(t.y);
    if (lane == 0) scratch[32] = t;
  }
  __syncthreads();
  return scratch[32];
}

// What a sub-layer gave, on its way through the norm behind it: y (+ bias) or a pair of outputs, each RMS-normed with a weight
// of its own and added.
template <typename TD>
struct NormedOutput {
  const TD* y;
  const float* bias;                                           // null: none
  const TD* y2;                                                // null: no pair
  const float* bias2;
  const float* weight_left;
  const float* weight_right;
  float pair_eps;
  const float* weight;                                         // of the norm behind the sub-layer
  float eps;
};

// One block a row, V columns a thread at a time, up to kNormHeld pieces a thread, all in registers.  With ``rows`` nothing
// is stored back and ``out`` holds the gathered rows.
constexpr int kNormHeld = 4;
template <typename TD, typename TO, int V>
__global__ void __launch_bounds__(1024)
stream_norm_norm_kernel(float* __restrict__ h, const NormedOutput<TD> add, const float* __restrict__ weight,
                        TO* __restrict__ out, const int* __restrict__ rows, int width, float eps) {
  __shared__ float2 scratch[33];
  wait_for_prior_kernels();
  launch_dependents();
  const int row = rows != nullptr ? rows[blockIdx.x] : blockIdx.x;
  float* hr = h + static_cast<long long>(row) * width;
  const TD* yr = add.y + static_cast<long long>(row) * width;
  const TD* yr2 = add.y2 != nullptr ? add.y2 + static_cast<long long>(row) * width : nullptr;
  const int step = static_cast<int>(blockDim.x) * V, c0 = static_cast<int>(threadIdx.x) * V;
  const float n = static_cast<float>(width);
  float u[kNormHeld][V], v[kNormHeld][V];
  float2 ss = make_float2(0.0f, 0.0f);
  auto with_bias = [&](float (&x)[V], const float* bias, int c) {
    if (bias != nullptr) {
      float b[V];
      load_floats<V>(b, bias + c);
#pragma unroll
      for (int i = 0; i < V; ++i) x[i] += b[i];
    }
  };
#pragma unroll
  for (int k = 0; k < kNormHeld; ++k) {
    const int c = c0 + k * step;
    if (c >= width) continue;
    load_floats<V>(u[k], yr + c);
    with_bias(u[k], add.bias, c);
#pragma unroll
    for (int i = 0; i < V; ++i) ss.x = fmaf(u[k][i], u[k][i], ss.x);
    if (yr2 != nullptr) {
      load_floats<V>(v[k], yr2 + c);
      with_bias(v[k], add.bias2, c);
#pragma unroll
      for (int i = 0; i < V; ++i) ss.y = fmaf(v[k][i], v[k][i], ss.y);
    }
  }
  ss = block_sum_pair(ss, scratch);
  if (yr2 != nullptr) {
    const float left = 1.0f / sqrtf(ss.x / n + add.pair_eps), right = 1.0f / sqrtf(ss.y / n + add.pair_eps);
    ss = make_float2(0.0f, 0.0f);
#pragma unroll
    for (int k = 0; k < kNormHeld; ++k) {
      const int c = c0 + k * step;
      if (c >= width) continue;
      float wl[V], wr[V];
      load_floats<V>(wl, add.weight_left + c);
      load_floats<V>(wr, add.weight_right + c);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        u[k][i] = fmaf(v[k][i] * right, wr[i], u[k][i] * left * wl[i]);
        ss.x = fmaf(u[k][i], u[k][i], ss.x);
      }
    }
    ss = block_sum_pair(ss, scratch);
  }
  const float behind = 1.0f / sqrtf(ss.x / n + add.eps);
  ss = make_float2(0.0f, 0.0f);
#pragma unroll
  for (int k = 0; k < kNormHeld; ++k) {
    const int c = c0 + k * step;
    if (c >= width) continue;
    float w[V];
    load_floats<V>(w, add.weight + c);
    load_floats<V>(v[k], hr + c);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      v[k][i] = fmaf(u[k][i] * behind, w[i], v[k][i]);
      ss.x = fmaf(v[k][i], v[k][i], ss.x);
    }
    if (rows == nullptr) store_floats<V>(hr + c, v[k]);
  }
  ss = block_sum_pair(ss, scratch);
  const float scale = 1.0f / sqrtf(ss.x / n + eps);
  TO* o = out + static_cast<long long>(blockIdx.x) * width;
#pragma unroll
  for (int k = 0; k < kNormHeld; ++k) {
    const int c = c0 + k * step;
    if (c >= width) continue;
    float w[V];
    load_floats<V>(w, weight + c);
#pragma unroll
    for (int i = 0; i < V; ++i) v[k][i] = v[k][i] * scale * w[i];
    store_floats<V>(o + c, v[k]);
  }
}

// Block (32 channels, 8 token lanes) computes 128 rows of a request for 32 channels; blockIdx.z counts the stretches of
// 128 rows (launched for the step's row count; stretches beyond a request's rows leave).
// in(s) = x[s] + in_bias for s >= 0, the history for -(taps-1) <= s < 0 (zeros at the start of a sequence).
// out[t] = act( sum_j w[c][j] in(t - (taps-1) + j) + out_bias ).  The history is only read here; causal_conv_history
// replaces it afterwards.
constexpr int kConvRows = 128;

// kTaps: the number of taps at most; an instance of the usual sizes shifts and multiplies no more than it has to.
template <typename T, int kTaps>
__global__ void __launch_bounds__(256)
causal_conv_kernel(const T* __restrict__ x, long long ldx, const T* __restrict__ w, const float* __restrict__ in_bias,
                   const float* __restrict__ out_bias, T* __restrict__ out, long long ldo, int channels, int taps,
                   int activation, const float* __restrict__ state, long long state_stride, long long state_offset,
                   const int* __restrict__ cu_q, const int* __restrict__ state_slots) {
  wait_for_prior_kernels();
  launch_dependents();
  const int r = blockIdx.x;
  const int c = blockIdx.y * 32 + threadIdx.x;
  const int lo = cu_q[r], n = cu_q[r + 1] - lo;
  const int slot = state_slots[r];
  const int t_first = blockIdx.z * kConvRows;
  if (n <= t_first || slot < 0 || c >= channels) return;
  const int hist_n = taps - 1;
  const float* st = state + slot * state_stride + state_offset;       // [taps-1][channels]
  float wr[kTaps];
#pragma unroll
  for (int j = 0; j < kTaps; ++j) wr[j] = j < taps ? to_float<T>(w[static_cast<long long>(c) * taps + j]) : 0.0f;
  const float ib = in_bias != nullptr ? in_bias[c] : 0.0f;
  const float ob = out_bias != nullptr ? out_bias[c] : 0.0f;
  // a token lane takes a run of consecutive rows and keeps the last taps inputs in registers: every input is read once
  const int per = kConvRows / static_cast<int>(blockDim.y);
  const int t0 = t_first + static_cast<int>(threadIdx.y) * per, t1 = min(n, t0 + per);
  if (t0 >= t1) return;
  auto input = [&](int s) {
    return s >= 0 ? to_float<T>(x[static_cast<long long>(lo + s) * ldx + c]) + ib
                  : st[static_cast<long long>(hist_n + s) * channels + c];
  };
  float held[kTaps];                                       // held[j] = in(t - hist_n + j), j < taps
#pragma unroll
  for (int j = 0; j < kTaps; ++j) held[j] = (j + 1 < taps) ? input(t0 - hist_n + j) : 0.0f;
#pragma unroll 4
  for (int t = t0; t < t1; ++t) {
    const float newest = input(t);
    float acc = 0.0f;
#pragma unroll
    for (int j = 0; j < kTaps; ++j) {
      if (j < taps) {
        const float v = j + 1 == taps ? newest : held[j];
        acc = fmaf(wr[j], v, acc);
      }
    }
#pragma unroll
    for (int j = 0; j + 1 < kTaps; ++j) held[j] = j + 2 == taps ? newest : held[j + 1];
    acc += ob;
    if (activation == 1) acc = acc / (1.0f + expf(-acc));
    out[static_cast<long long>(lo + t) * ldo + c] = from_float<T>(acc);
  }
}

// Thread a (request, channel): the history becomes the last taps-1 inputs of [old history, the step's rows].
template <typename T>
__global__ void __launch_bounds__(128)
causal_conv_history_kernel(const T* __restrict__ x, long long ldx, const float* __restrict__ in_bias, int channels, int taps,
                           float* __restrict__ state, long long state_stride, long long state_offset,
                           const int* __restrict__ cu_q, const int* __restrict__ state_slots) {
  wait_for_prior_kernels();
  launch_dependents();
  const int r = blockIdx.x;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  const int lo = cu_q[r], n = cu_q[r + 1] - lo;
  const int slot = state_slots[r];
  if (n <= 0 || slot < 0 || c >= channels) return;
  const int hist_n = taps - 1;
  float* st = state + slot * state_stride + state_offset;
  const float ib = in_bias != nullptr ? in_bias[c] : 0.0f;
  float keep[kMaxTaps];
#pragma unroll
  for (int j = 0; j < kMaxTaps; ++j) {
    keep[j] = 0.0f;
    if (j < hist_n) {
      const int s = n - hist_n + j;
      keep[j] = s >= 0 ? to_float<T>(x[static_cast<long long>(lo + s) * ldx + c]) + ib
                       : st[static_cast<long long>(hist_n + s) * channels + c];
    }
  }
#pragma unroll
  for (int j = 0; j < kMaxTaps; ++j)
    if (j < hist_n) st[static_cast<long long>(j) * channels + c] = keep[j];
}

// Block (row, part): part 0 the vectors and the write strengths — and the decays, where it is the only part —, part p > 0 the
// decays kDecaySlice (p - 1) and on.  qk: [rows, ld] with q heads at column 0 and k heads at column kv_heads*dim (after convolution and
// activation); b: [rows, ldb] write-strength logits a head; a: [rows, lda] decay logits, one a head or (``channels``) one a
// head and key channel, [heads, dim], with a bias of the same layout; decay_log: one a head.
// qn, kn: fp32 [rows, kv_heads, dim]; qk_dot: their product k . q, fp32 [rows, kv_heads]; decay (as g - 1): fp32 [rows,
// heads] or [rows, heads, dim]; beta: fp32 [rows, heads].
constexpr int kDecaySlice = 512;

template <typename T, typename TA>
__global__ void __launch_bounds__(128)
delta_prepare_kernel(const T* __restrict__ qk, long long ld, const T* __restrict__ b, long long ldb,
                     const TA* __restrict__ a, long long lda, int channels,
                     const float* __restrict__ decay_log, const float* __restrict__ decay_bias, float* __restrict__ qn,
                     float* __restrict__ kn, float* __restrict__ qk_dot, float* __restrict__ decay, float* __restrict__ beta,
                     int heads, int kv_heads, int dim, float unit_eps, float q_scale) {
  wait_for_prior_kernels();
  launch_dependents();
  const int row = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  for (int g = warp; g < kv_heads && blockIdx.y == 0; g += warps) {
    const T* q = qk + static_cast<long long>(row) * ld + static_cast<long long>(g) * dim;
    const T* k = q + static_cast<long long>(kv_heads) * dim;
    float sq = 0.0f, sk = 0.0f;
    for (int i = lane; i < dim; i += 32) {
      const float x = to_float<T>(q[i]), y = to_float<T>(k[i]);
      sq = fmaf(x, x, sq);
      sk = fmaf(y, y, sk);
    }
    sq = (1.0f / sqrtf(warp_sum(sq) + unit_eps)) * q_scale;
    sk = 1.0f / sqrtf(warp_sum(sk) + unit_eps);
    const long long at = (static_cast<long long>(row) * kv_heads + g) * dim;
    float dot = 0.0f;
    for (int i = lane; i < dim; i += 32) {
      const float x = to_float<T>(q[i]) * sq, y = to_float<T>(k[i]) * sk;
      qn[at + i] = x;
      kn[at + i] = y;
      dot = fmaf(x, y, dot);
    }
    dot = warp_sum(dot);
    if (lane == 0) qk_dot[static_cast<long long>(row) * kv_heads + g] = dot;
  }
  for (int h = threadIdx.x; h < heads && blockIdx.y == 0; h += blockDim.x) {
    beta[static_cast<long long>(row) * heads + h] = sigmoid_f(to_float<T>(b[static_cast<long long>(row) * ldb + h]));
  }
  // g - 1 rather than g: a decay next to 1 keeps its distance from 1 to full precision (see rglru_gates_kernel)
  const int per = channels ? dim : 1;
  const long long row_a = static_cast<long long>(row) * lda, row_g = static_cast<long long>(row) * heads * per;
  const bool sliced = gridDim.y > 1;
  if (sliced && blockIdx.y == 0) return;
  const int from = sliced ? (static_cast<int>(blockIdx.y) - 1) * kDecaySlice : 0;
  const int to = sliced ? min(heads * per, from + kDecaySlice) : heads * per;
  for (int i = from + threadIdx.x; i < to; i += blockDim.x)
    decay[row_g + i] = expm1f(-expf(decay_log[i / per]) * softplus_f(to_float<TA>(a[row_a + i]) + decay_bias[i]));
}

// Block (request, head, slice of value columns); thread j owns column v0 + j of S (all ``dim`` rows, in shared memory:
// S[i][j], conflict-free).  The next token's k and q (and, with kChannel, its decay a key channel) are fetched into
// registers while this token is computed.
template <typename T, bool kChannel>
__global__ void delta_recurrence_kernel(const float* __restrict__ qn, const float* __restrict__ kn, const T* __restrict__ v,
                                        long long ldv, const float* __restrict__ decay, const float* __restrict__ beta,
                                        float* __restrict__ out, float* __restrict__ state, long long state_stride,
                                        const int* __restrict__ cu_q, const int* __restrict__ state_slots, int heads,
                                        int kv_heads, int dim, int vdim) {
  extern __shared__ float smem[];
  wait_for_prior_kernels();
  launch_dependents();
  const int r = blockIdx.x, h = blockIdx.y;
  const int cols = blockDim.x;
  const int j = threadIdx.x, col = blockIdx.z * cols + j;
  const int lo = cu_q[r], hi = cu_q[r + 1];
  const int slot = state_slots[r];
  if (hi <= lo || slot < 0) return;
  const int kh = h / (heads / kv_heads);
  float* S = smem;                          // [dim][cols]
  constexpr int kVecs = kChannel ? 3 : 2;
  float* kq = smem + dim * cols;            // [2 buffers][k: dim | q: dim | decay - 1: dim]
  const bool live = col < vdim;
  float* Sg = state + slot * state_stride + (static_cast<long long>(h) * dim) * vdim;
  for (int i = 0; i < dim; ++i) S[i * cols + j] = live ? Sg[static_cast<long long>(i) * vdim + col] : 0.0f;
  const int per = (kVecs * dim + cols - 1) / cols;               // numbers of k|q|decay a thread fetches
  auto fetch = [&](int t, int e) -> float {
    const int idx = j + e * cols;
    if (idx >= kVecs * dim) return 0.0f;
    if (kChannel && idx >= 2 * dim) return decay[(static_cast<long long>(t) * heads + h) * dim + (idx - 2 * dim)];
    const float* src = idx < dim ? kn : qn;
    return src[(static_cast<long long>(t) * kv_heads + kh) * dim + (idx < dim ? idx : idx - dim)];
  };
  constexpr int kMaxPer = 8 * kVecs;        // dim <= 8 * cols
  float nxt[kMaxPer];
#pragma unroll
  for (int e = 0; e < kMaxPer; ++e) nxt[e] = e < per ? fetch(lo, e) : 0.0f;
  for (int t = lo; t < hi; ++t) {
    float* cur = kq + (t & 1) * kVecs * dim;
#pragma unroll
    for (int e = 0; e < kMaxPer; ++e)
      if (e < per && j + e * cols < kVecs * dim) cur[j + e * cols] = nxt[e];
    __syncthreads();
    if (t + 1 < hi) {
#pragma unroll
      for (int e = 0; e < kMaxPer; ++e) nxt[e] = e < per ? fetch(t + 1, e) : 0.0f;
    }
    const float b = beta[static_cast<long long>(t) * heads + h];
    const float vj = live ? to_float<T>(v[static_cast<long long>(t) * ldv + static_cast<long long>(h) * vdim + col]) : 0.0f;
    const float* k = cur;
    const float* q = cur + dim;
    // g - 1; g x is formed as x + (g - 1) x.  One decay a head multiplies the finished dot product, one a key channel the
    // rows of S first
    const float* gc = cur + 2 * dim;
    const float gm1 = kChannel ? 0.0f : decay[static_cast<long long>(t) * heads + h];
    auto decayed = [&](int i) {
      const float x = S[i * cols + j];
      return fmaf(kChannel ? gc[i] : gm1, x, x);
    };
    float a0 = 0.0f, a1 = 0.0f, a2 = 0.0f, a3 = 0.0f;
    int i = 0;
    for (; i + 4 <= dim; i += 4) {
      a0 = fmaf(kChannel ? decayed(i + 0) : S[(i + 0) * cols + j], k[i + 0], a0);
      a1 = fmaf(kChannel ? decayed(i + 1) : S[(i + 1) * cols + j], k[i + 1], a1);
      a2 = fmaf(kChannel ? decayed(i + 2) : S[(i + 2) * cols + j], k[i + 2], a2);
      a3 = fmaf(kChannel ? decayed(i + 3) : S[(i + 3) * cols + j], k[i + 3], a3);
    }
    for (; i < dim; ++i) a0 = fmaf(kChannel ? decayed(i) : S[i * cols + j], k[i], a0);
    const float dot = (a0 + a1) + (a2 + a3);
    const float u = b * (vj - (kChannel ? dot : fmaf(gm1, dot, dot)));
    float o0 = 0.0f, o1 = 0.0f, o2 = 0.0f, o3 = 0.0f;
    i = 0;
    for (; i + 4 <= dim; i += 4) {
      const float s0 = fmaf(k[i + 0], u, decayed(i + 0));
      const float s1 = fmaf(k[i + 1], u, decayed(i + 1));
      const float s2 = fmaf(k[i + 2], u, decayed(i + 2));
      const float s3 = fmaf(k[i + 3], u, decayed(i + 3));
      S[(i + 0) * cols + j] = s0; S[(i + 1) * cols + j] = s1; S[(i + 2) * cols + j] = s2; S[(i + 3) * cols + j] = s3;
      o0 = fmaf(s0, q[i + 0], o0); o1 = fmaf(s1, q[i + 1], o1); o2 = fmaf(s2, q[i + 2], o2); o3 = fmaf(s3, q[i + 3], o3);
    }
    for (; i < dim; ++i) {
      const float s0 = fmaf(k[i], u, decayed(i));
      S[i * cols + j] = s0;
      o0 = fmaf(s0, q[i], o0);
    }
    if (live) out[(static_cast<long long>(t) * heads + h) * vdim + col] = (o0 + o1) + (o2 + o3);
  }
  if (live)
    for (int i = 0; i < dim; ++i) Sg[static_cast<long long>(i) * vdim + col] = S[i * cols + j];
}

// The same recurrence with S in registers, for the key sizes that have an instance.  Block (request, head, 16 value
// columns); a column of S is held by 8 threads (4 for small keys, 16 for 256), thread (column c = tid / parts, part p = tid %
// parts) every parts-th piece of four rows from piece p on: the parts of a column sit in neighbouring lanes, meet through
// shuffles, and read neighbouring 16-byte pieces of k and q (no bank conflicts).
//
// What a token costs is the chain from its state to the next one's, so both products that read the state are taken from the
// SAME (decayed) state g S and meet in the same shuffles: with a = (g S)^T k and b = (g S)^T q,
//     u = beta (v - a),    o = b + (k . q) u,    S <- g S + k u^T
// — the read-out of the state after the write, without reading it again; k . q comes from delta_prepare.  Products and
// updates take two numbers an instruction (fma.rn.f32x2: each half rounds as fma.rn.f32 does).
//
// What the recurrence reads of a token (k, q, k . q, the block's values, decay, write strength) is staged in shared memory
// a chunk of tokens at a time, two buffers: the next chunk's numbers are copied asynchronously while this chunk is computed,
// so no load from memory and only one barrier a chunk lie on the chain from token to token; a token's numbers go from there
// to registers one token ahead.  The order of the additions is fixed by the kernel, not by the step's make-up or by where a
// chunk begins.  With kChannel the decay (as g - 1, [rows, heads, kDim]) multiplies the rows of S; it is staged like k and q.
__device__ __forceinline__ void async_copy_16(void* smem_dst, const void* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(smem_dst))), "l"(src));
}
__device__ __forceinline__ void async_copy_4(void* smem_dst, const void* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(smem_dst))), "l"(src));
}
__device__ __forceinline__ void async_copies_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void async_copies_wait() { asm volatile("cp.async.wait_all;" ::: "memory"); }

template <int kDim, bool kChannel>
struct DeltaShape {
  static constexpr int kParts = kDim >= 256 ? 16 : (kDim >= 64 ? 8 : 4);   // threads a column of S
  static constexpr int kCols = 16;                        // value columns a block
  static constexpr int kThreads = kCols * kParts;
  static constexpr int kRows = kDim / kParts;             // rows of S a thread holds
  static constexpr int kVecs = kChannel ? 3 : 2;          // vectors of kDim numbers staged a token: k | q (| decay - 1)
  static constexpr int kChunk = kDim <= 128 ? 16 : 8;     // tokens staged at a time (even)
  static constexpr int kTail = kVecs * kDim;              // where what is not a vector of kDim numbers begins
  // words staged a token: vectors | decay - 1, write strength, k . q, pad | the block's values
  static constexpr int words(int value_bytes) { return kTail + 4 + kCols * value_bytes / 4; }
};

template <typename T, int kDim, bool kChannel>
__global__ void __launch_bounds__(DeltaShape<kDim, kChannel>::kThreads)
delta_recurrence_reg_kernel(const float* __restrict__ qn, const float* __restrict__ kn, const float* __restrict__ qk_dot,
                            const T* __restrict__ v, long long ldv, const float* __restrict__ decay,
                            const float* __restrict__ beta, float* __restrict__ out, float* __restrict__ state,
                            long long state_stride, const int* __restrict__ cu_q, const int* __restrict__ state_slots,
                            int heads, int kv_heads, int vdim) {
  typedef DeltaShape<kDim, kChannel> Shape;
  constexpr int kParts = Shape::kParts, kThreads = Shape::kThreads, kRows = Shape::kRows;
  constexpr int kChunk = Shape::kChunk, kCols = Shape::kCols, kPairs = kRows / 2, kTail = Shape::kTail;
  constexpr int kVWords = kCols * sizeof(T) / 4;          // the block's values of a token, in 32-bit words
  constexpr int kTok = Shape::words(sizeof(T));
  extern __shared__ __align__(16) float stage[];          // [2][kChunk][kTok]
  wait_for_prior_kernels();
  launch_dependents();
  const int r = blockIdx.x, h = blockIdx.y;
  const int tid = threadIdx.x, part = tid % kParts, cl = tid / kParts, col0 = blockIdx.z * kCols, col = col0 + cl;
  const int lo = cu_q[r], hi = cu_q[r + 1];
  const int slot = state_slots[r];
  if (hi <= lo || slot < 0) return;
  const int kh = h / (heads / kv_heads);
  const bool live = col < vdim;
  float* Sg = state + slot * state_stride + static_cast<long long>(h) * kDim * vdim + col;
  // S[i]: rows row_of(i) and row_of(i) + 1
  auto row_of = [&](int i) { return 4 * (part + kParts * (i >> 1)) + 2 * (i & 1); };
  float2 S[kPairs];
#pragma unroll
  for (int i = 0; i < kPairs; ++i) {
    const float* at = Sg + static_cast<long long>(row_of(i)) * vdim;
    S[i] = live ? make_float2(at[0], at[vdim]) : make_float2(0.0f, 0.0f);
  }
  // the copies of the chunk that starts at token t0, into buffer b: straight from memory into shared memory, so that
  // they are under way while the chunk before is computed.  A thread copies the same piece of every kStep-th token.
  constexpr int kPieces = kDim / 4, kStep = kThreads / kPieces;
  constexpr int kVStep = kThreads / kVWords;
  const int c_tok = tid / kPieces, c_at = (tid % kPieces) * 4;
  const int v_tok = tid / kVWords, v_word = tid % kVWords;
  const bool v_there = col0 + v_word * (4 / static_cast<int>(sizeof(T))) < vdim;
  const T* v_src = v + static_cast<long long>(h) * vdim + col0 + v_word * (4 / static_cast<int>(sizeof(T)));
  auto issue = [&](int t0, int b) {
    const int n_tok = min(kChunk, hi - t0);
    float* base = stage + b * kChunk * kTok;
#pragma unroll
    for (int tok = c_tok; tok < kChunk; tok += kStep) {
      if (tok < n_tok) {
        float* dst = base + tok * kTok + c_at;
        const long long at = (static_cast<long long>(t0 + tok) * kv_heads + kh) * kDim + c_at;
        async_copy_16(dst, kn + at);
        async_copy_16(dst + kDim, qn + at);
        if constexpr (kChannel)
          async_copy_16(dst + 2 * kDim, decay + (static_cast<long long>(t0 + tok) * heads + h) * kDim + c_at);
      }
    }
#pragma unroll
    for (int tok = v_tok; tok < kChunk; tok += kVStep)
      if (tok < n_tok && v_there) async_copy_4(base + tok * kTok + kTail + 4 + v_word, v_src + (t0 + tok) * ldv);
    const int tok = tid >> 2, which = tid & 3;               // 0: decay - 1, 1: write strength, 2: k . q
    if (tok < n_tok && which < 3 && !(kChannel && which == 0)) {
      const long long at = static_cast<long long>(t0 + tok) * heads + h;
      async_copy_4(base + tok * kTok + kTail + which,
                   which == 2 ? qk_dot + static_cast<long long>(t0 + tok) * kv_heads + kh : (which ? beta : decay) + at);
    }
    async_copies_commit();
  };
  // a token's numbers from the staging buffer into registers, one token ahead of the arithmetic
  struct Tok { float2 k[kPairs], q[kPairs], g[kChannel ? kPairs : 1]; float b, kq, v; };
  auto load_vec = [&](float2* dst, const float* src) {
#pragma unroll
    for (int i = 0; i < kPairs; i += 2) {
      const float4 f = *reinterpret_cast<const float4*>(src + 2 * kParts * i + 4 * part);
      dst[i] = make_float2(f.x, f.y);
      dst[i + 1] = make_float2(f.z, f.w);
    }
  };
  auto load = [&](Tok& x, const float* cur) {
    load_vec(x.k, cur);
    load_vec(x.q, cur + kDim);
    if constexpr (kChannel) {
      load_vec(x.g, cur + 2 * kDim);
    } else {
      x.g[0] = make_float2(cur[kTail], cur[kTail]);
    }
    x.b = cur[kTail + 1];
    x.kq = cur[kTail + 2];
    x.v = to_float<T>(reinterpret_cast<const T*>(cur + kTail + 4)[cl]);
  };
  auto compute = [&](const Tok& x, int t) {
    // two chains a product; the parts' sums of both products go through the shuffles side by side
    float2 a0 = make_float2(0.0f, 0.0f), a1 = a0, b0 = a0, b1 = a0;
#pragma unroll
    for (int i = 0; i < kPairs; i += 2) {
      S[i] = fma2(x.g[kChannel ? i : 0], S[i], S[i]);            // g S, formed as S + (g - 1) S
      S[i + 1] = fma2(x.g[kChannel ? i + 1 : 0], S[i + 1], S[i + 1]);
      a0 = fma2(S[i], x.k[i], a0);
      a1 = fma2(S[i + 1], x.k[i + 1], a1);
      b0 = fma2(S[i], x.q[i], b0);
      b1 = fma2(S[i + 1], x.q[i + 1], b1);
    }
    float a = (a0.x + a1.x) + (a0.y + a1.y), b = (b0.x + b1.x) + (b0.y + b1.y);
#pragma unroll
    for (int m = 1; m < kParts; m <<= 1) {
      const float pa = __shfl_xor_sync(0xffffffffu, a, m), pb = __shfl_xor_sync(0xffffffffu, b, m);
      a += pa;
      b += pb;
    }
    const float u = x.b * (x.v - a);
    const float2 uu = make_float2(u, u);
#pragma unroll
    for (int i = 0; i < kPairs; ++i) S[i] = fma2(x.k[i], uu, S[i]);
    if (live && part == 0) out[(static_cast<long long>(t) * heads + h) * vdim + col] = fmaf(x.kq, u, b);
  };
  issue(lo, 0);
  async_copies_wait();
  __syncthreads();
  int buf = 0;
  for (int t0 = lo; t0 < hi; t0 += kChunk) {
    if (t0 + kChunk < hi) issue(t0 + kChunk, buf ^ 1);
    const int n_tok = min(kChunk, hi - t0);
    const float* base = stage + buf * kChunk * kTok;
    Tok x0, x1;
    load(x0, base);
    if (n_tok == kChunk) {                                       // no branch a token: loads and sums of neighbours overlap
#pragma unroll 2
      for (int tok = 0; tok < kChunk; tok += 2) {
        load(x1, base + (tok + 1) * kTok);
        compute(x0, t0 + tok);
        load(x0, base + min(tok + 2, kChunk - 1) * kTok);        // (the last one is not used)
        compute(x1, t0 + tok + 1);
      }
    } else {
      for (int tok = 0; tok < n_tok; ++tok) {
        load(x0, base + tok * kTok);
        compute(x0, t0 + tok);
      }
    }
    async_copies_wait();
    __syncthreads();
    buf ^= 1;
  }
  if (live) {
#pragma unroll
    for (int i = 0; i < kPairs; ++i) {
      float* at = Sg + static_cast<long long>(row_of(i)) * vdim;
      at[0] = S[i].x;
      at[vdim] = S[i].y;
    }
  }
}

// One warp a (row, head): o fp32 [rows, heads, vdim]; gate [rows, ldg] and out [rows, ldo] with head h at column h * vdim.
// activation 0: silu(gate), 1: sigmoid(gate); out_scale multiplies.  divisor: fp32 [rows, heads] or null, divides o before the
// norm; head_weight: how far the weights of two heads lie apart (0: one weight for all heads).
template <typename TG, typename T>
__global__ void __launch_bounds__(128)
gated_rmsnorm_kernel(const float* __restrict__ o, const TG* __restrict__ gate, long long ldg, const float* __restrict__ weight,
                     T* __restrict__ out, long long ldo, long long rows_heads, int heads, int vdim, float eps, int activation,
                     float out_scale, const float* __restrict__ divisor, int head_weight) {
  wait_for_prior_kernels();
  launch_dependents();
  const long long item = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (item >= rows_heads) return;
  const int lane = threadIdx.x & 31;
  const long long row = item / heads;
  const int h = static_cast<int>(item % heads);
  const float* src = o + item * vdim;
  const float share = divisor != nullptr ? 1.0f / divisor[item] : 1.0f;
  weight += static_cast<long long>(h) * head_weight;
  float ss = 0.0f;
  for (int i = lane; i < vdim; i += 32) {
    const float x = src[i] * share;
    ss = fmaf(x, x, ss);
  }
  ss = warp_sum(ss);
  const float scale = share / sqrtf(ss / static_cast<float>(vdim) + eps) * out_scale;
  const TG* g = gate + row * ldg + static_cast<long long>(h) * vdim;
  T* dst = out + row * ldo + static_cast<long long>(h) * vdim;
  for (int i = lane; i < vdim; i += 32) {
    const float z = to_float<TG>(g[i]);
    dst[i] = from_float<T>(src[i] * scale * weight[i] * ((activation == 1 ? 1.0f : z) / (1.0f + expf(-z))));
  }
}

// Block (row, part): y fp32 [rows, width] times silu(gate [rows, ldg]), the part's own RMS norm, a weight a column.
template <typename T>
__global__ void __launch_bounds__(512)
gated_part_rmsnorm_kernel(const float* __restrict__ y, const T* __restrict__ gate, long long ldg,
                          const float* __restrict__ weight, T* __restrict__ out, long long ldo, int width, int part,
                          float eps, float out_scale) {
  __shared__ float scratch[33];
  wait_for_prior_kernels();
  launch_dependents();
  constexpr int kHeld = 4;
  const long long row = blockIdx.x;
  const int c0 = blockIdx.y * part;
  const float* yr = y + row * width + c0;
  const T* gr = gate + row * ldg + c0;
  auto gated = [&](int i) {
    const float z = to_float<T>(gr[i]);
    return yr[i] * (z / (1.0f + expf(-z)));
  };
  float held[kHeld];
  float ss = 0.0f;
#pragma unroll
  for (int k = 0; k < kHeld; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    held[k] = i < part ? gated(i) : 0.0f;
    ss = fmaf(held[k], held[k], ss);
  }
  for (int i = threadIdx.x + kHeld * blockDim.x; i < part; i += blockDim.x) {
    const float v = gated(i);
    ss = fmaf(v, v, ss);
  }
  ss = block_sum(ss, scratch);
  const float scale = out_scale / sqrtf(ss / static_cast<float>(part) + eps);
  T* o = out + row * ldo + c0;
#pragma unroll
  for (int k = 0; k < kHeld; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < part) o[i] = from_float<T>(held[k] * scale * weight[c0 + i]);
  }
  for (int i = threadIdx.x + kHeld * blockDim.x; i < part; i += blockDim.x) o[i] = from_float<T>(gated(i) * scale * weight[c0 + i]);
}

// The unit in two kernels.  rglru_gates (a thread a (row, channel), every row at once): from the gate logits
// (gates: fp32 [rows, blocks, 2 * bw]: block b's decay-gate logits, then its input-gate logits, without their biases),
// the convolution's output u and the other branch y_pre [rows, ldy] before its bias and GELU, the three numbers that
// the recurrence needs of a token: coef[row][c] = (a - 1, sqrt(1 - a^2) * i * u, gelu(y), 0).  rglru_chain (a thread a
// (request, channel)): S <- S + (a - 1) S + b, out = S * y over the request's rows in order, eight tokens' numbers in
// flight ahead of the chain (sixteen tokens fetched while sixteen are computed).
template <typename T>
__global__ void __launch_bounds__(256)
rglru_gates_kernel(const T* __restrict__ u, long long ldu, const float* __restrict__ gates, const T* __restrict__ y_pre,
                   long long ldy, const float* __restrict__ y_bias, const float* __restrict__ r_bias,
                   const float* __restrict__ i_bias, const float* __restrict__ lam, float decay_scale,
                   float4* __restrict__ coef, int rows, int width, int blocks) {
  wait_for_prior_kernels();
  launch_dependents();
  const long long idx = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (idx >= static_cast<long long>(rows) * width) return;
  const int t = static_cast<int>(idx / width), c = static_cast<int>(idx % width);
  const int bw = width / blocks, b = c / bw, o = c % bw;
  const float* g = gates + (static_cast<long long>(t) * blocks + b) * (2 * bw);
  const float rg = sigmoid_f(g[o] + r_bias[c]);
  const float ig = sigmoid_f(g[bw + o] + i_bias[c]);
  const float log_a = -(decay_scale * softplus_f(lam[c])) * rg;
  // a = exp(log_a) lies next to 1 for a channel that remembers long, where 32-bit numbers are 6e-8 apart: a rounded
  // there would be off by a few percent of 1 - a, and a thousand steps would multiply that up.  So a - 1 and
  // 1 - a^2 come from expm1, and a S is formed as S + (a - 1) S.
  const float am1 = expm1f(log_a);
  const float mult = sqrtf(-expm1f(2.0f * log_a));
  const float y = gelu_tanh_f(to_float<T>(y_pre[static_cast<long long>(t) * ldy + c]) + y_bias[c]);
  coef[idx] = make_float4(am1, mult, ig * to_float<T>(u[static_cast<long long>(t) * ldu + c]), y);
}

template <typename T>
__global__ void __launch_bounds__(128)
rglru_chain_kernel(const float4* __restrict__ coef, T* __restrict__ out, long long ldo, float* __restrict__ state,
                   long long state_stride, const int* __restrict__ cu_q, const int* __restrict__ state_slots, int width) {
  wait_for_prior_kernels();
  launch_dependents();
  const int r = blockIdx.x;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  const int lo = cu_q[r], hi = cu_q[r + 1];
  const int slot = state_slots[r];
  if (hi <= lo || slot < 0 || c >= width) return;
  float S = state[slot * state_stride + c];
  constexpr int kAhead = 16;
  float4 cur[kAhead], nxt[kAhead];
  auto fetch = [&](float4 (&f)[kAhead], int t0) {
#pragma unroll
    for (int i = 0; i < kAhead; ++i)
      f[i] = t0 + i < hi ? coef[static_cast<long long>(t0 + i) * width + c] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  };
  auto chain = [&](const float4 (&f)[kAhead], int t0) {
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      if (t0 + i < hi) {
        S = fmaf(f[i].x, S, fmaf(f[i].y, f[i].z, S));
        out[static_cast<long long>(t0 + i) * ldo + c] = from_float<T>(S * f[i].w);
      }
    }
  };
  fetch(cur, lo);
  for (int t0 = lo; t0 < hi; t0 += 2 * kAhead) {           // the next sixteen tokens' numbers are under way during the chain
    fetch(nxt, t0 + kAhead);
    chain(cur, t0);
    fetch(cur, t0 + 2 * kAhead);
    chain(nxt, t0 + kAhead);
  }
  state[slot * state_stride + c] = S;
}


}  // namespace pih

using namespace pih;
typedef __nv_bfloat16 bf16;

extern "C" int pih_embedding_stream(int dtype, const void* table, const void* ids, void* out, int rows, int hidden,
                                    int vocab, float scale, void* err, void* stream) {
  if (rows <= 0) return 0;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int threads = hidden >= 256 ? 256 : 64;
  if (dtype == PIH_F32)
    launch_kernel(embedding_stream_kernel<float>, dim3(rows), dim3(threads), 0, s, static_cast<const float*>(table),
                  static_cast<const int*>(ids), static_cast<float*>(out), hidden, vocab, scale, static_cast<uint32_t*>(err));
  else if (dtype == PIH_BF16)
    launch_kernel(embedding_stream_kernel<bf16>, dim3(rows), dim3(threads), 0, s, static_cast<const bf16*>(table),
                  static_cast<const int*>(ids), static_cast<float*>(out), hidden, vocab, scale, static_cast<uint32_t*>(err));
  else
    return PIH_ERR_BAD_ARGUMENT;
  PIH_LAUNCH_CHECK();
  return 0;
}

// h [.., width] fp32: h += delta_scale * (delta + bias), then += table_scale * table[ids[row]] (where table is given: of
// the delta's dtype, [vocab, width]) and += vec (fp32 [width]); out: the normed rows.  delta, bias, table, vec nullable; a
// bias comes with a delta only.
extern "C" int pih_rmsnorm_stream(int delta_dtype, int out_dtype, void* h, const void* delta, float delta_scale,
                                  const void* bias, const void* table, const void* ids, int vocab, float table_scale,
                                  const void* vec, const void* weight, int weight_len, void* out, const void* rows, int n_out,
                                  int width, float eps, void* stream) {
  if (n_out <= 0) return 0;
  if (weight_len != 1 && weight_len != width) return PIH_ERR_BAD_ARGUMENT;
  if ((bias != nullptr && delta == nullptr) || (table != nullptr && (ids == nullptr || vocab < 1))) return PIH_ERR_BAD_ARGUMENT;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool four = width % 4 == 0 && aligned(h) && aligned(delta) && aligned(bias) && aligned(table) && aligned(vec) &&
                    aligned(weight) && aligned(out);
  const int threads = width <= 512 ? 128 : (width <= 4096 ? 256 : 512);
#define PIH_NORM_V(TD, TO, V)                                                                                         \
  do {                                                                                                                \
    StreamAdd<TD> add;                                                                                                \
    add.delta = static_cast<const TD*>(delta);                                                                        \
    add.scale = delta_scale;                                                                                          \
    add.bias = static_cast<const float*>(bias);                                                                       \
    add.table = static_cast<const TD*>(table);                                                                        \
    add.ids = static_cast<const int*>(ids);                                                                           \
    add.vocab = vocab;                                                                                                \
    add.table_scale = table_scale;                                                                                    \
    add.vec = static_cast<const float*>(vec);                                                                         \
    launch_kernel(rmsnorm_stream_kernel<TD, TO, V>, dim3(n_out), dim3(threads), 0, s, static_cast<float*>(h), add,     \
                  static_cast<const float*>(weight), weight_len, static_cast<TO*>(out), static_cast<const int*>(rows), \
                  width, eps);                                                                                        \
  } while (0)
#define PIH_NORM(TD, TO)                                                                                              \
  do { if (four) PIH_NORM_V(TD, TO, 4); else PIH_NORM_V(TD, TO, 1); } while (0)
  if (delta_dtype == PIH_F32 && out_dtype == PIH_F32) PIH_NORM(float, float);
  else if (delta_dtype == PIH_BF16 && out_dtype == PIH_BF16) PIH_NORM(bf16, bf16);
  else if (delta_dtype == PIH_F32 && out_dtype == PIH_BF16) PIH_NORM(float, bf16);
  else if (delta_dtype == PIH_BF16 && out_dtype == PIH_F32) PIH_NORM(bf16, float);
  else return PIH_ERR_BAD_ARGUMENT;
#undef PIH_NORM
#undef PIH_NORM_V
  PIH_LAUNCH_CHECK();
  return 0;
}

// h [.., width] fp32: h += rms(y + bias) * add_weight (add_eps), or with y2 the pair in y's place (see NormedOutput), then out =
// rms(h) * weight (eps).  y, y2 [.., width] of delta_dtype; bias, bias2 nullable; the weights fp32 [width].
extern "C" int pih_stream_norm_norm(int delta_dtype, int out_dtype, void* h, const void* y, const void* bias, const void* y2,
                                    const void* bias2, const void* weight_left, const void* weight_right, float pair_eps,
                                    const void* add_weight, float add_eps, const void* weight, float eps, void* out,
                                    const void* rows, int n_out, int width, void* stream) {
  if (n_out <= 0) return 0;
  if (y == nullptr || add_weight == nullptr || weight == nullptr ||
      (y2 != nullptr && (weight_left == nullptr || weight_right == nullptr)))
    return PIH_ERR_BAD_ARGUMENT;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool four = width % 4 == 0 && aligned(h) && aligned(y) && aligned(bias) && aligned(y2) && aligned(bias2) &&
                    aligned(weight_left) && aligned(weight_right) && aligned(add_weight) && aligned(weight) && aligned(out);
  const int pieces = four ? width / 4 : width;
  int threads = pieces <= 512 ? (pieces + 31) / 32 * 32 : 512;
  if (pieces > threads * kNormHeld) threads = 1024;
  if (pieces > threads * kNormHeld) return PIH_ERR_UNSUPPORTED;
#define PIH_NN_V(TD, TO, V)                                                                                           \
  do {                                                                                                                \
    NormedOutput<TD> add;                                                                                             \
    add.y = static_cast<const TD*>(y);                                                                                \
    add.bias = static_cast<const float*>(bias);                                                                       \
    add.y2 = static_cast<const TD*>(y2);                                                                              \
    add.bias2 = static_cast<const float*>(bias2);                                                                     \
    add.weight_left = static_cast<const float*>(weight_left);                                                         \
    add.weight_right = static_cast<const float*>(weight_right);                                                       \
    add.pair_eps = pair_eps;                                                                                          \
    add.weight = static_cast<const float*>(add_weight);                                                               \
    add.eps = add_eps;                                                                                                \
    launch_kernel(stream_norm_norm_kernel<TD, TO, V>, dim3(n_out), dim3(threads), 0, s, static_cast<float*>(h), add,   \
                  static_cast<const float*>(weight), static_cast<TO*>(out), static_cast<const int*>(rows), width, eps); \
  } while (0)
#define PIH_NN(TD, TO)                                                                                                \
  do { if (four) PIH_NN_V(TD, TO, 4); else PIH_NN_V(TD, TO, 1); } while (0)
  if (delta_dtype == PIH_F32 && out_dtype == PIH_F32) PIH_NN(float, float);
  else if (delta_dtype == PIH_BF16 && out_dtype == PIH_BF16) PIH_NN(bf16, bf16);
  else return PIH_ERR_BAD_ARGUMENT;
#undef PIH_NN
#undef PIH_NN_V
  PIH_LAUNCH_CHECK();
  return 0;
}

extern "C" int pih_causal_conv(int dtype, const void* x, long long ldx, const void* w, const void* in_bias,
                               const void* out_bias, void* out, long long ldo, int channels, int taps, int activation,
                               void* state, long long state_stride, long long state_offset, const void* cu_q,
                               const void* state_slots, int rows, int requests, void* stream) {
  if (requests <= 0 || channels <= 0 || rows <= 0) return 0;
  if (taps < 1 || taps > kMaxTaps) return PIH_ERR_UNSUPPORTED;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  dim3 grid(requests, (channels + 31) / 32, (rows + kConvRows - 1) / kConvRows), block(32, 8);
  dim3 grid_h(requests, (channels + 127) / 128);
  if (grid.y > 65535 || grid.z > 65535) return PIH_ERR_UNSUPPORTED;
#define PIH_CONV_TAPS(T, N)                                                                                            \
  launch_kernel(causal_conv_kernel<T, N>, grid, block, 0, s, static_cast<const T*>(x), ldx, static_cast<const T*>(w),  \
                static_cast<const float*>(in_bias), static_cast<const float*>(out_bias), static_cast<T*>(out), ldo,    \
                channels, taps, activation, static_cast<const float*>(state), state_stride, state_offset,              \
                static_cast<const int*>(cu_q), static_cast<const int*>(state_slots))
#define PIH_CONV(T)                                                                                                    \
  do {                                                                                                                 \
    if (taps <= 2) PIH_CONV_TAPS(T, 2);                                                                                \
    else if (taps == 3) PIH_CONV_TAPS(T, 3);                                                                           \
    else if (taps == 4) PIH_CONV_TAPS(T, 4);                                                                           \
    else PIH_CONV_TAPS(T, kMaxTaps);                                                                                   \
    PIH_LAUNCH_CHECK();                                                                                                \
    if (taps > 1)                                                                                                      \
      launch_kernel(causal_conv_history_kernel<T>, grid_h, dim3(128), 0, s, static_cast<const T*>(x), ldx,             \
                    static_cast<const float*>(in_bias), channels, taps, static_cast<float*>(state), state_stride,      \
                    state_offset, static_cast<const int*>(cu_q), static_cast<const int*>(state_slots));                \
  } while (0)
  if (dtype == PIH_F32) PIH_CONV(float);
  else if (dtype == PIH_BF16) PIH_CONV(bf16);
  else return PIH_ERR_BAD_ARGUMENT;
#undef PIH_CONV
#undef PIH_CONV_TAPS
  PIH_LAUNCH_CHECK();
  return 0;
}

// The gated delta rule over a step's rows.  qkv [rows, ld]: q heads, k heads, v heads (after convolution and SiLU);
// b [rows, ldb]: write-strength logits a head; a [rows, lda] (a_dtype): decay logits, one a head or (channels) one a head and
// key channel, with decay_bias of the same layout; decay_log [heads].  scratch: fp32, rows * (2 * kv_heads * dim + kv_heads +
// heads + heads * (channels ? dim : 1)), 16-byte aligned.  out: fp32 [rows, heads, vdim].  The state S [heads, dim, vdim] lies at the
// start of a request's slot.
template <typename T, int D, bool CH>
static void launch_delta_reg(cudaStream_t s, const float* qn, const float* kn, const float* qk_dot, const T* v, long long ld, const float* decay,
                             const float* beta, float* out, float* state, long long state_stride, const int* cu_q,
                             const int* state_slots, int requests, int heads, int kv_heads, int vdim) {
  typedef DeltaShape<D, CH> Shape;
  const size_t needed = 2 * static_cast<size_t>(Shape::kChunk) * Shape::words(sizeof(T)) * sizeof(float);
  const dim3 grid(requests, heads, (vdim + Shape::kCols - 1) / Shape::kCols);
  // The chain from token to token is what a prompt costs: with no more blocks than SMs, every block asks for more than half
  // of an SM's shared memory and so gets an SM alone.
  const bool alone = static_cast<long long>(grid.x) * grid.y * grid.z <= 148;
  const size_t staged = alone && needed < 116 * 1024 ? 116 * 1024 : needed;
  static size_t raised = 48 * 1024;                            // (per instance)
  if (staged > raised) {
    cudaFuncSetAttribute(delta_recurrence_reg_kernel<T, D, CH>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                         static_cast<int>(staged));
    raised = staged;
  }
  launch_kernel(delta_recurrence_reg_kernel<T, D, CH>, grid,
                dim3(Shape::kThreads), staged, s, qn, kn, qk_dot, v, ld, decay, beta, out, state, state_stride, cu_q, state_slots, heads, kv_heads, vdim);
}

template <typename T, bool CH>
static int launch_delta(cudaStream_t s, const float* qn, const float* kn, const float* qk_dot, const T* v, long long ld, const float* decay,
                        const float* beta, float* out, float* state, long long state_stride, const int* cu_q,
                        const int* state_slots, int requests, int heads, int kv_heads, int dim, int vdim) {
  const bool words = sizeof(T) == 4 || (ld % 2 == 0 && vdim % 2 == 0 && (reinterpret_cast<uintptr_t>(v) & 3) == 0);
  switch (words ? dim : 0) {                                   // (values are copied in 32-bit words)
#define PIH_DELTA_REG(D)                                                                                               \
  case D:                                                                                                              \
    launch_delta_reg<T, D, CH>(s, qn, kn, qk_dot, v, ld, decay, beta, out, state, state_stride, cu_q, state_slots, requests,   \
                               heads, kv_heads, vdim);                                                                 \
    break
    PIH_DELTA_REG(16);
    PIH_DELTA_REG(32);
    PIH_DELTA_REG(64);
    PIH_DELTA_REG(128);
    PIH_DELTA_REG(256);
#undef PIH_DELTA_REG
    default: {
      const int cols = vdim >= 64 ? 64 : 32;
      if (dim > 8 * cols) return PIH_ERR_UNSUPPORTED;
      const size_t smem = (static_cast<size_t>(dim) * cols + 2 * (CH ? 3 : 2) * static_cast<size_t>(dim)) * sizeof(float);
      if (smem > 200 * 1024) return PIH_ERR_UNSUPPORTED;
      if (smem > 48 * 1024)
        cudaFuncSetAttribute(delta_recurrence_kernel<T, CH>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                             static_cast<int>(smem));
      const dim3 grid(requests, heads, (vdim + cols - 1) / cols);
      launch_kernel(delta_recurrence_kernel<T, CH>, grid, dim3(cols), smem, s, qn, kn, v, ld, decay, beta, out, state,
                    state_stride, cu_q, state_slots, heads, kv_heads, dim, vdim);
    }
  }
  PIH_LAUNCH_CHECK();
  return 0;
}

extern "C" int pih_gated_delta_rule(int dtype, const void* qkv, long long ld, const void* b, long long ldb, int a_dtype,
                                    const void* a, long long lda, int channels, const void* decay_log,
                                    const void* decay_bias, void* scratch, void* out, void* state, long long state_stride,
                                    const void* cu_q, const void* state_slots, int rows, int requests, int heads,
                                    int kv_heads, int dim, int vdim, float unit_eps, float q_scale, void* stream) {
  if (rows <= 0 || requests <= 0) return 0;
  if (heads % kv_heads) return PIH_ERR_BAD_ARGUMENT;
  if (heads > 65535 || (vdim + 15) / 16 > 65535) return PIH_ERR_UNSUPPORTED;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const long long qk_size = static_cast<long long>(kv_heads) * dim;
  float* qn = static_cast<float*>(scratch);
  float* kn = qn + rows * qk_size;
  float* decay = kn + rows * qk_size;
  float* beta = decay + static_cast<long long>(rows) * heads * (channels ? dim : 1);
  float* qk_dot = beta + static_cast<long long>(rows) * heads;
  const int numbers = heads * (channels ? dim : 1);
  const int parts = numbers > kDecaySlice ? 1 + (numbers + kDecaySlice - 1) / kDecaySlice : 1;
#define PIH_DELTA(T, TA)                                                                                               \
  do {                                                                                                                 \
    launch_kernel(delta_prepare_kernel<T, TA>, dim3(rows, parts), dim3(128), 0, s, static_cast<const T*>(qkv), ld,            \
                  static_cast<const T*>(b), ldb, static_cast<const TA*>(a), lda, channels,                             \
                  static_cast<const float*>(decay_log), static_cast<const float*>(decay_bias), qn, kn, qk_dot, decay,  \
                  beta, heads, kv_heads, dim, unit_eps, q_scale);                                                            \
    PIH_LAUNCH_CHECK();                                                                                                \
    const T* v = static_cast<const T*>(qkv) + 2 * qk_size;                                                             \
    float* o = static_cast<float*>(out);                                                                               \
    float* st = static_cast<float*>(state);                                                                            \
    const int* cu = static_cast<const int*>(cu_q);                                                                     \
    const int* slots = static_cast<const int*>(state_slots);                                                           \
    return channels ? launch_delta<T, true>(s, qn, kn, qk_dot, v, ld, decay, beta, o, st, state_stride, cu, slots, requests,   \
                                            heads, kv_heads, dim, vdim)                                                \
                    : launch_delta<T, false>(s, qn, kn, qk_dot, v, ld, decay, beta, o, st, state_stride, cu, slots, requests,  \
                                             heads, kv_heads, dim, vdim);                                              \
  } while (0)
  if (dtype == PIH_F32 && a_dtype == PIH_F32) PIH_DELTA(float, float);
  if (dtype == PIH_BF16 && a_dtype == PIH_BF16) PIH_DELTA(bf16, bf16);
  if (dtype == PIH_BF16 && a_dtype == PIH_F32) PIH_DELTA(bf16, float);
  return PIH_ERR_BAD_ARGUMENT;
#undef PIH_DELTA
}

// o fp32 [rows, heads, vdim]; gate [rows, ldg] (gate_dtype), out [rows, ldo] (dtype); activation 0: SiLU, 1: sigmoid; divisor
// fp32 [rows, heads] or null; head_weight 0: weight [vdim], else weight [heads, head_weight].
extern "C" int pih_gated_rmsnorm(int dtype, int gate_dtype, const void* o, const void* gate, long long ldg,
                                 const void* weight, void* out, long long ldo, int rows, int heads, int vdim, float eps,
                                 int activation, float out_scale, const void* divisor, int head_weight, void* stream) {
  if (rows <= 0) return 0;
  if (activation < 0 || activation > 1 || (head_weight != 0 && head_weight < vdim)) return PIH_ERR_BAD_ARGUMENT;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const long long items = static_cast<long long>(rows) * heads;
  dim3 grid(static_cast<unsigned>((items + 3) / 4));
#define PIH_GN(TG, T)                                                                                                  \
  launch_kernel(gated_rmsnorm_kernel<TG, T>, grid, dim3(128), 0, s, static_cast<const float*>(o), static_cast<const TG*>(gate), \
                ldg, static_cast<const float*>(weight), static_cast<T*>(out), ldo, items, heads, vdim, eps, activation, out_scale, \
                static_cast<const float*>(divisor), head_weight)
  if (dtype == PIH_F32 && gate_dtype == PIH_F32) PIH_GN(float, float);
  else if (dtype == PIH_BF16 && gate_dtype == PIH_BF16) PIH_GN(bf16, bf16);
  else if (dtype == PIH_BF16 && gate_dtype == PIH_F32) PIH_GN(float, bf16);
  else return PIH_ERR_BAD_ARGUMENT;
#undef PIH_GN
  PIH_LAUNCH_CHECK();
  return 0;
}

// y fp32 [rows, width] contiguous; gate [rows, ldg], out [rows, ldo] of ``dtype``; ``parts`` equal stretches of the row are
// normed each by itself after the gate
extern "C" int pih_gated_part_rmsnorm(int dtype, const void* y, const void* gate, long long ldg, const void* weight, void* out,
                                      long long ldo, int rows, int width, int parts, float eps, float out_scale,
                                      void* stream) {
  if (rows <= 0) return 0;
  if (parts < 1 || width < 1 || width % parts) return PIH_ERR_BAD_ARGUMENT;
  if (parts > 65535) return PIH_ERR_UNSUPPORTED;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int part = width / parts;
  const int threads = part >= 2048 ? 512 : (part >= 1024 ? 256 : (part >= 256 ? 128 : (part >= 64 ? 64 : 32)));
#define PIH_GPN(T)                                                                                                     \
  launch_kernel(gated_part_rmsnorm_kernel<T>, dim3(rows, parts), dim3(threads), 0, s, static_cast<const float*>(y),      \
                static_cast<const T*>(gate), ldg, static_cast<const float*>(weight), static_cast<T*>(out), ldo, width,  \
                part, eps, out_scale)
  if (dtype == PIH_F32) PIH_GPN(float);
  else if (dtype == PIH_BF16) PIH_GPN(bf16);
  else return PIH_ERR_BAD_ARGUMENT;
#undef PIH_GPN
  PIH_LAUNCH_CHECK();
  return 0;
}

// coef: scratch, 4 * rows * width floats (16-byte aligned)
extern "C" int pih_rglru_scan(int dtype, const void* u, long long ldu, const void* gates, const void* y_pre, long long ldy,
                              const void* y_bias, const void* r_bias, const void* i_bias, const void* lam,
                              float decay_scale, void* coef, void* out, long long ldo, void* state, long long state_stride,
                              const void* cu_q, const void* state_slots, int rows, int requests, int width, int blocks,
                              void* stream) {
  if (requests <= 0 || width <= 0 || rows <= 0) return 0;
  if (blocks < 1 || width % blocks) return PIH_ERR_BAD_ARGUMENT;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  dim3 grid(requests, (width + 127) / 128);
  const long long items = static_cast<long long>(rows) * width;
  if (grid.y > 65535 || (items + 255) / 256 > 2147483647LL) return PIH_ERR_UNSUPPORTED;
#define PIH_SCAN(T)                                                                                                    \
  do {                                                                                                                 \
    launch_kernel(rglru_gates_kernel<T>, dim3(static_cast<unsigned>((items + 255) / 256)), dim3(256), 0, s,            \
                  static_cast<const T*>(u), ldu, static_cast<const float*>(gates), static_cast<const T*>(y_pre), ldy,  \
                  static_cast<const float*>(y_bias), static_cast<const float*>(r_bias),                                \
                  static_cast<const float*>(i_bias), static_cast<const float*>(lam), decay_scale,                      \
                  static_cast<float4*>(coef), rows, width, blocks);                                                    \
    PIH_LAUNCH_CHECK();                                                                                                \
    launch_kernel(rglru_chain_kernel<T>, grid, dim3(128), 0, s, static_cast<const float4*>(coef), static_cast<T*>(out), \
                  ldo, static_cast<float*>(state), state_stride, static_cast<const int*>(cu_q),                        \
                  static_cast<const int*>(state_slots), width);                                                        \
  } while (0)
  if (dtype == PIH_F32) PIH_SCAN(float);
  else if (dtype == PIH_BF16) PIH_SCAN(bf16);
  else return PIH_ERR_BAD_ARGUMENT;
#undef PIH_SCAN
  PIH_LAUNCH_CHECK();
  return 0;
}
