// Linear attention with a decaying matrix state per (request, head), for three ways of making the decay and the write
// strength of a token.  S [dim, vdim] starts at zero; token by token
//
//   S <- diag(a) S + w k v^T,      o = S^T q * q_scale (+ skip[head] v)
//
//   kChannel   gated linear attention: a = sigmoid(z + bias) ^ (1 / temperature), one number a head and key channel; w = 1
//   kStep      state-space duality (Mamba-2): dt = softplus(z + bias); a = exp(A[head] dt), one number a head; w = dt; k and q
//              are B and C, whose groups serve equal runs of heads
//   kExp       matrix memory with exponential gates (mLSTM): i = cap tanh((zi + bi) / cap), f = logsigmoid(cap tanh((zf + bf) /
//              cap)), m' = max(f + m, i), a = exp(f + m - m'), w = exp(i - m'); beside S a key sum n <- a n + w k and the
//              divisor max(|n . q| q_scale, exp(-m')) + floor
//
// A step's rows are packed: request r owns rows cu_q[r] .. cu_q[r+1]-1, its state lies at state + slot * stride: S [heads,
// dim, vdim]; kExp then n [heads, dim] and m [heads, copies]: every block of value columns of memory_recurrence keeps a
// running maximum of its own (all equal), so that no block reads what another one writes.
//
//   memory_recurrence   token by token, S in registers, gates formed on the way; any size up to 1024 key channels.  A warp
//                       holds 32 value columns (a lane a column) of some of the rows of S; nothing of a token's read-out enters the
//                       next token's state, so the warps' shares of the read-outs of a chunk of tokens meet once a chunk.
//                       The order of the additions is fixed by the sizes: neither a cut nor the batch changes a bit.
//
// bf16, requests of more than small_rows rows, on tensor cores (mma.sync m16n8k16) in chunks of 64 rows of a request, all
// chunks side by side.  With L the sum of the log decays from the chunk's start, up to and with a token:
//
//   memory_gates, _channels   L and w of every token (kExp: the running maximum goes from chunk to chunk as max(m + sum f, .),
//                             inside a chunk as a scan)
//   memory_chunk_state        U = sum_j exp(L_end - L_j) w_j k_j v_j^T, what a chunk adds to the state
//   memory_state_pass         the chunks in order: the state in front of each takes U's place; S <- exp(L_end) S + U
//   memory_chunk_out          o_i = sum_{j <= i} (q_i . k_j) exp(L_i - L_j) w_j v_j + exp(L_i) S^T q_i
//
// Every exponent is at most zero but one: with a decay a channel the factor exp(L_i - L_j) goes into q and k, taken from the
// start of the 16 rows of i, so that rows j of the same 16 have exp(-L) of up to 16 rows; where that could leave the range of
// the numbers, these 16 x 16 scores are formed one by one.  q, k and v enter the products as they are; what is 32-bit (scaled q
// and k, scores, states) as the pair of its bf16 rounding and the rounding of the remainder; sums are 32-bit.
//
// States, decays, gates and sums are 32-bit whatever the storage type T.  The decay is applied as S + (a - 1) S with a - 1
// formed by expm1, so that a state that remembers long keeps the distance of its decay from one.
#include "common.cuh"
#include "mma.cuh"

namespace pih {

enum MemoryGate : int { kChannel = 0, kStep = 1, kExp = 2 };

struct MemoryArgs {
  const void* q;                            // [rows, ldq]: group g's numbers at column g * dim
  long long ldq;
  const void* k;
  long long ldk;
  const void* v;                            // [rows, ldv]: head h's numbers at column h * vdim
  long long ldv;
  const void* gate0;                        // kChannel: z, fp32 [rows, ld0] at h * dim; kStep: z of T at h; kExp: zi of T at h
  long long ld0;
  const void* gate1;                        // kExp: zf of T at h
  long long ld1;
  const float* bias0;                       // of gate0: [heads * dim] or [heads]
  const float* bias1;
  const float* A;                           // kStep: [heads], negative
  float constant;                           // kChannel: 1 / temperature; kExp: cap
  float floor;                              // kExp
  float q_scale;
  const float* skip;                        // [heads] or null
  float* out;                               // [rows, heads, vdim]
  float* divisor;                           // kExp: [rows, heads]
  float* state;
  long long state_stride;
  const int* cu_q;
  const int* state_slots;
  int heads, per_group, dim, vdim, copies;
  int small_rows;                           // requests of more rows than this go by chunks
  // scratch of the kernels that go by chunks
  float* log_decay;                         // L: [rows, heads] or (kChannel) [rows, heads * dim]
  float* strength;                          // w: [rows, heads]
  float* lowest;                            // kExp: exp(-m), [rows, heads]
  float* chunk_states;                      // [chunks, heads, dim, ld_state]: value columns, kExp: then the key sum's
  int ld_state;
  int requests;
};

__device__ __forceinline__ float log_sigmoid_f(float z) { return -softplus_f(-z); }
__device__ __forceinline__ float capped_gate(float z, float cap) { return cap * tanhf(z / cap); }

template <int D>
struct MemoryShape {
  static constexpr int kParts = D <= 16 ? 4 : (D <= 128 ? 8 : 16);     // warps: each holds D / kParts rows of S
  static constexpr int kRows = D / kParts;
  static constexpr int kThreads = 32 * kParts;
  static constexpr int kTokens = D <= 256 ? 16 : 8;                    // of a chunk
  static constexpr size_t bytes(int gate) {
    return sizeof(float) * kTokens * ((gate == kChannel ? 3 : 2) * static_cast<size_t>(D) + 32 + 32 * kParts + 4);
  }
};

// Block (request, head, 32 value columns; kExp: one more for the key sum).
template <typename T, int D, int GATE>
__global__ void __launch_bounds__(MemoryShape<D>::kThreads)
memory_recurrence_kernel(const MemoryArgs p) {
  typedef MemoryShape<D> Shape;
  constexpr int P = Shape::kParts, R = Shape::kRows, TH = Shape::kThreads, C = Shape::kTokens;
  extern __shared__ __align__(16) float memory_smem[];
  float* ks = memory_smem;                                             // [C][D]
  float* qs = ks + C * D;                                              // [C][D]
  float* as = qs + C * D;                                              // kChannel: a - 1, [C][D]
  float* vs = as + (GATE == kChannel ? C * D : 0);                     // [C][32]
  float* shares = vs + C * 32;                                         // [C][P][32]
  float* scalars = shares + C * P * 32;                                // [C][4]: a - 1, w, exp(-m), unused
  wait_for_prior_kernels();
  launch_dependents();
  const int r = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, part = tid >> 5;
  const int lo = p.cu_q[r], hi = p.cu_q[r + 1], slot = p.state_slots[r];
  if (hi <= lo || slot < 0 || hi - lo > p.small_rows) return;
  const bool sums = GATE == kExp && blockIdx.z + 1 == gridDim.z;       // the block of the key sum: its one column is all ones
  const int col = static_cast<int>(blockIdx.z) * 32 + lane;
  const bool live = sums ? lane == 0 : col < p.vdim;
  float* base = p.state + slot * p.state_stride;
  const long long matrix = static_cast<long long>(p.heads) * p.dim * p.vdim;
  float* Sg = sums ? base + matrix + static_cast<long long>(h) * p.dim : base + static_cast<long long>(h) * p.dim * p.vdim + col;
  const long long row_step = sums ? 1 : p.vdim;
  float* mg = base + matrix + static_cast<long long>(p.heads) * p.dim + static_cast<long long>(h) * p.copies + blockIdx.z;
  float2 S[R / 2];
#pragma unroll
  for (int i = 0; i < R / 2; ++i) {
    const int row = part * R + 2 * i;
    S[i].x = live && row < p.dim ? Sg[row * row_step] : 0.0f;
    S[i].y = live && row + 1 < p.dim ? Sg[(row + 1) * row_step] : 0.0f;
  }
  float top = GATE == kExp && part == 0 ? mg[0] : 0.0f;                // (warp 0 makes the gates)
  const int g = h / p.per_group;
  const T* q = static_cast<const T*>(p.q) + static_cast<long long>(g) * p.dim;
  const T* k = static_cast<const T*>(p.k) + static_cast<long long>(g) * p.dim;
  const T* v = static_cast<const T*>(p.v) + static_cast<long long>(h) * p.vdim;
  for (int t0 = lo; t0 < hi; t0 += C) {
    const int n = min(C, hi - t0);
    for (int e = tid; e < n * D; e += TH) {
      const int tok = e / D, c = e % D;
      const long long t = t0 + tok;
      const bool there = c < p.dim;
      ks[e] = there ? to_float<T>(k[t * p.ldk + c]) : 0.0f;
      qs[e] = there ? to_float<T>(q[t * p.ldq + c]) : 0.0f;
      if (GATE == kChannel) {
        const int at = h * p.dim + c;
        as[e] = there ? expm1f(log_sigmoid_f(static_cast<const float*>(p.gate0)[t * p.ld0 + at] + p.bias0[at]) * p.constant) : 0.0f;
      }
    }
    for (int e = tid; e < n * 32; e += TH) {
      const int tok = e >> 5;
      vs[e] = sums ? 1.0f : (live ? to_float<T>(v[(t0 + tok) * p.ldv + col]) : 0.0f);       // (e & 31 == lane)
    }
    if (GATE != kChannel && part == 0) {
      const bool mine = lane < n;
      const long long t = t0 + lane;
      if (GATE == kStep) {
        const float dt = mine ? softplus_f(to_float<T>(static_cast<const T*>(p.gate0)[t * p.ld0 + h]) + p.bias0[h]) : 0.0f;
        if (mine) {
          scalars[4 * lane] = expm1f(p.A[h] * dt);
          scalars[4 * lane + 1] = dt;
        }
      } else {
        float li = 0.0f, lf = 0.0f, before = 0.0f, after = 0.0f;
        if (mine) {
          li = capped_gate(to_float<T>(static_cast<const T*>(p.gate0)[t * p.ld0 + h]) + p.bias0[h], p.constant);
          lf = log_sigmoid_f(capped_gate(to_float<T>(static_cast<const T*>(p.gate1)[t * p.ld1 + h]) + p.bias1[h], p.constant));
        }
        for (int j = 0; j < n; ++j) {                                  // the running maximum, token by token
          const float fj = __shfl_sync(0xffffffffu, lf, j), ij = __shfl_sync(0xffffffffu, li, j);
          const float next = fmaxf(fj + top, ij);
          if (lane == j) { before = fj + top; after = next; }
          top = next;
        }
        if (mine) {
          scalars[4 * lane] = expm1f(before - after);
          scalars[4 * lane + 1] = expf(li - after);
          scalars[4 * lane + 2] = expf(-after);
        }
      }
    }
    __syncthreads();
#pragma unroll 2
    for (int tok = 0; tok < n; ++tok) {
      const float4* k4 = reinterpret_cast<const float4*>(ks + tok * D + part * R);
      const float4* q4 = reinterpret_cast<const float4*>(qs + tok * D + part * R);
      const float4* a4 = reinterpret_cast<const float4*>(as + tok * D + part * R);
      float vw = vs[tok * 32 + lane];
      float2 a = make_float2(0.0f, 0.0f);
      if (GATE != kChannel) {
        a.x = a.y = scalars[4 * tok];
        vw *= scalars[4 * tok + 1];
      }
      const float2 vv = make_float2(vw, vw);
      float2 o0 = make_float2(0.0f, 0.0f), o1 = o0;
#pragma unroll
      for (int i = 0; i < R / 4; ++i) {
        const float4 kk = k4[i], qq = q4[i];
        float2 a0 = a, a1 = a;
        if (GATE == kChannel) {
          const float4 aa = a4[i];
          a0 = make_float2(aa.x, aa.y);
          a1 = make_float2(aa.z, aa.w);
        }
        S[2 * i] = fma2(make_float2(kk.x, kk.y), vv, fma2(a0, S[2 * i], S[2 * i]));
        S[2 * i + 1] = fma2(make_float2(kk.z, kk.w), vv, fma2(a1, S[2 * i + 1], S[2 * i + 1]));
        o0 = fma2(S[2 * i], make_float2(qq.x, qq.y), o0);
        o1 = fma2(S[2 * i + 1], make_float2(qq.z, qq.w), o1);
      }
      shares[(tok * P + part) * 32 + lane] = (o0.x + o1.x) + (o0.y + o1.y);
    }
    __syncthreads();
    for (int e = tid; e < n * 32; e += TH) {                           // (e & 31 == lane)
      const int tok = e >> 5;
      float o = 0.0f;
#pragma unroll
      for (int i = 0; i < P; ++i) o += shares[(tok * P + i) * 32 + lane];
      o *= p.q_scale;
      const long long item = static_cast<long long>(t0 + tok) * p.heads + h;
      if (sums) {
        if (lane == 0) p.divisor[item] = fmaxf(fabsf(o), scalars[4 * tok + 2]) + p.floor;
      } else if (live) {
        if (p.skip != nullptr) o = fmaf(p.skip[h], vs[e], o);
        p.out[item * p.vdim + col] = o;
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < R / 2; ++i) {
    const int row = part * R + 2 * i;
    if (live && row < p.dim) Sg[row * row_step] = S[i].x;
    if (live && row + 1 < p.dim) Sg[(row + 1) * row_step] = S[i].y;
  }
  if (GATE == kExp && tid == 0) mg[0] = top;
}

// ---- by chunks of 64 rows ---------------------------------------------------------------------------------------------
constexpr int kChunkRows = 64;

struct ChunkPlace { int request, first, rows, index; };      // rows first .. first + rows - 1 of the step; index: of the step

// The x-th chunk of the step's requests that have more than small_rows rows (request -1: there is none).
__device__ __forceinline__ ChunkPlace find_chunk(const MemoryArgs& p, int x) {
  ChunkPlace c = {-1, 0, 0, x};
  int t = x;
  for (int r = 0; r < p.requests; ++r) {
    const int lo = p.cu_q[r], n = p.cu_q[r + 1] - lo;
    if (n <= p.small_rows || p.state_slots[r] < 0) continue;
    const int chunks = (n + kChunkRows - 1) / kChunkRows;
    if (t < chunks) {
      c.request = r;
      c.first = lo + t * kChunkRows;
      c.rows = min(kChunkRows, n - t * kChunkRows);
      break;
    }
    t -= chunks;
  }
  return c;
}
__device__ __forceinline__ ChunkPlace find_chunk_shared(const MemoryArgs& p, int x, ChunkPlace* place) {
  if (threadIdx.x == 0) *place = find_chunk(p, x);
  __syncthreads();
  return *place;
}

__device__ __forceinline__ float warp_scan_sum(float v, int lane) {
#pragma unroll
  for (int d = 1; d < 32; d <<= 1) {
    const float o = __shfl_up_sync(0xffffffffu, v, d);
    if (lane >= d) v += o;
  }
  return v;
}
__device__ __forceinline__ float warp_scan_max(float v, int lane) {
#pragma unroll
  for (int d = 1; d < 32; d <<= 1) {
    const float o = __shfl_up_sync(0xffffffffu, v, d);
    if (lane >= d) v = fmaxf(v, o);
  }
  return v;
}

// One number a head and token.  Block (request, head), a warp a chunk (32 chunks at a time), a lane two neighbouring rows.
constexpr int kGateWarps = 32;
template <typename T, int GATE>
__global__ void __launch_bounds__(32 * kGateWarps)
memory_gates_kernel(const MemoryArgs p) {
  __shared__ float2 ends[kGateWarps];                        // kExp: a chunk's sum of log decays, its largest i_s - F_s
  __shared__ float tops[kGateWarps + 1];                     // the running maximum in front of a chunk
  wait_for_prior_kernels();
  launch_dependents();
  const int r = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int lo = p.cu_q[r], n = p.cu_q[r + 1] - lo, slot = p.state_slots[r];
  if (n <= p.small_rows || slot < 0) return;
  float* mg = nullptr;
  if (GATE == kExp) {
    mg = p.state + slot * p.state_stride + static_cast<long long>(p.heads) * p.dim * (p.vdim + 1) +
         static_cast<long long>(h) * p.copies;
    if (threadIdx.x == 0) tops[kGateWarps] = mg[0];
    __syncthreads();
  }
  for (int base = 0; base < n; base += kGateWarps * kChunkRows) {
    const int t = base + warp * kChunkRows + 2 * lane;       // and t + 1
    float f[2], w[2], F[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      f[u] = 0.0f;
      w[u] = GATE == kExp ? -INFINITY : 0.0f;
      if (t + u < n) {
        const long long row = lo + t + u;
        const float z = to_float<T>(static_cast<const T*>(p.gate0)[row * p.ld0 + h]) + p.bias0[h];
        if (GATE == kStep) {
          w[u] = softplus_f(z);
          f[u] = p.A[h] * w[u];
        } else {
          w[u] = capped_gate(z, p.constant);
          f[u] = log_sigmoid_f(capped_gate(to_float<T>(static_cast<const T*>(p.gate1)[row * p.ld1 + h]) + p.bias1[h], p.constant));
        }
      }
    }
    const float both = f[0] + f[1];
    const float upto = warp_scan_sum(both, lane);
    F[0] = upto - both + f[0];
    F[1] = upto;
    if (GATE == kStep) {
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        if (t + u >= n) continue;
        const long long item = static_cast<long long>(lo + t + u) * p.heads + h;
        p.log_decay[item] = F[u];
        p.strength[item] = w[u];
      }
    } else {
      const float a0 = w[0] - F[0], a1 = w[1] - F[1];
      const float M = warp_scan_max(fmaxf(a0, a1), lane);
      float before = __shfl_up_sync(0xffffffffu, M, 1);
      if (lane == 0) before = -INFINITY;
      const float top[2] = {fmaxf(before, a0), M};
      if (lane == 31) ends[warp] = make_float2(F[1], M);
      __syncthreads();
      if (threadIdx.x == 0) {
        float m = tops[kGateWarps];
        const int chunks = min(kGateWarps, (n - base + kChunkRows - 1) / kChunkRows);
        for (int c = 0; c < chunks; ++c) {
          tops[c] = m;
          m = ends[c].x + fmaxf(m, ends[c].y);
        }
        tops[kGateWarps] = m;
      }
      __syncthreads();
      const float m0 = t < n ? tops[warp] : 0.0f;
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        if (t + u >= n) continue;
        const long long item = static_cast<long long>(lo + t + u) * p.heads + h;
        const float rise = fmaxf(m0, top[u]);                // m - F
        p.log_decay[item] = fminf(m0 - rise, 0.0f);
        p.strength[item] = expf(fminf(w[u] - F[u] - rise, 0.0f));
        p.lowest[item] = expf(-(F[u] + rise));
      }
      __syncthreads();                                       // (the next 32 chunks write ends and tops again)
    }
  }
  if (GATE == kExp)
    for (int c = threadIdx.x; c < p.copies; c += blockDim.x) mg[c] = tops[kGateWarps];
}

// kChannel: a thread a (chunk, channel), the chunk's rows in order.
__global__ void __launch_bounds__(128)
memory_channels_kernel(const MemoryArgs p) {
  __shared__ ChunkPlace place;
  wait_for_prior_kernels();
  launch_dependents();
  const ChunkPlace c = find_chunk_shared(p, blockIdx.x, &place);
  if (c.request < 0) return;
  const int at = blockIdx.y * 128 + threadIdx.x, channels = p.heads * p.dim;
  if (at >= channels) return;
  const float* z = static_cast<const float*>(p.gate0) + static_cast<long long>(c.first) * p.ld0 + at;
  float* L = p.log_decay + static_cast<long long>(c.first) * channels + at;
  const float bias = p.bias0[at];
  float sum = 0.0f;
  constexpr int kAhead = 16;                                 // rows asked for together
  for (int t0 = 0; t0 < c.rows; t0 += kAhead) {
    float x[kAhead];
#pragma unroll
    for (int i = 0; i < kAhead; ++i) x[i] = t0 + i < c.rows ? z[(t0 + i) * p.ld0] : 0.0f;
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      if (t0 + i >= c.rows) continue;
      // log sigmoid by the special-function unit: its error is far below a bf16 rounding of z's inputs
      const float y = -(x[i] + bias);
      sum -= (fmaxf(y, 0.0f) + __logf(1.0f + __expf(-fabsf(y)))) * p.constant;
      L[static_cast<long long>(t0 + i) * channels] = sum;
    }
  }
}

__device__ __forceinline__ float2 unpack2(uint32_t w) { return make_float2(__uint_as_float(w << 16), __uint_as_float(w & 0xffff0000u)); }
constexpr float kLog2E = 1.4426950408889634f;
__device__ __forceinline__ float exp_fast(float x) { return mma::exp2_fast(x * kLog2E); }

constexpr int kTileDim = 64;                                 // key channels a tile
constexpr int kKeyLd = kTileDim + 8;                         // row strides that keep ldmatrix free of bank conflicts
constexpr int kDecayLd = kTileDim + 4;

// 64 rows by 64 columns of a bf16 matrix (row stride ld) into shared memory [64][kKeyLd], zeros beyond rows and cols.
__device__ __forceinline__ void load_rows(__nv_bfloat16* dst, const __nv_bfloat16* src, long long ld, int rows, int cols) {
  for (int e = threadIdx.x; e < kChunkRows * (kTileDim / 8); e += blockDim.x) {
    const int row = e / (kTileDim / 8), c = (e % (kTileDim / 8)) * 8;
    __nv_bfloat16* d = dst + row * kKeyLd + c;
    if (row < rows && c < cols) mma::copy_async_16(d, src + row * ld + c);
    else *reinterpret_cast<uint4*>(d) = make_uint4(0u, 0u, 0u, 0u);
  }
}
template <int VT>
__device__ __forceinline__ void load_values(__nv_bfloat16* dst, const __nv_bfloat16* src, long long ld, int rows, int cols) {
  for (int e = threadIdx.x; e < kChunkRows * (VT / 8); e += blockDim.x) {
    const int row = e / (VT / 8), c = (e % (VT / 8)) * 8;
    __nv_bfloat16* d = dst + row * (VT + 8) + c;
    if (row < rows && c < cols) mma::copy_async_16(d, src + row * ld + c);
    else *reinterpret_cast<uint4*>(d) = make_uint4(0u, 0u, 0u, 0u);
  }
}

// Block (chunk, head, tile of 64 key channels x tile of VT value columns), a warp 16 key channels.
template <int VT, int GATE>
__global__ void __launch_bounds__(128)
memory_chunk_state_kernel(const MemoryArgs p) {
  typedef __nv_bfloat16 bf16;
  extern __shared__ __align__(16) unsigned char chunk_state_smem[];
  bf16* kh = reinterpret_cast<bf16*>(chunk_state_smem);      // [64 rows][kKeyLd]: scaled keys, rounded; the remainders
  bf16* kl = kh + kChunkRows * kKeyLd;
  bf16* vs = kl + kChunkRows * kKeyLd;                       // [64 rows][VT + 8]
  __shared__ ChunkPlace place;
  wait_for_prior_kernels();
  launch_dependents();
  const ChunkPlace c = find_chunk_shared(p, blockIdx.x, &place);
  if (c.request < 0) return;
  const int h = blockIdx.y, vtiles = (p.vdim + VT - 1) / VT;
  const int d0 = static_cast<int>(blockIdx.z) / vtiles * kTileDim, v0 = static_cast<int>(blockIdx.z) % vtiles * VT;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int dims = min(kTileDim, p.dim - d0), cols = min(VT, p.vdim - v0), g = h / p.per_group;
  load_values<VT>(vs, static_cast<const bf16*>(p.v) + static_cast<long long>(c.first) * p.ldv + static_cast<long long>(h) * p.vdim + v0,
                  p.ldv, c.rows, cols);
  mma::copy_async_commit();
  const bf16* k = static_cast<const bf16*>(p.k) + static_cast<long long>(c.first) * p.ldk + static_cast<long long>(g) * p.dim + d0;
  const int channels = p.heads * p.dim;
  const long long last = c.first + c.rows - 1;
  const float end = GATE == kChannel ? 0.0f : p.log_decay[last * p.heads + h];
  constexpr int kPieces = kChunkRows * (kTileDim / 8) / 128;   // of 8 keys a thread; all asked for before the first is used
  uint4 raw[kPieces];
  float4 L4[GATE == kChannel ? kPieces : 1][2], E4[2];
  float f[kPieces];
  const int col = (threadIdx.x % (kTileDim / 8)) * 8, row0 = threadIdx.x / (kTileDim / 8);
  constexpr int kRowStep = 128 / (kTileDim / 8);
  const long long channel = static_cast<long long>(h) * p.dim + d0 + col;
  const bool inside = col < dims;
  if (GATE == kChannel && inside) {
    E4[0] = *reinterpret_cast<const float4*>(p.log_decay + last * channels + channel);
    E4[1] = *reinterpret_cast<const float4*>(p.log_decay + last * channels + channel + 4);
  }
#pragma unroll
  for (int i = 0; i < kPieces; ++i) {
    const int row = row0 + i * kRowStep;
    raw[i] = make_uint4(0u, 0u, 0u, 0u);
    f[i] = 0.0f;
    if (!inside || row >= c.rows) continue;
    raw[i] = *reinterpret_cast<const uint4*>(k + row * p.ldk + col);
    if (GATE == kChannel) {
      const float* L = p.log_decay + (static_cast<long long>(c.first) + row) * channels + channel;
      L4[i][0] = *reinterpret_cast<const float4*>(L);
      L4[i][1] = *reinterpret_cast<const float4*>(L + 4);
    } else {
      const long long item = (static_cast<long long>(c.first) + row) * p.heads + h;
      f[i] = exp_fast(end - p.log_decay[item]) * p.strength[item];
    }
  }
#pragma unroll
  for (int i = 0; i < kPieces; ++i) {
    const int row = row0 + i * kRowStep;
    uint4 hi = make_uint4(0u, 0u, 0u, 0u), lo = hi;
    if (inside && row < c.rows) {
      const uint32_t words[4] = {raw[i].x, raw[i].y, raw[i].z, raw[i].w};
      uint32_t a[4], b[4];
      float scale[8];
      if (GATE == kChannel) {
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          scale[4 * j] = exp_fast(E4[j].x - L4[i][j].x);
          scale[4 * j + 1] = exp_fast(E4[j].y - L4[i][j].y);
          scale[4 * j + 2] = exp_fast(E4[j].z - L4[i][j].z);
          scale[4 * j + 3] = exp_fast(E4[j].w - L4[i][j].w);
        }
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) scale[j] = f[i];
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 x = unpack2(words[j]);
        const float x0 = x.x * scale[2 * j], x1 = x.y * scale[2 * j + 1];
        a[j] = mma::pack(x0, x1);
        b[j] = mma::pack_remainder(x0, x1, a[j]);
      }
      hi = make_uint4(a[0], a[1], a[2], a[3]);
      lo = make_uint4(b[0], b[1], b[2], b[3]);
    }
    *reinterpret_cast<uint4*>(kh + row * kKeyLd + col) = hi;
    *reinterpret_cast<uint4*>(kl + row * kKeyLd + col) = lo;
  }
  mma::copy_async_wait<0>();
  __syncthreads();
  if (warp * 16 >= dims) return;
  float U[VT / 8][4], sum[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
  for (int i = 0; i < VT / 8; ++i) U[i][0] = U[i][1] = U[i][2] = U[i][3] = 0.0f;
  const int steps = (c.rows + 15) / 16;
  for (int kk = 0; kk < steps; ++kk) {
    uint32_t ah[4], al[4];
    const int at = (kk * 16 + (lane >> 4) * 8 + (lane & 7)) * kKeyLd + warp * 16 + ((lane >> 3) & 1) * 8;
    mma::load_matrices_transposed(ah, kh + at);
    mma::load_matrices_transposed(al, kl + at);
#pragma unroll
    for (int u = 0; u < VT / 16; ++u) {
      uint32_t b[4];
      mma::load_matrices_transposed(b, vs + (kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * (VT + 8) + u * 16 + (lane >> 4) * 8);
      mma::multiply_add(U[2 * u], ah, b[0], b[1]);
      mma::multiply_add(U[2 * u + 1], ah, b[2], b[3]);
      mma::multiply_add(U[2 * u], al, b[0], b[1]);
      mma::multiply_add(U[2 * u + 1], al, b[2], b[3]);
    }
    if (GATE == kExp) {                                      // the key sum: a column of ones
      mma::multiply_add(sum, ah, 0x3f803f80u, 0x3f803f80u);
      mma::multiply_add(sum, al, 0x3f803f80u, 0x3f803f80u);
    }
  }
  const int da = d0 + warp * 16 + (lane >> 2), db = da + 8;
  float* base = p.chunk_states + (static_cast<long long>(c.index) * p.heads + h) * p.dim * p.ld_state;
#pragma unroll
  for (int i = 0; i < VT / 8; ++i) {
    const int col = v0 + i * 8 + 2 * (lane & 3);
    if (col >= p.vdim) continue;                             // (vdim is a multiple of 8: the pair is inside)
    if (da < p.dim) *reinterpret_cast<float2*>(base + static_cast<long long>(da) * p.ld_state + col) = make_float2(U[i][0], U[i][1]);
    if (db < p.dim) *reinterpret_cast<float2*>(base + static_cast<long long>(db) * p.ld_state + col) = make_float2(U[i][2], U[i][3]);
  }
  if (GATE == kExp && v0 == 0 && (lane & 3) == 0) {
    if (da < p.dim) base[static_cast<long long>(da) * p.ld_state + p.vdim] = sum[0];
    if (db < p.dim) base[static_cast<long long>(db) * p.ld_state + p.vdim] = sum[2];
  }
}

// Block (request, head, 128 pieces of four columns of a row of S); kExp: the key sum is one more piece a row.
template <int GATE>
__global__ void __launch_bounds__(128)
memory_state_pass_kernel(const MemoryArgs p) {
  __shared__ int first_chunk;
  wait_for_prior_kernels();
  launch_dependents();
  const int r = blockIdx.x, h = blockIdx.y;
  const int lo = p.cu_q[r], n = p.cu_q[r + 1] - lo, slot = p.state_slots[r];
  if (n <= p.small_rows || slot < 0) return;
  if (threadIdx.x == 0) {
    int at = 0;
    for (int o = 0; o < r; ++o) {
      const int m = p.cu_q[o + 1] - p.cu_q[o];
      if (m > p.small_rows && p.state_slots[o] >= 0) at += (m + kChunkRows - 1) / kChunkRows;
    }
    first_chunk = at;
  }
  __syncthreads();
  const int pieces = p.vdim / 4 + (GATE == kExp ? 1 : 0);
  const int at = blockIdx.z * 128 + threadIdx.x;
  if (at >= p.dim * pieces) return;
  const int d = at / pieces, c4 = at % pieces;
  const bool sums = GATE == kExp && c4 == p.vdim / 4;
  float* base = p.state + slot * p.state_stride;
  float* Sg = sums ? base + static_cast<long long>(p.heads) * p.dim * p.vdim + static_cast<long long>(h) * p.dim + d
                   : base + (static_cast<long long>(h) * p.dim + d) * p.vdim + c4 * 4;
  float4 S = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  const bool wide = !sums && (reinterpret_cast<uintptr_t>(Sg) & 15) == 0;
  if (sums) S.x = Sg[0];
  else if (wide) S = *reinterpret_cast<const float4*>(Sg);
  else S = make_float4(Sg[0], Sg[1], Sg[2], Sg[3]);
  const long long step = static_cast<long long>(p.heads) * p.dim * p.ld_state;
  float* U = p.chunk_states + (static_cast<long long>(first_chunk) * p.heads + h) * p.dim * p.ld_state +
             static_cast<long long>(d) * p.ld_state + c4 * 4;
  const int chunks = (n + kChunkRows - 1) / kChunkRows;
  auto end_of = [&](int c) {
    const long long row = lo + min(n, (c + 1) * kChunkRows) - 1;
    return GATE == kChannel ? p.log_decay[row * p.heads * p.dim + static_cast<long long>(h) * p.dim + d] : p.log_decay[row * p.heads + h];
  };
  constexpr int kAhead = 8;                                  // chunks asked for together, ahead of the ones that are added
  float4 u[2][kAhead];
  float f[2][kAhead];
  auto fetch = [&](int c0, float4 (&uu)[kAhead], float (&ff)[kAhead]) {
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      if (c0 + i >= chunks) continue;
      ff[i] = end_of(c0 + i);
      if (sums) uu[i] = make_float4(U[(c0 + i) * step], 0.0f, 0.0f, 0.0f);
      else uu[i] = *reinterpret_cast<const float4*>(U + (c0 + i) * step);
    }
  };
  auto add = [&](int c0, const float4 (&uu)[kAhead], const float (&ff)[kAhead]) {
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      if (c0 + i >= chunks) continue;
      if (sums) U[(c0 + i) * step] = S.x;
      else *reinterpret_cast<float4*>(U + (c0 + i) * step) = S;
      const float decay = exp_fast(ff[i]);
      S.x = fmaf(decay, S.x, uu[i].x);
      S.y = fmaf(decay, S.y, uu[i].y);
      S.z = fmaf(decay, S.z, uu[i].z);
      S.w = fmaf(decay, S.w, uu[i].w);
    }
  };
  fetch(0, u[0], f[0]);
  for (int c0 = 0; c0 < chunks; c0 += 2 * kAhead) {
    fetch(c0 + kAhead, u[1], f[1]);
    add(c0, u[0], f[0]);
    fetch(c0 + 2 * kAhead, u[0], f[0]);
    add(c0 + kAhead, u[1], f[1]);
  }
  if (sums) Sg[0] = S.x;
  else if (wide) *reinterpret_cast<float4*>(Sg) = S;
  else { Sg[0] = S.x; Sg[1] = S.y; Sg[2] = S.z; Sg[3] = S.w; }
}

// the A fragment's (or a B fragment's) numbers times a factor each, as the pair of roundings and remainders
__device__ __forceinline__ void scale_pair(uint32_t raw, float f0, float f1, uint32_t& hi, uint32_t& lo) {
  const float2 x = unpack2(raw);
  const float a = x.x * f0, b = x.y * f1;
  hi = mma::pack(a, b);
  lo = mma::pack_remainder(a, b, hi);
}

constexpr float kSafeRange = 80.0f;                          // exp(80) times a number of ordinary size is far from overflow

template <int VT, int GATE>
struct ChunkOutShape {
  static constexpr size_t bytes = (2 * static_cast<size_t>(kChunkRows) * kKeyLd + 2 * kTileDim * (VT + 8) + kChunkRows * (VT + 8)) * 2 +
                                  (GATE == kChannel ? kChunkRows * kDecayLd * sizeof(float) : 0);
};

// Block (chunk, head, tile of VT value columns), a warp 16 rows of the chunk.
template <int VT, int GATE>
__global__ void __launch_bounds__(128)
memory_chunk_out_kernel(const MemoryArgs p) {
  typedef __nv_bfloat16 bf16;
  extern __shared__ __align__(16) unsigned char chunk_out_smem[];
  bf16* qs = reinterpret_cast<bf16*>(chunk_out_smem);        // [64 rows][kKeyLd]
  bf16* ks = qs + kChunkRows * kKeyLd;                       // [64 rows][kKeyLd]
  bf16* sh = ks + kChunkRows * kKeyLd;                       // the state in front of the chunk, [64 channels][VT + 8]: roundings ...
  bf16* sl = sh + kTileDim * (VT + 8);                       // ... and remainders
  bf16* vs = sl + kTileDim * (VT + 8);                       // [64 rows][VT + 8]
  float* Ls = reinterpret_cast<float*>(vs + kChunkRows * (VT + 8));   // kChannel: [64 rows][kDecayLd]
  __shared__ ChunkPlace place;
  __shared__ float L_s[kChunkRows], w_s[kChunkRows];         // kStep, kExp
  wait_for_prior_kernels();
  launch_dependents();
  const ChunkPlace c = find_chunk_shared(p, blockIdx.x, &place);
  if (c.request < 0) return;
  const int h = blockIdx.y, v0 = static_cast<int>(blockIdx.z) * VT, g = h / p.per_group;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, quad = lane & 3;
  const int cols = min(VT, p.vdim - v0), channels = p.heads * p.dim;
  const int ra = warp * 16 + (lane >> 2), rb = ra + 8;       // the thread's two rows
  load_values<VT>(vs, static_cast<const bf16*>(p.v) + static_cast<long long>(c.first) * p.ldv + static_cast<long long>(h) * p.vdim + v0,
                  p.ldv, c.rows, cols);
  if (GATE != kChannel && tid < kChunkRows) {
    const long long item = (static_cast<long long>(c.first) + min(tid, c.rows - 1)) * p.heads + h;
    L_s[tid] = p.log_decay[item];
    w_s[tid] = p.strength[item];
  }
  const float* state = p.chunk_states + (static_cast<long long>(c.index) * p.heads + h) * p.dim * p.ld_state;
  float O[VT / 8][4], P[8][4], N[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
  for (int i = 0; i < VT / 8; ++i) O[i][0] = O[i][1] = O[i][2] = O[i][3] = 0.0f;
#pragma unroll
  for (int i = 0; i < 8; ++i) P[i][0] = P[i][1] = P[i][2] = P[i][3] = 0.0f;
  const int rows_in_use = (c.rows + 15) / 16;                // warps with rows
  for (int d0 = 0; d0 < p.dim; d0 += kTileDim) {
    const int dims = min(kTileDim, p.dim - d0);
    if (d0 > 0) __syncthreads();                             // (the tile before is done with)
    load_rows(qs, static_cast<const bf16*>(p.q) + static_cast<long long>(c.first) * p.ldq + static_cast<long long>(g) * p.dim + d0, p.ldq,
              c.rows, dims);
    load_rows(ks, static_cast<const bf16*>(p.k) + static_cast<long long>(c.first) * p.ldk + static_cast<long long>(g) * p.dim + d0, p.ldk,
              c.rows, dims);
    if (GATE == kChannel) {
      const float* L = p.log_decay + static_cast<long long>(c.first) * channels + static_cast<long long>(h) * p.dim + d0;
      for (int e = tid; e < kChunkRows * (kTileDim / 4); e += 128) {
        const int row = e / (kTileDim / 4), col = (e % (kTileDim / 4)) * 4;
        float* dst = Ls + row * kDecayLd + col;
        if (col < dims) mma::copy_async_16(dst, L + static_cast<long long>(min(row, c.rows - 1)) * channels + col);
        else *reinterpret_cast<float4*>(dst) = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      }
    }
    mma::copy_async_commit();
    constexpr int kBatch = 8;                                // pieces of the state asked for together
    static_assert(kTileDim * (VT / 4) % (128 * kBatch) == 0, "whole batches");
    for (int e0 = tid; e0 < kTileDim * (VT / 4); e0 += 128 * kBatch) {
      float4 x[kBatch];
#pragma unroll
      for (int i = 0; i < kBatch; ++i) {
        const int e = e0 + 128 * i, d = e / (VT / 4), col = (e % (VT / 4)) * 4;
        x[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (d < dims && col < cols)
          x[i] = *reinterpret_cast<const float4*>(state + static_cast<long long>(d0 + d) * p.ld_state + v0 + col);
      }
#pragma unroll
      for (int i = 0; i < kBatch; ++i) {
        const int e = e0 + 128 * i, d = e / (VT / 4), col = (e % (VT / 4)) * 4;
        const uint2 hi = make_uint2(mma::pack(x[i].x, x[i].y), mma::pack(x[i].z, x[i].w));
        const uint2 lo = make_uint2(mma::pack_remainder(x[i].x, x[i].y, hi.x), mma::pack_remainder(x[i].z, x[i].w, hi.y));
        *reinterpret_cast<uint2*>(sh + d * (VT + 8) + col) = hi;
        *reinterpret_cast<uint2*>(sl + d * (VT + 8) + col) = lo;
      }
    }
    mma::copy_async_wait<0>();
    __syncthreads();
    if (warp >= rows_in_use) continue;
    // kChannel: the decays of the warp's rows are counted from the row in front of them
    const float* Lref = GATE == kChannel && warp > 0 ? Ls + (warp * 16 - 1) * kDecayLd : nullptr;
    bool one_by_one = false;
    if (GATE == kChannel) {
      const float* Lend = Ls + min(warp * 16 + 15, c.rows - 1) * kDecayLd;
      float range = 0.0f;
      for (int d = lane; d < dims; d += 32) range = fmaxf(range, (Lref != nullptr ? Lref[d] : 0.0f) - Lend[d]);
      one_by_one = __any_sync(0xffffffffu, range > kSafeRange);
    }
#pragma unroll
    for (int kk = 0; kk < kTileDim / 16; ++kk) {
      if (kk * 16 >= dims) break;
      uint32_t a[4];
      mma::load_matrices(a, qs + (warp * 16 + (lane & 15)) * kKeyLd + kk * 16 + (lane >> 4) * 8);
      uint32_t th[4], tl[4];                                 // kChannel: q exp(L - Lref), for the scores
      uint32_t sq[4], sr[4];                                 // kChannel: q exp(L), for the state
      float ref[4];                                          // Lref of channels 2 quad, + 1, + 8, + 9 of the step
      if (GATE == kChannel) {
#pragma unroll
        for (int i = 0; i < 4; ++i) ref[i] = Lref != nullptr ? Lref[kk * 16 + 2 * quad + (i >> 1) * 8 + (i & 1)] : 0.0f;
#pragma unroll
        for (int i = 0; i < 4; ++i) {                          // a[i]: row ra (i even) or rb, channels 2 quad (+ 8: i >= 2), + 1
          const float* L = Ls + ((i & 1) ? rb : ra) * kDecayLd + kk * 16 + 2 * quad + (i >> 1) * 8;
          const float l0 = L[0], l1 = L[1];
          scale_pair(a[i], exp_fast(l0 - ref[(i >> 1) * 2]), exp_fast(l1 - ref[(i >> 1) * 2 + 1]), th[i], tl[i]);
          scale_pair(a[i], exp_fast(l0), exp_fast(l1), sq[i], sr[i]);
        }
      }
      // scores against the rows of the chunk up to the warp's own
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        if (np > warp || (GATE == kChannel && one_by_one && np == warp)) continue;
        uint32_t b[4];
        mma::load_matrices(b, ks + (np * 16 + (lane >> 4) * 8 + (lane & 7)) * kKeyLd + kk * 16 + ((lane >> 3) & 1) * 8);
        if (GATE == kChannel) {
          uint32_t bh[4], bl[4];
#pragma unroll
          for (int i = 0; i < 4; ++i) {                        // b[i]: row lane / 4 (+ 8: i >= 2) of the 16, channels 2 quad (+ 8: i odd), + 1
            const float* L = Ls + (np * 16 + (i >> 1) * 8 + (lane >> 2)) * kDecayLd + kk * 16 + 2 * quad + (i & 1) * 8;
            scale_pair(b[i], exp_fast(ref[(i & 1) * 2] - L[0]), exp_fast(ref[(i & 1) * 2 + 1] - L[1]), bh[i], bl[i]);
          }
          mma::multiply_add(P[2 * np], th, bh[0], bh[1]);
          mma::multiply_add(P[2 * np + 1], th, bh[2], bh[3]);
          mma::multiply_add(P[2 * np], th, bl[0], bl[1]);
          mma::multiply_add(P[2 * np + 1], th, bl[2], bl[3]);
          mma::multiply_add(P[2 * np], tl, bh[0], bh[1]);
          mma::multiply_add(P[2 * np + 1], tl, bh[2], bh[3]);
        } else {
          mma::multiply_add(P[2 * np], a, b[0], b[1]);
          mma::multiply_add(P[2 * np + 1], a, b[2], b[3]);
        }
      }
      // the state
#pragma unroll
      for (int u = 0; u < VT / 16; ++u) {
        uint32_t bh[4], bl[4];
        const int at = (kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * (VT + 8) + u * 16 + (lane >> 4) * 8;
        mma::load_matrices_transposed(bh, sh + at);
        mma::load_matrices_transposed(bl, sl + at);
        if (GATE == kChannel) {
          mma::multiply_add(O[2 * u], sq, bh[0], bh[1]);
          mma::multiply_add(O[2 * u + 1], sq, bh[2], bh[3]);
          mma::multiply_add(O[2 * u], sq, bl[0], bl[1]);
          mma::multiply_add(O[2 * u + 1], sq, bl[2], bl[3]);
          mma::multiply_add(O[2 * u], sr, bh[0], bh[1]);
          mma::multiply_add(O[2 * u + 1], sr, bh[2], bh[3]);
        } else {
          mma::multiply_add(O[2 * u], a, bh[0], bh[1]);
          mma::multiply_add(O[2 * u + 1], a, bh[2], bh[3]);
          mma::multiply_add(O[2 * u], a, bl[0], bl[1]);
          mma::multiply_add(O[2 * u + 1], a, bl[2], bl[3]);
        }
      }
      if (GATE == kExp && v0 == 0) {                           // the key sum in front of the chunk, as the first of 8 columns
        uint32_t bh[2] = {0u, 0u}, bl[2] = {0u, 0u};
        if (lane < 4) {
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const int d = kk * 16 + 2 * quad + i * 8;
            const float* n = state + static_cast<long long>(d0 + d) * p.ld_state + p.vdim;
            const float n0 = d < dims ? n[0] : 0.0f, n1 = d + 1 < dims ? n[p.ld_state] : 0.0f;
            bh[i] = mma::pack(n0, n1);
            bl[i] = mma::pack_remainder(n0, n1, bh[i]);
          }
        }
        mma::multiply_add(N, a, bh[0], bh[1]);
        mma::multiply_add(N, a, bl[0], bl[1]);
      }
    }
    if (GATE == kChannel && one_by_one) {
      // the warp's 16 x 16 scores against its own rows, each factor exp(L_i - L_j) by itself
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int ri = (i & 2) ? rb : ra, rj = warp * 16 + (i >> 2) * 8 + 2 * quad + (i & 1);
        if (rj > ri) continue;
        float s = 0.0f;
        for (int d = 0; d < dims; ++d)
          s = fmaf(__bfloat162float(qs[ri * kKeyLd + d]) * __bfloat162float(ks[rj * kKeyLd + d]),
                   exp_fast(Ls[ri * kDecayLd + d] - Ls[rj * kDecayLd + d]), s);
        // (the loop over i is unrolled; P is indexed by constants but for the warp)
#pragma unroll
        for (int np = 0; np < 4; ++np)
          if (np == warp) P[2 * np + (i >> 2)][i & 3] += s;
      }
    }
  }
  if (warp >= rows_in_use) return;
  // the scores' factors and the causal mask; the state's part takes its decay
  const float La = GATE == kChannel ? 0.0f : L_s[ra], Lb = GATE == kChannel ? 0.0f : L_s[rb];
  float fa = 1.0f, fb = 1.0f, den_a = 0.0f, den_b = 0.0f;
  if (GATE != kChannel) {
    fa = exp_fast(La);
    fb = exp_fast(Lb);
#pragma unroll
    for (int i = 0; i < VT / 8; ++i) {
      O[i][0] *= fa;
      O[i][1] *= fa;
      O[i][2] *= fb;
      O[i][3] *= fb;
    }
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    if (i / 2 > warp) continue;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int j = i * 8 + 2 * quad + e;
      float wa = 1.0f, wb = 1.0f;
      if (GATE != kChannel) {
        wa = exp_fast(fminf(La - L_s[j], 0.0f)) * w_s[j];
        wb = exp_fast(fminf(Lb - L_s[j], 0.0f)) * w_s[j];
      }
      P[i][e] = j <= ra ? P[i][e] * wa : 0.0f;
      P[i][2 + e] = j <= rb ? P[i][2 + e] * wb : 0.0f;
      if (GATE == kExp) {
        den_a += P[i][e];
        den_b += P[i][2 + e];
      }
    }
  }
#pragma unroll
  for (int kk = 0; kk < 4; ++kk) {
    if (kk > warp) continue;
    uint32_t hi[4], lo[4];
    hi[0] = mma::pack(P[2 * kk][0], P[2 * kk][1]);
    hi[1] = mma::pack(P[2 * kk][2], P[2 * kk][3]);
    hi[2] = mma::pack(P[2 * kk + 1][0], P[2 * kk + 1][1]);
    hi[3] = mma::pack(P[2 * kk + 1][2], P[2 * kk + 1][3]);
    lo[0] = mma::pack_remainder(P[2 * kk][0], P[2 * kk][1], hi[0]);
    lo[1] = mma::pack_remainder(P[2 * kk][2], P[2 * kk][3], hi[1]);
    lo[2] = mma::pack_remainder(P[2 * kk + 1][0], P[2 * kk + 1][1], hi[2]);
    lo[3] = mma::pack_remainder(P[2 * kk + 1][2], P[2 * kk + 1][3], hi[3]);
#pragma unroll
    for (int u = 0; u < VT / 16; ++u) {
      uint32_t b[4];
      mma::load_matrices_transposed(b, vs + (kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * (VT + 8) + u * 16 + (lane >> 4) * 8);
      mma::multiply_add(O[2 * u], hi, b[0], b[1]);
      mma::multiply_add(O[2 * u + 1], hi, b[2], b[3]);
      mma::multiply_add(O[2 * u], lo, b[0], b[1]);
      mma::multiply_add(O[2 * u + 1], lo, b[2], b[3]);
    }
  }
  const long long item_a = (static_cast<long long>(c.first) + ra) * p.heads + h, item_b = item_a + 8LL * p.heads;
  if (GATE == kExp && v0 == 0) {
    den_a += __shfl_xor_sync(0xffffffffu, den_a, 1);
    den_a += __shfl_xor_sync(0xffffffffu, den_a, 2);
    den_b += __shfl_xor_sync(0xffffffffu, den_b, 1);
    den_b += __shfl_xor_sync(0xffffffffu, den_b, 2);
    if (quad == 0) {
      if (ra < c.rows) p.divisor[item_a] = fmaxf(fabsf(fmaf(fa, N[0], den_a) * p.q_scale), p.lowest[item_a]) + p.floor;
      if (rb < c.rows) p.divisor[item_b] = fmaxf(fabsf(fmaf(fb, N[2], den_b) * p.q_scale), p.lowest[item_b]) + p.floor;
    }
  }
  const float skip = p.skip != nullptr ? p.skip[h] : 0.0f;
#pragma unroll
  for (int i = 0; i < VT / 8; ++i) {
    const int col = i * 8 + 2 * quad;
    if (col >= cols) continue;
    if (ra < c.rows) {
      const float2 x = unpack2(*reinterpret_cast<const uint32_t*>(vs + ra * (VT + 8) + col));
      *reinterpret_cast<float2*>(p.out + item_a * p.vdim + v0 + col) =
          make_float2(fmaf(skip, x.x, O[i][0] * p.q_scale), fmaf(skip, x.y, O[i][1] * p.q_scale));
    }
    if (rb < c.rows) {
      const float2 x = unpack2(*reinterpret_cast<const uint32_t*>(vs + rb * (VT + 8) + col));
      *reinterpret_cast<float2*>(p.out + item_b * p.vdim + v0 + col) =
          make_float2(fmaf(skip, x.x, O[i][2] * p.q_scale), fmaf(skip, x.y, O[i][3] * p.q_scale));
    }
  }
}

}  // namespace pih

using namespace pih;
typedef __nv_bfloat16 bf16;

template <typename T, int D, int GATE>
static int launch_memory_recurrence(cudaStream_t s, const MemoryArgs& p, int requests) {
  typedef MemoryShape<D> Shape;
  constexpr size_t bytes = Shape::bytes(GATE);
  static bool raised = false;                                          // (per instance)
  if (bytes > 48 * 1024 && !raised) {
    cudaFuncSetAttribute(memory_recurrence_kernel<T, D, GATE>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                         static_cast<int>(bytes));
    raised = true;
  }
  const dim3 grid(requests, p.heads, (p.vdim + 31) / 32 + (GATE == kExp ? 1 : 0));
  launch_kernel(memory_recurrence_kernel<T, D, GATE>, grid, dim3(Shape::kThreads), bytes, s, p);
  PIH_LAUNCH_CHECK();
  return 0;
}

template <typename T, int GATE>
static int memory_recurrence_by_size(cudaStream_t s, const MemoryArgs& p, int requests) {
  if (p.dim <= 16) return launch_memory_recurrence<T, 16, GATE>(s, p, requests);
  if (p.dim <= 32) return launch_memory_recurrence<T, 32, GATE>(s, p, requests);
  if (p.dim <= 64) return launch_memory_recurrence<T, 64, GATE>(s, p, requests);
  if (p.dim <= 128) return launch_memory_recurrence<T, 128, GATE>(s, p, requests);
  if (p.dim <= 256) return launch_memory_recurrence<T, 256, GATE>(s, p, requests);
  if (p.dim <= 512) return launch_memory_recurrence<T, 512, GATE>(s, p, requests);
  return launch_memory_recurrence<T, 1024, GATE>(s, p, requests);
}

static long long chunks_at_most(int rows, int requests) { return rows / kChunkRows + requests; }

static bool goes_by_chunks(int dtype, const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv,
                           int dim, int vdim) {
  auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  return dtype == PIH_BF16 && dim % 8 == 0 && vdim % 8 == 0 && ldq % 8 == 0 && ldk % 8 == 0 && ldv % 8 == 0 && aligned(q) &&
         aligned(k) && aligned(v);
}

template <int VT, int GATE>
static int launch_memory_chunks(cudaStream_t s, const MemoryArgs& p, int rows, int requests) {
  const long long chunks = chunks_at_most(rows, requests);
  const int vtiles = (p.vdim + VT - 1) / VT, dtiles = (p.dim + kTileDim - 1) / kTileDim;
  if (vtiles * dtiles > 65535) return PIH_ERR_UNSUPPORTED;
  if (GATE == kChannel)
    launch_kernel(memory_channels_kernel, dim3(static_cast<unsigned>(chunks), (p.heads * p.dim + 127) / 128), dim3(128), 0, s, p);
  else
    launch_kernel(memory_gates_kernel<bf16, GATE>, dim3(requests, p.heads), dim3(32 * kGateWarps), 0, s, p);
  PIH_LAUNCH_CHECK();
  constexpr size_t state_bytes = (2 * static_cast<size_t>(kChunkRows) * kKeyLd + kChunkRows * (VT + 8)) * sizeof(bf16);
  static_assert(state_bytes <= 48 * 1024, "no opt-in needed");
  launch_kernel(memory_chunk_state_kernel<VT, GATE>, dim3(static_cast<unsigned>(chunks), p.heads, vtiles * dtiles), dim3(128),
                state_bytes, s, p);
  PIH_LAUNCH_CHECK();
  const int pieces = p.dim * (p.vdim / 4 + (GATE == kExp ? 1 : 0));
  launch_kernel(memory_state_pass_kernel<GATE>, dim3(requests, p.heads, (pieces + 127) / 128), dim3(128), 0, s, p);
  PIH_LAUNCH_CHECK();
  constexpr size_t out_bytes = ChunkOutShape<VT, GATE>::bytes;
  static bool raised = false;                                          // (per instance)
  if (out_bytes > 48 * 1024 && !raised) {
    cudaFuncSetAttribute(memory_chunk_out_kernel<VT, GATE>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                         static_cast<int>(out_bytes));
    raised = true;
  }
  launch_kernel(memory_chunk_out_kernel<VT, GATE>, dim3(static_cast<unsigned>(chunks), p.heads, vtiles), dim3(128), out_bytes, s, p);
  PIH_LAUNCH_CHECK();
  return 0;
}

// fp32 numbers of scratch that a step of ``rows`` rows needs where requests of more than small_rows rows go by chunks; 0:
// they do not (pih_linear_memory's ``chunked`` has to be 0 then).
extern "C" long long pih_linear_memory_scratch(int dtype, int gate, const void* q, long long ldq, const void* k, long long ldk,
                                               const void* v, long long ldv, int rows, int requests, int heads, int dim,
                                               int vdim) {
  if (!goes_by_chunks(dtype, q, ldq, k, ldk, v, ldv, dim, vdim)) return 0;
  const long long ld_state = vdim + (gate == kExp ? 8 : 0);
  const long long items = (static_cast<long long>(rows) * heads + 3) / 4 * 4;
  return (gate == kChannel ? items * dim : 3 * items) + chunks_at_most(rows, requests) * heads * dim * ld_state;
}

// How many running maxima a head keeps in its state (kExp): one a block of memory_recurrence.
extern "C" int pih_memory_copies(int vdim) { return (vdim + 31) / 32 + 1; }

// The state update and read-out of a step's rows; ``gate`` a MemoryGate.  q, k, v views of ``dtype`` with row strides; gate0
// fp32 for kChannel, else of ``dtype``; constant 1 / temperature (kChannel) or the cap (kExp); out fp32 [rows, heads, vdim];
// divisor fp32 [rows, heads] (kExp).  scratch: null, or pih_linear_memory_scratch numbers, 16-byte aligned: requests of more
// than 16 rows go by chunks on tensor cores; ``small`` 0 says that there are no others.
extern "C" int pih_linear_memory(int dtype, int gate, const void* q, long long ldq, const void* k, long long ldk, const void* v,
                                 long long ldv, const void* gate0, long long ld0, const void* gate1, long long ld1,
                                 const void* bias0, const void* bias1, const void* A, float constant, float floor,
                                 float q_scale, const void* skip, void* out, void* divisor, void* state,
                                 long long state_stride, const void* cu_q, const void* state_slots, int rows, int requests,
                                 int heads, int groups, int dim, int vdim, void* scratch, int small, void* stream) {
  if (rows <= 0 || requests <= 0) return 0;
  if (heads < 1 || groups < 1 || heads % groups || dim < 1 || vdim < 1) return PIH_ERR_BAD_ARGUMENT;
  if ((gate == kChannel || gate == kExp) && groups != heads) return PIH_ERR_BAD_ARGUMENT;
  if (gate == kExp && (divisor == nullptr || gate1 == nullptr || bias1 == nullptr)) return PIH_ERR_BAD_ARGUMENT;
  if (gate == kStep && A == nullptr) return PIH_ERR_BAD_ARGUMENT;
  if (dim > 1024 || heads > 65535 || vdim > 32 * 65000) return PIH_ERR_UNSUPPORTED;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  MemoryArgs p;
  p.q = q; p.ldq = ldq; p.k = k; p.ldk = ldk; p.v = v; p.ldv = ldv;
  p.gate0 = gate0; p.ld0 = ld0; p.gate1 = gate1; p.ld1 = ld1;
  p.bias0 = static_cast<const float*>(bias0);
  p.bias1 = static_cast<const float*>(bias1);
  p.A = static_cast<const float*>(A);
  p.constant = constant; p.floor = floor; p.q_scale = q_scale;
  p.skip = static_cast<const float*>(skip);
  p.out = static_cast<float*>(out);
  p.divisor = static_cast<float*>(divisor);
  p.state = static_cast<float*>(state);
  p.state_stride = state_stride;
  p.cu_q = static_cast<const int*>(cu_q);
  p.state_slots = static_cast<const int*>(state_slots);
  p.heads = heads; p.per_group = heads / groups; p.dim = dim; p.vdim = vdim; p.copies = pih_memory_copies(vdim);
  p.small_rows = scratch != nullptr ? 16 : 0x7fffffff;
  p.requests = requests;
  p.ld_state = vdim + (gate == kExp ? 8 : 0);
  p.log_decay = p.strength = p.lowest = p.chunk_states = nullptr;
  if (scratch != nullptr) {
    if (!goes_by_chunks(dtype, q, ldq, k, ldk, v, ldv, dim, vdim) || (reinterpret_cast<uintptr_t>(scratch) & 15))
      return PIH_ERR_UNSUPPORTED;
    const long long items = (static_cast<long long>(rows) * heads + 3) / 4 * 4;
    p.log_decay = static_cast<float*>(scratch);
    p.strength = p.log_decay + items;
    p.lowest = p.strength + items;
    p.chunk_states = p.log_decay + (gate == kChannel ? items * dim : 3 * items);
    int rc;
#define PIH_CHUNKS(GATE)                                                                                               \
  rc = vdim <= 64 ? launch_memory_chunks<64, GATE>(s, p, rows, requests) : launch_memory_chunks<128, GATE>(s, p, rows, requests)
    switch (gate) {
      case kChannel: PIH_CHUNKS(kChannel); break;
      case kStep: PIH_CHUNKS(kStep); break;
      case kExp: PIH_CHUNKS(kExp); break;
      default: return PIH_ERR_BAD_ARGUMENT;
    }
#undef PIH_CHUNKS
    if (rc != 0) return rc;
    if (!small) return 0;
  }
#define PIH_MEM(T)                                                                                                     \
  switch (gate) {                                                                                                      \
    case kChannel: return memory_recurrence_by_size<T, kChannel>(s, p, requests);                                      \
    case kStep: return memory_recurrence_by_size<T, kStep>(s, p, requests);                                            \
    case kExp: return memory_recurrence_by_size<T, kExp>(s, p, requests);                                              \
    default: return PIH_ERR_BAD_ARGUMENT;                                                                              \
  }
  if (dtype == PIH_F32) { PIH_MEM(float) }
  if (dtype == PIH_BF16) { PIH_MEM(bf16) }
  return PIH_ERR_BAD_ARGUMENT;
#undef PIH_MEM
}
