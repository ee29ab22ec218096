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
// States, decays, gates and sums are 32-bit whatever the storage type T.  The decay is applied as S + (a - 1) S with a - 1
// formed by expm1, so that a state that remembers long keeps the distance of its decay from one.
#include "common.cuh"

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
  int small_rows;                           // requests of more rows than this are another kernel's
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

// How many running maxima a head keeps in its state (kExp): one a block of memory_recurrence.
extern "C" int pih_memory_copies(int vdim) { return (vdim + 31) / 32 + 1; }

// The state update and read-out of a step's rows; ``gate`` a MemoryGate.  q, k, v views of ``dtype`` with row strides; gate0
// fp32 for kChannel, else of ``dtype``; constant 1 / temperature (kChannel) or the cap (kExp); out fp32 [rows, heads, vdim];
// divisor fp32 [rows, heads] (kExp).
extern "C" int pih_linear_memory(int dtype, int gate, const void* q, long long ldq, const void* k, long long ldk, const void* v,
                                 long long ldv, const void* gate0, long long ld0, const void* gate1, long long ld1,
                                 const void* bias0, const void* bias1, const void* A, float constant, float floor,
                                 float q_scale, const void* skip, void* out, void* divisor, void* state,
                                 long long state_stride, const void* cu_q, const void* state_slots, int rows, int requests,
                                 int heads, int groups, int dim, int vdim, void* stream) {
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
  p.small_rows = 0x7fffffff;
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
