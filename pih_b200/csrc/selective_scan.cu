// Selective scan: a diagonal recurrence with ``state`` numbers a channel whose step size, input and read-out vectors come
// from the token.  Per channel c and state n, token by token, S starting at zero:
//
//   dt = softplus(logit[c] + bias[c])
//   S[c][n] <- exp(dt A[c][n]) S[c][n] + dt x[c] B[n]
//   y[c]     = sum_n S[c][n] C[n] + D[c] x[c];     out[c] = y[c] silu(z[c]) times one number
//
// (the recurrence of Gu and Dao, "Mamba: Linear-Time Sequence Modeling with Selective State Spaces").
//
// A block is CH channels of one request; kParts neighbouring lanes hold a channel, kN states each, S and A in registers.
// The request's rows go by in chunks of 16.  A chunk: (1) every thread makes (dt, dt x) of its (row, channel) pairs and
// B, C go to shared memory in 32-bit; (2) the recurrence runs over the chunk's rows, a lane's share of y for each of the 16
// rows in a register; these shares meet over the lanes of a channel by halving exchanges (a lane hands the half of the
// rows that it does not keep to its partner: 15 shuffles for 16 rows and 16 lanes instead of 64); (3) every thread
// finishes the (row, channel) pairs that it began.  The next chunk's numbers are asked for before (2).
//
// State, step sizes, exponentials and sums are 32-bit.  The 32-bit path forms exp(dt A) S as S + expm1(dt A) S, so that a
// state that remembers long keeps the distance of its decay from one; the bf16 path takes the special-function unit's 2^x.
// The order of additions of a row does not depend on the row's place in its chunk, so a cut of the prompt changes nothing.
#include "common.cuh"
#include "mma.cuh"

namespace pih {

constexpr int kScanRows = 16;               // rows of a chunk

struct ScanArgs {
  const void* u;                            // [rows, ldu]: the channels' inputs
  long long ldu;
  const float* dt;                          // [rows, lddt]: step-size logits without their bias
  long long lddt;
  const float* dt_bias;                     // [inner]
  const float* A;                           // [inner, state]
  const void* bc;                           // [rows, ldbc]: B, then C
  long long ldbc;
  const float* D;                           // [inner]
  const void* z;                            // [rows, ldz]
  long long ldz;
  void* out;                                // [rows, ldo]
  long long ldo;
  float out_scale;
  float* state;                             // a slot: [inner, state] at its start
  long long state_stride;
  const int* cu_q;
  const int* state_slots;
  int inner, states;
};

// v[0 .. COUNT-1]: a lane's shares of COUNT rows.  Afterwards v[0 .. max(1, COUNT / 2^steps)-1] are whole sums (over the lanes
// that differ in the bits of MASK and below) of the rows from the returned one on.
template <int COUNT, int MASK>
__device__ __forceinline__ int fold_shares(float* v, int part) {
  if constexpr (MASK == 0) {
    return 0;
  } else if constexpr (COUNT == 1) {
    v[0] += __shfl_xor_sync(0xffffffffu, v[0], MASK);
    return fold_shares<1, MASK / 2>(v, part);
  } else {
    constexpr int H = COUNT / 2;
    const bool upper = (part & MASK) != 0;
#pragma unroll
    for (int i = 0; i < H; ++i) {
      const float send = upper ? v[i] : v[i + H], keep = upper ? v[i + H] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, send, MASK);
    }
    return (upper ? H : 0) + fold_shares<H, MASK / 2>(v, part);
  }
}

template <int kParts>
struct ScanShape {
  static constexpr int CH = kParts >= 4 ? 16 : 64 / kParts;            // channels a block
  static constexpr int kThreads = CH * kParts;
};

template <typename T, int kParts, int kN>
__global__ void __launch_bounds__(ScanShape<kParts>::kThreads)
selective_scan_kernel(const ScanArgs p) {
  constexpr bool kExact = sizeof(T) == 4;
  constexpr int CH = ScanShape<kParts>::CH, TH = ScanShape<kParts>::kThreads;
  constexpr int NP = kParts * kN;                                       // states with the padding
  constexpr int E = (kScanRows * CH + TH - 1) / TH;                     // (row, channel) pairs a thread
  constexpr int EB = kScanRows * 2 * NP / TH;                           // numbers of B and C a thread
  static_assert(kScanRows * 2 * NP % TH == 0 && kN % 2 == 0, "whole shares, 8-byte loads");
  extern __shared__ __align__(16) float scan_smem[];
  typedef float2 (*Steps)[CH];
  typedef float (*Vectors)[2][NP];
  typedef float (*Outputs)[CH];
  Vectors bc_s = reinterpret_cast<Vectors>(scan_smem);                  // [rows][B, C][NP]
  Steps steps = reinterpret_cast<Steps>(scan_smem + kScanRows * 2 * NP);                    // [rows][CH]: (dt, dt x)
  Outputs y_s = reinterpret_cast<Outputs>(scan_smem + kScanRows * (2 * NP + 2 * CH));       // [rows][CH]
  wait_for_prior_kernels();
  launch_dependents();
  const int r = blockIdx.x, c0 = blockIdx.y * CH, tid = threadIdx.x;
  const int lo = p.cu_q[r], hi = p.cu_q[r + 1], slot = p.state_slots[r];
  if (hi <= lo || slot < 0) return;
  const T* u = static_cast<const T*>(p.u);
  const T* bc = static_cast<const T*>(p.bc);
  const T* z = static_cast<const T*>(p.z);
  T* out = static_cast<T*>(p.out);
  const int part = tid % kParts, cl = tid / kParts, c = c0 + cl, n0 = part * kN;
  const bool live = c < p.inner;
  float* Sg = p.state + slot * p.state_stride + static_cast<long long>(c) * p.states;
  float S[kN], A[kN];
#pragma unroll
  for (int i = 0; i < kN; ++i) {
    const bool there = live && n0 + i < p.states;
    S[i] = there ? Sg[n0 + i] : 0.0f;
    A[i] = there ? p.A[static_cast<long long>(c) * p.states + n0 + i] * (kExact ? 1.0f : 1.4426950408889634f) : 0.0f;
  }
  // pair e of this thread: row (tid + e TH) / CH of the chunk, channel (tid + e TH) % CH of the block
  float bias[E], skip[E];
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const int ce = c0 + (tid + e * TH) % CH;
    bias[e] = ce < p.inner ? p.dt_bias[ce] : 0.0f;
    skip[e] = ce < p.inner ? p.D[ce] : 0.0f;
  }
  // the next chunk's numbers, as they lie in memory: nothing is computed from them before they are needed
  T nx[E], nz[E], nbc[EB];
  float nt[E];
  const T zero = from_float<T>(0.0f);
  auto fetch = [&](int t0) {
#pragma unroll
    for (int e = 0; e < E; ++e) {
      const int idx = tid + e * TH, t = t0 + idx / CH, ce = c0 + idx % CH;
      const bool there = idx < kScanRows * CH && t < hi && ce < p.inner;
      nx[e] = there ? u[t * p.ldu + ce] : zero;
      nz[e] = there ? z[t * p.ldz + ce] : zero;
      nt[e] = there ? p.dt[t * p.lddt + ce] : 0.0f;
    }
#pragma unroll
    for (int e = 0; e < EB; ++e) {
      const int idx = tid + e * TH, t = t0 + idx / (2 * NP), which = (idx / NP) & 1, n = idx % NP;
      nbc[e] = t < hi && n < p.states ? bc[t * p.ldbc + which * p.states + n] : zero;
    }
  };
  fetch(lo);
  for (int t0 = lo; t0 < hi; t0 += kScanRows) {
    const int n_rows = min(kScanRows, hi - t0);
    float x[E];
    T zz[E];
#pragma unroll
    for (int e = 0; e < E; ++e) {
      const int idx = tid + e * TH;
      x[e] = to_float<T>(nx[e]);
      zz[e] = nz[e];
      const float dt = softplus_f(nt[e] + bias[e]);
      if (idx < kScanRows * CH) steps[idx / CH][idx % CH] = make_float2(dt, dt * x[e]);
    }
#pragma unroll
    for (int e = 0; e < EB; ++e) scan_smem[tid + e * TH] = to_float<T>(nbc[e]);
    __syncthreads();
    if (t0 + kScanRows < hi) fetch(t0 + kScanRows);
    float share[kScanRows];
    auto row = [&](int t) {
      const float2 st = steps[t][cl];
      float B[kN], C[kN];
#pragma unroll
      for (int i = 0; i < kN; i += 2) {
        const float2 b2 = *reinterpret_cast<const float2*>(&bc_s[t][0][n0 + i]);
        const float2 c2 = *reinterpret_cast<const float2*>(&bc_s[t][1][n0 + i]);
        B[i] = b2.x; B[i + 1] = b2.y;
        C[i] = c2.x; C[i + 1] = c2.y;
      }
      float y = 0.0f;
#pragma unroll
      for (int i = 0; i < kN; ++i) {
        if (kExact) S[i] = fmaf(expm1f(st.x * A[i]), S[i], fmaf(st.y, B[i], S[i]));
        else S[i] = fmaf(mma::exp2_fast(st.x * A[i]), S[i], st.y * B[i]);
        y = fmaf(S[i], C[i], y);
      }
      share[t] = y;
    };
    if (n_rows == kScanRows) {                                          // (the same for the whole block; no branch a row, so
#pragma unroll                                                          // that the rows' loads and exponentials overlap)
      for (int t = 0; t < kScanRows; ++t) row(t);
    } else {
#pragma unroll
      for (int t = 0; t < kScanRows; ++t) {
        share[t] = 0.0f;
        if (t < n_rows) row(t);
      }
    }
    const int first = fold_shares<kScanRows, kParts / 2>(share, part);
    constexpr int kKept = kScanRows / kParts > 0 ? kScanRows / kParts : 1;
#pragma unroll
    for (int i = 0; i < kKept; ++i) y_s[first + i][cl] = share[i];      // (more lanes than rows: two write the same sum)
    __syncthreads();
#pragma unroll
    for (int e = 0; e < E; ++e) {
      const int idx = tid + e * TH, t = idx / CH, ce = c0 + idx % CH;
      if (idx < kScanRows * CH && t < n_rows && ce < p.inner) {
        const float y = fmaf(skip[e], x[e], y_s[t][idx % CH]);
        out[(t0 + t) * p.ldo + ce] = from_float<T>(silu_times<T>(to_float<T>(zz[e]), y) * p.out_scale);
      }
    }
    // (y_s is written again only behind the next chunk's first barrier, steps and bc_s only behind this chunk's second)
  }
  if (live) {
#pragma unroll
    for (int i = 0; i < kN; ++i)
      if (n0 + i < p.states) Sg[n0 + i] = S[i];
  }
}

template <typename T, int kParts, int kN>
static void launch_scan(const ScanArgs& p, int requests, cudaStream_t s) {
  constexpr int CH = ScanShape<kParts>::CH;
  const dim3 grid(requests, (p.inner + CH - 1) / CH);
  const int needed = kScanRows * (2 * kParts * kN + 3 * CH) * static_cast<int>(sizeof(float));
  // the rows follow one another: with no more blocks than SMs every block asks for more than half of an SM's shared memory
  // and so gets an SM alone
  const bool alone = static_cast<long long>(grid.x) * grid.y <= 148;
  const int smem = alone && needed < 116 * 1024 ? 116 * 1024 : needed;
  static int raised = 48 * 1024;                               // (per instance)
  if (smem > raised) {
    cudaFuncSetAttribute(selective_scan_kernel<T, kParts, kN>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    raised = smem;
  }
  launch_kernel(selective_scan_kernel<T, kParts, kN>, grid, dim3(ScanShape<kParts>::kThreads), smem, s, p);
}

template <typename T>
static int dispatch_scan(const ScanArgs& p, int requests, cudaStream_t s) {
  const int n = p.states;
  if (n <= 4) launch_scan<T, 2, 2>(p, requests, s);
  else if (n <= 8) launch_scan<T, 4, 2>(p, requests, s);
  else if (n <= 16) launch_scan<T, 8, 2>(p, requests, s);
  else if (n <= 32) launch_scan<T, 16, 2>(p, requests, s);
  else if (n <= 64) launch_scan<T, 32, 2>(p, requests, s);
  else if (n <= 128) launch_scan<T, 32, 4>(p, requests, s);
  else if (n <= 256) launch_scan<T, 32, 8>(p, requests, s);
  else return PIH_ERR_UNSUPPORTED;
  PIH_LAUNCH_CHECK();
  return 0;
}

}  // namespace pih

using namespace pih;

// u, bc, z, out of ``dtype``, everything else fp32 (see ScanArgs).  ``state`` at most 256.
extern "C" int pih_selective_scan(int dtype, const void* u, long long ldu, const void* dt, long long lddt, const void* dt_bias,
                                  const void* A, const void* bc, long long ldbc, const void* D, const void* z, long long ldz,
                                  void* out, long long ldo, float out_scale, void* state, long long state_stride,
                                  const void* cu_q, const void* state_slots, int rows, int requests, int inner, int states,
                                  void* stream) {
  if (rows <= 0 || requests <= 0) return 0;
  if (inner < 1 || states < 1) return PIH_ERR_BAD_ARGUMENT;
  if ((inner + 15) / 16 > 65535) return PIH_ERR_UNSUPPORTED;
  ScanArgs p;
  p.u = u, p.ldu = ldu;
  p.dt = static_cast<const float*>(dt), p.lddt = lddt;
  p.dt_bias = static_cast<const float*>(dt_bias);
  p.A = static_cast<const float*>(A);
  p.bc = bc, p.ldbc = ldbc;
  p.D = static_cast<const float*>(D);
  p.z = z, p.ldz = ldz;
  p.out = out, p.ldo = ldo, p.out_scale = out_scale;
  p.state = static_cast<float*>(state), p.state_stride = state_stride;
  p.cu_q = static_cast<const int*>(cu_q);
  p.state_slots = static_cast<const int*>(state_slots);
  p.inner = inner, p.states = states;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == PIH_F32) return dispatch_scan<float>(p, requests, s);
  if (dtype == PIH_BF16) return dispatch_scan<__nv_bfloat16>(p, requests, s);
  return PIH_ERR_BAD_ARGUMENT;
}
