// The real-gated linear recurrent unit: an elementwise linear recurrence per channel whose decay is computed from the data.
//
//   r = sigmoid(pr + br), i = sigmoid(pi + bi)          pr, pi: products of the channel's block of inputs, float32
//   log a = r * c                                       c = -8 softplus(lam) per channel, made when the weights are bound
//   S_t = exp(log a) S_(t-1) + sqrt(1 - exp(2 log a)) * i * u_t
//   out_t = S_t * gelu_tanh(y_t)                        rounded once to the activation dtype
//
// The decay is formed as 1 + x and the factor as sqrt(-x (2 + x)) with x = exp(log a) - 1 (expm1f): both keep their
// accuracy where a is close to one.  (A channel that forgets slowly multiplies by nearly the same a for a thousand rows: the
// error of a float32 exponential, a unit or two in the last place, adds up; that of 1 + x is half a unit at most.)
//
// S is float32, one number per channel and request ([slots, W]), read at the start of the run of rows a step brings for
// the request (req_first_token[r] .., as many as carry its index in token_req) and written back at its end.
//
// A linear recurrence is associative, so a run is cut into pieces of RG_LEN rows: each thread walks one piece of one
// channel from zero (end state B, product of decays A, the rows' a and b kept in registers), the pieces' (A, B) are
// chained through shared memory, and each thread walks its piece once more from the state the chain gives it.  A block
// takes RG_CHANNELS neighbouring channels and RG_PIECES pieces at a time, and goes on along the run; the rows of the
// pieces after these are asked for before these are walked.
#include "common.cuh"

MLXB_DEFINE_LAST_ERROR()

__device__ __forceinline__ int run_length_2d(const int* __restrict__ token_req, int t0, int t1, int r) {
  int n = 0;
  const int nt = blockDim.x * blockDim.y, tid = threadIdx.y * blockDim.x + threadIdx.x;
  for (int base = t0; base < t1; base += nt) {
    const int t = base + tid;
    n += __syncthreads_count(t < t1 && token_req[t] == r);
  }
  return n;
}

constexpr int RG_CHANNELS = 16;    // channels of a block
constexpr int RG_LEN = 8;          // rows of a piece
constexpr int RG_PIECES = 32;      // pieces a block walks at a time

template <typename T>
__device__ __forceinline__ float gelu_y(float v);
template <>
__device__ __forceinline__ float gelu_y<float>(float v) { return gelu_new_f(v); }
template <>
__device__ __forceinline__ float gelu_y<__nv_bfloat16>(float v) { return gelu_new_fast(v); }

__device__ __forceinline__ float sigmoid_f(float v) { return 1.f / (1.f + expf(-v)); }

// Columns of the gates' products: channel c of block b = c / n, j = c % n: pr at b * 2n + j, pi at b * 2n + n + j.
// Requests that bring a single row are left to rglru_row_kernel.
template <typename T>
__global__ void __launch_bounds__(RG_CHANNELS * RG_PIECES)
rglru_scan_kernel(const float* gates, int ldg, const float* __restrict__ br, const float* __restrict__ bi,
                  const float* __restrict__ cdecay, const T* u, int ldu, const T* y, int ldy, float* state,
                  const int* __restrict__ slots, const int* __restrict__ token_req,
                  const int* __restrict__ req_first_token, T* __restrict__ out, int ldo, int W, int n_block) {
  __shared__ float2 chain[2][RG_PIECES][RG_CHANNELS];      // (A, B) of a piece; two sets, so that one barrier a round is enough
  const int lane = threadIdx.x, piece = threadIdx.y;
  const int c = blockIdx.x * RG_CHANNELS + lane, r = blockIdx.y;
  const int t0 = req_first_token[r], t1 = req_first_token[r + 1];
  const int n = run_length_2d(token_req, t0, t1, r);
  if (n < 2) return;
  const bool valid = c < W;
  const int cc = valid ? c : 0;
  const int blk = cc / n_block, j = cc - blk * n_block;
  const float b_r = br[cc], b_i = bi[cc], cd = cdecay[cc];
  float* sp = state + (size_t)slots[r] * W + cc;
  float carry = *sp;             // written in an earlier step: read before the wait
  pdl_wait();
  pdl_trigger();
  gates = after_wait(gates) + (size_t)blk * 2 * n_block + j;
  u = after_wait(u) + cc;
  y = after_wait(y) + cc;
  float pr[RG_LEN], pi[RG_LEN];
  T uu[RG_LEN], yy[RG_LEN];
  auto fetch = [&](int lo) {
#pragma unroll
    for (int e = 0; e < RG_LEN; ++e) {
      const size_t t = (size_t)(t0 + min(lo + e, n - 1));
      pr[e] = gates[t * ldg];
      pi[e] = gates[t * ldg + n_block];
      uu[e] = u[t * ldu];
      yy[e] = y[t * ldy];
    }
  };
  int set = 0;
  fetch(piece * RG_LEN);
  for (int base = 0; base < n; base += RG_PIECES * RG_LEN, set ^= 1) {
    const int lo = base + piece * RG_LEN;
    float a[RG_LEN], b[RG_LEN], g[RG_LEN];
    float A = 1.f, B = 0.f;
#pragma unroll
    for (int e = 0; e < RG_LEN; ++e) {
      const float x = expm1f(sigmoid_f(pr[e] + b_r) * cd);
      const bool in = lo + e < n;
      a[e] = in ? 1.f + x : 1.f;
      b[e] = in ? sqrtf(-x * (2.f + x)) * (sigmoid_f(pi[e] + b_i) * to_f(uu[e])) : 0.f;
      g[e] = gelu_y<T>(to_f(yy[e]));
      A *= a[e];
      B = fmaf(a[e], B, b[e]);
    }
    chain[set][piece][lane] = make_float2(A, B);
    const int next = lo + RG_PIECES * RG_LEN;
    if (base + RG_PIECES * RG_LEN < n) fetch(next);
    __syncthreads();
    float S = carry, s = carry;
#pragma unroll 8
    for (int p = 0; p < RG_PIECES; ++p) {
      if (p == piece) S = s;
      const float2 ab = chain[set][p][lane];
      s = fmaf(ab.x, s, ab.y);
    }
    carry = s;
#pragma unroll
    for (int e = 0; e < RG_LEN; ++e) {
      S = fmaf(a[e], S, b[e]);
      if (lo + e < n && valid) out[(size_t)(t0 + lo + e) * ldo + c] = from_f<T>(S * g[e]);
    }
  }
  if (piece == 0 && valid) *sp = carry;
}

// A single row a request: a thread per channel.
template <typename T>
__global__ void rglru_row_kernel(const float* gates, int ldg, const float* __restrict__ br, const float* __restrict__ bi,
                                 const float* __restrict__ cdecay, const T* u, int ldu, const T* y, int ldy, float* state,
                                 const int* __restrict__ slots, const int* __restrict__ token_req,
                                 const int* __restrict__ req_first_token, T* __restrict__ out, int ldo, int W, int n_block) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x, r = blockIdx.y;
  const int t0 = req_first_token[r], t1 = req_first_token[r + 1];
  if (c >= W || t0 >= t1 || token_req[t0] != r || (t0 + 1 < t1 && token_req[t0 + 1] == r)) return;
  const int blk = c / n_block, j = c - blk * n_block;
  const float b_r = br[c], b_i = bi[c], cd = cdecay[c];
  float* sp = state + (size_t)slots[r] * W + c;
  const float S0 = *sp;
  pdl_wait();
  pdl_trigger();
  gates = after_wait(gates);
  u = after_wait(u);
  y = after_wait(y);
  const float* gp = gates + (size_t)t0 * ldg + (size_t)blk * 2 * n_block + j;
  const float pr = gp[0], pi = gp[n_block], uu = to_f(u[(size_t)t0 * ldu + c]), yy = to_f(y[(size_t)t0 * ldy + c]);
  const float la = sigmoid_f(pr + b_r) * cd;
  const float x = expm1f(la);
  const float S = fmaf(1.f + x, S0, sqrtf(-x * (2.f + x)) * (sigmoid_f(pi + b_i) * uu));
  *sp = S;
  out[(size_t)t0 * ldo + c] = from_f<T>(S * gelu_y<T>(yy));
}

// gates: float32 [n_tokens, 2W] at row stride ldg (per block of n_block channels: n_block products of the recurrence
// gate, then n_block of the input gate); br, bi, cdecay: float32 [W]; u, y, out: [n_tokens, W] of `dtype`; state:
// float32 [slots, W]; singles / portions: whether any request brings one row / several rows (a launch each).
MLXB_EXPORT int mlxb_rglru_scan(int dtype, const float* gates, int ldg, const float* br, const float* bi,
                                const float* cdecay, const void* u, int ldu, const void* y, int ldy, float* state,
                                const int* slots, const int* token_req, const int* req_first_token, void* out, int ldo,
                                int W, int n_block, int n_requests, int singles, int portions, cudaStream_t stream) {
  if (n_requests <= 0) return 0;
  if (W <= 0 || n_block <= 0 || W % n_block || ldg < 2 * W || ldu < W || ldy < W || ldo < W || n_requests > 65535)
    return mlxb_fail(MLXB_BAD_ARG, "rglru_scan: %d channels in blocks of %d, strides %d / %d / %d / %d", W, n_block, ldg, ldu,
                     ldy, ldo);
  if (dtype != MLXB_F32 && dtype != MLXB_BF16) return mlxb_fail(MLXB_BAD_DTYPE, "rglru_scan: dtype code %d", dtype);
#define RG_GO(T)                                                                                                      \
  if (portions)                                                                                                       \
    launch_pdl(rglru_scan_kernel<T>, dim3((W + RG_CHANNELS - 1) / RG_CHANNELS, n_requests), dim3(RG_CHANNELS, RG_PIECES), 0, \
               stream, gates, ldg, br, bi, cdecay, (const T*)u, ldu, (const T*)y, ldy, state, slots, token_req,       \
               req_first_token, (T*)out, ldo, W, n_block);                                                     \
  if (singles)                                                                                                        \
    launch_pdl(rglru_row_kernel<T>, dim3((W + 127) / 128, n_requests), dim3(128), 0, stream, gates, ldg, br, bi, cdecay, \
               (const T*)u, ldu, (const T*)y, ldy, state, slots, token_req, req_first_token, (T*)out, ldo, W, n_block)
  if (dtype == MLXB_F32) { RG_GO(float); }
  else { RG_GO(__nv_bfloat16); }
#undef RG_GO
  return mlxb_check_launch("rglru_scan");
}
