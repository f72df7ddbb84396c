// Matrix memory with exponential gates (the mLSTM of xLSTM).  Per head, with q_t times qscale, k_t of K and v_t of V values,
// the logarithms of an input and a forget gate
//   i_t = cap tanh(zi_t / cap),   f_t = logsigmoid(cap tanh(zf_t / cap)),
// and a running maximum m (0 at the start of a sequence, like S and n):
//   m_t = max(f_t + m_(t-1), i_t)
//   S_t = exp(f_t + m_(t-1) - m_t) S_(t-1) + exp(i_t - m_t) k_t v_t^T,   n_t likewise with k_t alone
//   o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6)
// then every head's o divided by its root mean square, times a weight per column and sigmoid(gate).
//
// n is one more column of the state, whose v is 1: a head's state is V + 1 columns of K rows, float32, column by column
// ([slots, H, V + 1, K]); the maxima are a state of their own ([slots, H]).  q, k and v arrive in the activation dtype (a
// fused projection), the gates' inputs in float32; everything from there on is float32.
//
//   mlstm_gates         the maxima along every request's run of rows and, per (row, head), the four numbers the recurrence
//                       needs (below), by scans over tiles of rows.
//   mlstm_gates_single  the same for steps in which every request brings one row, with the gates' projections in it.
//   mlstm_scan          token by token (float32 runs, single rows, sizes the tiles do not take): o undivided, and n . q.
//   mlstm_chunks        runs of rows in tiles of up to 128 on tensor cores (bfloat16 runs).
//   mlstm_finish        the division, the heads' norm, weight and gate, where the tiles have not done it.
//
// The four numbers of a row, with b_t the sum of f and M the maximum m before the row's tile:
//   rows that go token by token   (exp(f + m_(t-1) - m_t), exp(i - m_t), -, exp(-m_t))
//   rows of a tile                (a_t, A_t, exp(M - A_t), exp(-m_t))   a_t = i_t - b_t,  A_t = max(M, max_(s<=t) a_s)
// so that m_t = b_t + A_t and the weight of row s in row t is exp(a_s - A_t).
#include "common.cuh"
#include "mma_bf16.cuh"
#include "recurrent_tiles.cuh"

MLXB_DEFINE_LAST_ERROR()

constexpr float ML_TINY = 1e-6f;

__device__ __forceinline__ float ml_cap(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float ml_logsigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
// 1 / (max(|n.q|, exp(-m)) + tiny)
__device__ __forceinline__ float ml_divisor(float den, float em) { return 1.f / (fmaxf(fabsf(den), em) + ML_TINY); }

constexpr int MLG_PER = 4;       // rows of a tile a lane takes at most: tiles of up to 128 rows
constexpr int MLG_WARPS = 8;     // tiles a block walks at a time

__global__ void __launch_bounds__(32 * MLG_WARPS)
mlstm_gates_kernel(const float* raw, int ld, int f_off, float cap, float* m_state, const int* __restrict__ slots,
                   const int* __restrict__ token_req, const int* __restrict__ req_first_token, float4* __restrict__ coef, int H,
                   int tile_rows, int tiled) {
  __shared__ float s_b[MLG_WARPS], s_a[MLG_WARPS];
  const int h = blockIdx.x, r = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  const int t0 = req_first_token[r], t1 = req_first_token[r + 1];
  const int n = run_length(token_req, t0, t1, r);
  if (n == 0) return;
  const bool tile_form = tiled && n > 1;
  float* mp = m_state + (size_t)slots[r] * H + h;
  float m_run = *mp;               // written by an earlier step
  const int per = (tile_rows + 31) / 32;
  pdl_wait();
  pdl_trigger();
  raw = after_wait(raw);
  for (int base = 0; base < n; base += nw * tile_rows) {
    const int row0 = base + warp * tile_rows;
    float f[MLG_PER], i[MLG_PER], b[MLG_PER], a[MLG_PER];
    float sum = 0.f, top = -INFINITY;
#pragma unroll
    for (int j = 0; j < MLG_PER; ++j) {
      const int lr = lane * per + j;
      const bool valid = j < per && lr < tile_rows && row0 + lr < n;
      f[j] = 0.f;
      i[j] = -INFINITY;
      if (valid) {
        const float* z = raw + (size_t)(t0 + row0 + lr) * ld + h;
        i[j] = ml_cap(z[0], cap);
        f[j] = ml_logsigmoid(ml_cap(z[f_off], cap));
      }
      sum += f[j];
      b[j] = sum;
    }
    float before = sum;             // inclusive over the lanes, then what lies before this lane
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, before, o);
      if (lane >= o) before += x;
    }
    const float tile_b = __shfl_sync(0xffffffffu, before, 31);
    before = __shfl_up_sync(0xffffffffu, before, 1);
    if (lane == 0) before = 0.f;
#pragma unroll
    for (int j = 0; j < MLG_PER; ++j) {
      b[j] += before;
      a[j] = i[j] - b[j];
      top = fmaxf(top, a[j]);
    }
    float upto = top;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, upto, o);
      if (lane >= o) upto = fmaxf(upto, x);
    }
    const float tile_a = __shfl_sync(0xffffffffu, upto, 31);
    upto = __shfl_up_sync(0xffffffffu, upto, 1);
    if (lane == 0) upto = -INFINITY;
    if (lane == 0) {
      s_b[warp] = tile_b;
      s_a[warp] = tile_a;
    }
    __syncthreads();
    float m_in = 0.f, m = m_run;    // a tile without rows leaves m as it is
    for (int w = 0; w < nw; ++w) {
      if (w == warp) m_in = m;
      m = s_b[w] + fmaxf(m, s_a[w]);
    }
    m_run = m;
    float mt[MLG_PER], A[MLG_PER];
#pragma unroll
    for (int j = 0; j < MLG_PER; ++j) {
      upto = fmaxf(upto, a[j]);
      A[j] = fmaxf(m_in, upto);
      mt[j] = b[j] + A[j];
    }
    float m_prev = __shfl_up_sync(0xffffffffu, mt[MLG_PER - 1], 1);
    if (lane == 0) m_prev = m_in;
#pragma unroll
    for (int j = 0; j < MLG_PER; ++j) {
      const int lr = lane * per + j;
      if (j < per && lr < tile_rows && row0 + lr < n)
        coef[(size_t)(t0 + row0 + lr) * H + h] = tile_form ? make_float4(a[j], A[j], expf(m_in - A[j]), expf(-mt[j]))
                                                           : make_float4(expf(f[j] + m_prev - mt[j]), expf(i[j] - mt[j]), 0.f, expf(-mt[j]));
      m_prev = mt[j];
    }
    __syncthreads();
  }
  if (threadIdx.x == 0) *mp = m_run;
}

// raw: float32 [n_tokens, .] at row stride ld, head h's input gate in column h, its forget gate in column f_off + h; m_state:
// float32 [slots, H]; coef: [n_tokens, H] groups of four floats.  tiled: runs of several rows get the numbers of the tiled form
// (tiles of tile_rows rows counted from the run's first), else every run those of the token-by-token form.
MLXB_EXPORT int mlxb_mlstm_gates(const float* raw, int ld, int f_off, float cap, float* m_state, const int* slots,
                                 const int* token_req, const int* req_first_token, float* coef, int H, int tile_rows, int tiled,
                                 int n_requests, cudaStream_t stream) {
  if (n_requests <= 0) return 0;
  if (H <= 0 || n_requests > 65535 || tile_rows <= 0 || tile_rows > 32 * MLG_PER || !(cap > 0.f) || ld < f_off + H || f_off < H ||
      (((uintptr_t)coef) & 15))
    return mlxb_fail(MLXB_BAD_ARG, "mlstm_gates: %d heads, cap %g, tiles of %d rows", H, (double)cap, tile_rows);
  launch_pdl(mlstm_gates_kernel, dim3(H, n_requests), dim3(32 * MLG_WARPS), 0, stream, raw, ld, f_off, cap, m_state, slots,
             token_req, req_first_token, (float4*)coef, H, tile_rows, tiled);
  return mlxb_check_launch("mlstm_gates");
}

// A warp per (request, head): the two gates' products over the row, then one step of the maximum.
template <typename T, bool VEC>
__global__ void __launch_bounds__(128)
mlstm_gates_single_kernel(const T* x, int ldx, const T* __restrict__ w, const float* __restrict__ bias, float cap, float* m_state,
                          const int* __restrict__ slots, const int* __restrict__ token_req,
                          const int* __restrict__ req_first_token, float4* __restrict__ coef, int H, int D, int n_requests,
                          int n_tokens) {
  const int lane = threadIdx.x & 31;
  const int item = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const bool live = item < n_requests * H;
  const int r = live ? item / H : 0, h = live ? item - r * H : 0;
  const T* wi = w + (size_t)h * D;
  const T* wf = w + (size_t)(H + h) * D;
  const int t = req_first_token[r];
  const bool go = live && t < n_tokens && token_req[t] == r;
  float* mp = m_state + (size_t)slots[r] * H + h;
  const float m0 = go ? *mp : 0.f;            // written by an earlier step
  if (go)
    for (int c = lane * 64; c < D; c += 32 * 64) {
      asm volatile("prefetch.global.L2 [%0];" ::"l"(wi + c));
      asm volatile("prefetch.global.L2 [%0];" ::"l"(wf + c));
    }
  pdl_wait();
  pdl_trigger();
  x = after_wait(x);
  if (!go) return;
  const T* xr = x + (size_t)t * ldx;
  float zi = 0.f, zf = 0.f;
  if (VEC) {
    constexpr int N = 16 / sizeof(T);
    for (int c = lane * N; c < D; c += 32 * N) {
      const uint4 ux = *reinterpret_cast<const uint4*>(xr + c), ui = *reinterpret_cast<const uint4*>(wi + c),
                  uf = *reinterpret_cast<const uint4*>(wf + c);
      const T *px = reinterpret_cast<const T*>(&ux), *pi = reinterpret_cast<const T*>(&ui), *pf = reinterpret_cast<const T*>(&uf);
#pragma unroll
      for (int e = 0; e < N; ++e) {
        zi = fmaf(to_f(px[e]), to_f(pi[e]), zi);
        zf = fmaf(to_f(px[e]), to_f(pf[e]), zf);
      }
    }
  } else {
    for (int c = lane; c < D; c += 32) {
      zi = fmaf(to_f(xr[c]), to_f(wi[c]), zi);
      zf = fmaf(to_f(xr[c]), to_f(wf[c]), zf);
    }
  }
  zi = warp_sum(zi) + bias[h];
  zf = warp_sum(zf) + bias[H + h];
  const float i = ml_cap(zi, cap), f = ml_logsigmoid(ml_cap(zf, cap));
  const float m = fmaxf(f + m0, i);
  if (lane == 0) {
    coef[(size_t)t * H + h] = make_float4(expf(f + m0 - m), expf(i - m), 0.f, expf(-m));
    *mp = m;
  }
}

// x: `dtype` [n_tokens, D] at row stride ldx; w: `dtype` [2 H, D], the input gates' rows first; bias: float32 [2 H].  For steps
// in which no request brings more than one row.
MLXB_EXPORT int mlxb_mlstm_gates_single(int dtype, const void* x, int ldx, const void* w, const float* bias, float cap,
                                        float* m_state, const int* slots, const int* token_req, const int* req_first_token,
                                        float* coef, int H, int D, int n_requests, int n_tokens, cudaStream_t stream) {
  if (n_requests <= 0) return 0;
  if (H <= 0 || D <= 0 || !(cap > 0.f) || ldx < D || (((uintptr_t)coef) & 15))
    return mlxb_fail(MLXB_BAD_ARG, "mlstm_gates: %d heads over rows of %d, cap %g", H, D, (double)cap);
  const dim3 grid((unsigned)(((long long)n_requests * H + 3) / 4)), block(128);
  const int n = dtype == MLXB_F32 ? 4 : 8;
  const bool vec = D % n == 0 && ldx % n == 0 && (((uintptr_t)x | (uintptr_t)w) & 15) == 0;
#define ML_SINGLE(T, VECV)                                                                                              \
  launch_pdl(mlstm_gates_single_kernel<T, VECV>, grid, block, 0, stream, (const T*)x, ldx, (const T*)w, bias, cap, m_state, \
             slots, token_req, req_first_token, (float4*)coef, H, D, n_requests, n_tokens)
  if (dtype == MLXB_F32) { if (vec) ML_SINGLE(float, true); else ML_SINGLE(float, false); }
  else if (dtype == MLXB_BF16) { if (vec) ML_SINGLE(__nv_bfloat16, true); else ML_SINGLE(__nv_bfloat16, false); }
  else return mlxb_fail(MLXB_BAD_DTYPE, "mlstm_gates: dtype code %d", dtype);
#undef ML_SINGLE
  return mlxb_check_launch("mlstm_gates (single rows)");
}

// ---------------------------------------------------------------- token by token
// A thread holds 16 consecutive rows of a state column in registers; the NS threads of a column are neighbouring lanes and
// add their partial sums by shuffles; 16 tokens at a time are staged in shared memory.  Column V is n.

constexpr int ML_NPT = 16;     // rows of a state column a thread holds
constexpr int ML_SEG = 20;     // floats between the staged runs of 16 rows (keeps 16-byte loads of neighbouring lanes apart)
constexpr int ML_CHUNK = 16;   // tokens staged at a time

// Runs longer than max_run rows are passed over (0: none are).
template <typename T, int NS>
__global__ void __launch_bounds__(256)
mlstm_scan_kernel(const T* qkv, int ld, int q_off, int k_off, int v_off, float qscale, const float4* coef, float* state,
                  const int* __restrict__ slots, const int* __restrict__ token_req, const int* __restrict__ req_first_token,
                  float* __restrict__ o, int ldo, float* __restrict__ den, int H, int K, int V, int VB, int max_run) {
  extern __shared__ __align__(16) float ml_sm[];
  constexpr int NP = NS * ML_SEG;
  float* sq = ml_sm;                       // [CHUNK][NP]
  float* sk = sq + ML_CHUNK * NP;          // [CHUNK][NP]
  float* sv = sk + ML_CHUNK * NP;          // [CHUNK][VB]
  __shared__ float2 sc[ML_CHUNK];          // what the state keeps, what the token adds
  const int h = blockIdx.x, r = blockIdx.y, vb = blockIdx.z;
  const int tid = threadIdx.x, nthreads = blockDim.x;
  const int s = tid % NS, vl = tid / NS, v = vb * VB + vl;
  const bool valid = v <= V;
  const int t0 = req_first_token[r], t1 = req_first_token[r + 1];
  const int n = run_length(token_req, t0, t1, r);
  if (n == 0 || (max_run > 0 && n > max_run)) return;
  // this thread's column; the kernel that wrote it ran in an earlier step, so it is asked for before the wait
  float* st = state + (((size_t)slots[r] * H + h) * (V + 1) + (valid ? v : 0)) * K;
  float S[ML_NPT];
  const bool vec_state = K % 4 == 0;
#pragma unroll
  for (int i = 0; i < ML_NPT; i += 4) {
    const int kk = s * ML_NPT + i;
    if (vec_state) {
      float4 q = make_float4(0.f, 0.f, 0.f, 0.f);
      if (valid && kk < K) q = *reinterpret_cast<const float4*>(st + kk);
      S[i] = q.x; S[i + 1] = q.y; S[i + 2] = q.z; S[i + 3] = q.w;
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) S[i + e] = (valid && kk + e < K) ? st[kk + e] : 0.f;
    }
  }
  for (int e = tid; e < 2 * ML_CHUNK * NP; e += nthreads) sq[e] = 0.f;     // rows beyond K stay zero
  pdl_wait();
  pdl_trigger();
  qkv = after_wait(qkv);
  coef = after_wait(coef);
  auto place = [](int kk) { return (kk / ML_NPT) * ML_SEG + (kk % ML_NPT); };
  for (int c0 = 0; c0 < n; c0 += ML_CHUNK) {
    const int nc = min(ML_CHUNK, n - c0);
    __syncthreads();
    if (tid < nc) {
      const float4 c = coef[(size_t)(t0 + c0 + tid) * H + h];
      sc[tid] = make_float2(c.x, c.y);
    }
    for (int e = tid; e < nc * K; e += nthreads) {
      const int tok = e / K, i = e - tok * K;
      const T* row = qkv + (size_t)(t0 + c0 + tok) * ld + (size_t)h * K + i;
      sq[tok * NP + place(i)] = to_f(row[q_off]) * qscale;
      sk[tok * NP + place(i)] = to_f(row[k_off]);
    }
    for (int e = tid; e < nc * VB; e += nthreads) {
      const int tok = e / VB, c = vb * VB + e - tok * VB;
      sv[e] = c < V ? to_f(qkv[(size_t)(t0 + c0 + tok) * ld + v_off + (size_t)h * V + c]) : (c == V ? 1.f : 0.f);
    }
    __syncthreads();
#pragma unroll 4
    for (int tok = 0; tok < nc; ++tok) {
      const float* pq = sq + tok * NP + s * ML_SEG;
      const float* pk = sk + tok * NP + s * ML_SEG;
      const float2 c = sc[tok];
      const float vv = sv[tok * VB + vl] * c.y;
      float a = 0.f;
#pragma unroll
      for (int i = 0; i < ML_NPT; i += 4) {
        const float4 q4 = *reinterpret_cast<const float4*>(pq + i);
        const float4 k4 = *reinterpret_cast<const float4*>(pk + i);
        S[i] = fmaf(c.x, S[i], k4.x * vv);
        S[i + 1] = fmaf(c.x, S[i + 1], k4.y * vv);
        S[i + 2] = fmaf(c.x, S[i + 2], k4.z * vv);
        S[i + 3] = fmaf(c.x, S[i + 3], k4.w * vv);
        a = fmaf(q4.x, S[i], a);
        a = fmaf(q4.y, S[i + 1], a);
        a = fmaf(q4.z, S[i + 2], a);
        a = fmaf(q4.w, S[i + 3], a);
      }
#pragma unroll
      for (int off = NS / 2; off > 0; off >>= 1) a += __shfl_xor_sync(0xffffffffu, a, off);
      if (s == 0 && valid) {
        if (v < V) o[(size_t)(t0 + c0 + tok) * ldo + (size_t)h * V + v] = a;
        else den[(size_t)(t0 + c0 + tok) * H + h] = a;
      }
    }
  }
  if (!valid) return;
#pragma unroll
  for (int i = 0; i < ML_NPT; i += 4) {
    const int kk = s * ML_NPT + i;
    if (vec_state) {
      if (kk < K) *reinterpret_cast<float4*>(st + kk) = make_float4(S[i], S[i + 1], S[i + 2], S[i + 3]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (kk + e < K) st[kk + e] = S[i + e];
    }
  }
}

// qkv: [n_tokens, .] (activation dtype) holding q and k (H*K columns each from q_off / k_off) and v (H*V columns from v_off);
// coef: what mlstm_gates left; state: float32 [slots, H, V + 1, K]; o: float32 [n_tokens, H*V] at row stride ldo, undivided;
// den: float32 [n_tokens, H]; max_run: runs of more rows are left to mlstm_chunks (0: all are taken here).
MLXB_EXPORT int mlxb_mlstm_scan(int dtype, const void* qkv, int ld, int q_off, int k_off, int v_off, float qscale,
                                const float* coef, float* state, const int* slots, const int* token_req,
                                const int* req_first_token, float* o, int ldo, float* den, int H, int K, int V, int n_requests,
                                int max_run, cudaStream_t stream) {
  if (n_requests <= 0) return 0;
  if (H <= 0 || K <= 0 || V <= 0 || K > 32 * ML_NPT || n_requests > 65535 || ldo < H * V || (((uintptr_t)state | (uintptr_t)coef) & 15))
    return mlxb_fail(MLXB_BAD_ARG, "mlstm_scan: %d heads with states of %d x %d (at most %d rows)", H, K, V, 32 * ML_NPT);
  int NS = 1;
  while (NS * ML_NPT < K) NS *= 2;
  // few (request, head) pairs: the columns of a pair over several blocks, never below two warps a block
  const long long pairs = (long long)H * n_requests;
  const int sms = mlxb_sm_count();
  int threads = 2 * pairs >= sms ? 256 : (4 * pairs >= sms ? 128 : 64);
  if (threads < 2 * NS) threads = 2 * NS;
  const int unit = NS >= 32 ? 1 : 32 / NS;                 // columns that make a whole warp
  int VB = threads / NS;
  const int v_up = (V + 1 + unit - 1) / unit * unit;
  if (VB > v_up) VB = v_up;
  threads = VB * NS;
  const dim3 grid(H, n_requests, (V + 1 + VB - 1) / VB);
  const size_t smem = sizeof(float) * ((size_t)ML_CHUNK * (2 * NS * ML_SEG + VB));
#define ML_GO(T, N)                                                                                                  \
  if (smem > 48 * 1024) {                                                                                            \
    const cudaError_t e = cudaFuncSetAttribute(mlstm_scan_kernel<T, N>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    if (e != cudaSuccess) return mlxb_fail((int)e, "mlstm_scan: %zu bytes of shared memory: %s", smem, cudaGetErrorString(e)); \
  }                                                                                                                  \
  launch_pdl(mlstm_scan_kernel<T, N>, grid, dim3(threads), smem, stream, (const T*)qkv, ld, q_off, k_off, v_off, qscale,   \
             (const float4*)coef, state, slots, token_req, req_first_token, o, ldo, den, H, K, V, VB, max_run)
#define ML_NS(T)                  \
  switch (NS) {                   \
    case 1: ML_GO(T, 1); break;   \
    case 2: ML_GO(T, 2); break;   \
    case 4: ML_GO(T, 4); break;   \
    case 8: ML_GO(T, 8); break;   \
    case 16: ML_GO(T, 16); break; \
    default: ML_GO(T, 32); break; \
  }
  if (dtype == MLXB_F32) { ML_NS(float) }
  else if (dtype == MLXB_BF16) { ML_NS(__nv_bfloat16) }
  else return mlxb_fail(MLXB_BAD_DTYPE, "mlstm_scan: dtype code %d", dtype);
#undef ML_NS
#undef ML_GO
  return mlxb_check_launch("mlstm_scan");
}

// One warp per (row, head): o divided by max(|n.q|, exp(-m)) + tiny and by its root mean square, times weight and sigmoid(gate).
template <typename T>
__global__ void __launch_bounds__(128)
mlstm_finish_kernel(const float* o, int ldo, const float* den, const float4* coef, const float* __restrict__ w, const T* gate,
                    int ldg, const int* __restrict__ token_req, float eps, T* __restrict__ y, int ldy, int H, int V, int n_tokens) {
  const int lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (item >= (long long)n_tokens * H) return;
  const int t = (int)(item / H), h = (int)(item - (long long)t * H);
  if (token_req[t] < 0) return;
  constexpr int NR = 8;             // columns a lane keeps in registers: heads of up to 256 columns are read once
  float wr[NR];
#pragma unroll
  for (int j = 0; j < NR; ++j) wr[j] = lane + 32 * j < V ? w[h * V + lane + 32 * j] : 0.f;
  pdl_wait();
  pdl_trigger();
  o = after_wait(o);
  den = after_wait(den);
  coef = after_wait(coef);
  gate = after_wait(gate);
  const float* op = o + (size_t)t * ldo + (size_t)h * V;
  const T* gp = gate + (size_t)t * ldg + (size_t)h * V;
  T* yp = y + (size_t)t * ldy + (size_t)h * V;
  const float s = ml_divisor(den[item], coef[item].w);
  float v[NR], g[NR];
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int c = lane + 32 * j;
    v[j] = g[j] = 0.f;
    if (c < V) {
      v[j] = op[c] * s;
      g[j] = to_f(gp[c]);
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < NR; ++j) ss = fmaf(v[j], v[j], ss);
  for (int c = lane + 32 * NR; c < V; c += 32) { const float x = op[c] * s; ss = fmaf(x, x, ss); }
  const float rinv = 1.f / sqrtf(warp_sum(ss) / (float)V + eps);
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int c = lane + 32 * j;
    if (c < V) yp[c] = from_f<T>(v[j] * rinv * wr[j] / (1.f + expf(-g[j])));
  }
  for (int c = lane + 32 * NR; c < V; c += 32)
    yp[c] = from_f<T>(op[c] * s * rinv * w[h * V + c] / (1.f + expf(-to_f(gp[c]))));
}

// o, den, coef: as mlstm_scan and mlstm_gates leave them; w: float32 [H*V]; gate, y: `dtype` [n_tokens, H*V].
MLXB_EXPORT int mlxb_mlstm_finish(int dtype, const float* o, int ldo, const float* den, const float* coef, const float* w,
                                  const void* gate, int ldg, const int* token_req, float eps, void* y, int ldy, int H, int V,
                                  int n_tokens, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (H <= 0 || V <= 0 || ldo < H * V || ldg < H * V || ldy < H * V)
    return mlxb_fail(MLXB_BAD_ARG, "mlstm_finish: %d heads of %d columns, strides %d / %d / %d", H, V, ldo, ldg, ldy);
  const dim3 grid((unsigned)(((long long)n_tokens * H + 3) / 4)), block(128);
  if (dtype == MLXB_F32)
    launch_pdl(mlstm_finish_kernel<float>, grid, block, 0, stream, o, ldo, den, (const float4*)coef, w, (const float*)gate, ldg,
               token_req, eps, (float*)y, ldy, H, V, n_tokens);
  else if (dtype == MLXB_BF16)
    launch_pdl(mlstm_finish_kernel<__nv_bfloat16>, grid, block, 0, stream, o, ldo, den, (const float4*)coef, w,
               (const __nv_bfloat16*)gate, ldg, token_req, eps, (__nv_bfloat16*)y, ldy, H, V, n_tokens);
  else
    return mlxb_fail(MLXB_BAD_DTYPE, "mlstm_finish: dtype code %d", dtype);
  return mlxb_check_launch("mlstm_finish");
}

// ---------------------------------------------------------------- runs of rows on tensor cores
//
// A run is cut into the tiles the attention kernels use (first token row, rows, request, first position).  With i, j counted
// inside a tile of n rows, S (n among its columns) the state before it and a, A, c = exp(M - A) the tile's numbers:
//   o_i = c_i S^T q_i + sum_(j <= i) exp(a_j - A_i) (q_i . k_j) v_j         (undivided; n . q the same with v = 1)
//   S'  = c_last S + sum_j exp(a_j - A_last) k_j v_j^T
// in three launches, the tiles side by side in the first and the last:
//   chunk_states   every tile's own contribution to S', float32, to scratch memory;
//   chunk_pass     along each run: the contribution gives way to the state before the tile, the last state is stored;
//   chunk_out      every tile's outputs from the state before it and its own rows.
// A tile's scratch slot follows from where its run lies among the step's rows: req_first_token[r] / tile + r + number of
// the tile in its run (slots of different runs never meet: a run of m tiles spans more than (m - 1) * tile rows).
//
// q, k and v are bfloat16 as they come.  What is float32 in the recurrence (states, weighted keys, weighted scores) enters the
// products as two bfloat16 halves (hi + lo); sums and states are float32.

constexpr int MC_ROWS = 128;       // rows of a tile at most
constexpr int MC_KB = 64;          // rows of k and v staged at a time in chunk_out

struct MlArgs {
  const __nv_bfloat16* qkv;
  int ld, q_off, k_off, v_off;
  float qscale;
  const float4* coef;       // [n_tokens, H]
  const int* tiles;         // [n_tiles, 4]: first token row, rows, request, first position
  int tile_rows;
  const int* req_first_token;
  const int* req_first_position;
  float* scratch;           // [slots, H, V + 1, K]
  int H, K, V;
};

__device__ __forceinline__ size_t ml_slot(const MlArgs& p, int r, int pos) {
  return (size_t)(p.req_first_token[r] / p.tile_rows + r + (pos - p.req_first_position[r]) / p.tile_rows);
}

// A tile's contribution to the state, columns v0 .. v0 + 63 of one head (and n, by the first of the head's blocks): warp w
// takes v rows 16 (w % 4) .. and half of the K columns.
template <int KP, bool VEC>
__global__ void __launch_bounds__(256, KP <= 64 ? 3 : 1)
mlstm_chunk_states_kernel(const MlArgs p) {
  extern __shared__ __align__(16) unsigned char mc_raw[];
  constexpr int LK = KP + 8, LV = 64 + 8;
  __nv_bfloat16* kh = reinterpret_cast<__nv_bfloat16*>(mc_raw);     // [128][LK]
  __nv_bfloat16* kl = kh + MC_ROWS * LK;
  __nv_bfloat16* sv = kl + MC_ROWS * LK;                            // [128][LV]
  __shared__ float sw[MC_ROWS];                                     // exp(a_j - A_last)
  const int h = blockIdx.y, v0 = blockIdx.z * 64;
  const int t0 = p.tiles[blockIdx.x * 4], n = p.tiles[blockIdx.x * 4 + 1], r = p.tiles[blockIdx.x * 4 + 2],
            pos = p.tiles[blockIdx.x * 4 + 3];
  if (n <= 0) return;
  pdl_wait();
  pdl_trigger();
  const __nv_bfloat16* qkv = after_wait(p.qkv);
  const float4* coef = after_wait(p.coef) + (size_t)t0 * p.H + h;
  const int rows = (n + 15) & ~15;
  if (threadIdx.x < rows)
    sw[threadIdx.x] = threadIdx.x < n ? expf(coef[(size_t)threadIdx.x * p.H].x - coef[(size_t)(n - 1) * p.H].y) : 0.f;
  stage_values<VEC>(qkv + p.v_off + (size_t)h * p.V, p.ld, t0, n, rows, v0, p.V, 64, sv, LV);
  __syncthreads();
  // the keys times their weights as two halves
  {
    const __nv_bfloat16* src = qkv + p.k_off + (size_t)h * p.K;
    if (VEC) {
      constexpr int PER = KP / 8;
#pragma unroll 4
      for (int e = threadIdx.x; e < rows * PER; e += blockDim.x) {
        const int tok = e / PER, c = (e - tok * PER) * 8;
        uint4 u = make_uint4(0u, 0u, 0u, 0u), hi, lo;
        if (tok < n && c < p.K) u = *reinterpret_cast<const uint4*>(src + (size_t)(t0 + tok) * p.ld + c);
        const float w = sw[tok];
        float x[8];
        unpack8(u, x);
        mb_split2(x[0] * w, x[1] * w, hi.x, lo.x);
        mb_split2(x[2] * w, x[3] * w, hi.y, lo.y);
        mb_split2(x[4] * w, x[5] * w, hi.z, lo.z);
        mb_split2(x[6] * w, x[7] * w, hi.w, lo.w);
        *reinterpret_cast<uint4*>(kh + tok * LK + c) = hi;
        *reinterpret_cast<uint4*>(kl + tok * LK + c) = lo;
      }
    } else {
      for (int e = threadIdx.x; e < rows * KP; e += blockDim.x) {
        const int tok = e / KP, c = e - tok * KP;
        const float x = (tok < n && c < p.K) ? to_f(src[(size_t)(t0 + tok) * p.ld + c]) * sw[tok] : 0.f;
        mb_split(x, kh[tok * LK + c], kl[tok * LK + c]);
      }
    }
  }
  __syncthreads();
  float* out = p.scratch + (ml_slot(p, r, pos) * p.H + h) * (size_t)(p.V + 1) * p.K;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int vr = (warp & 3) * 16, c0 = (warp >> 2) * (KP / 2);
  constexpr int NT = KP / 16;          // 8-column tiles of this warp's half
  float acc[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
  const unsigned va = mb_smem(sv + ((lane & 7) + ((lane >> 4) & 1) * 8) * LV + vr + ((lane >> 3) & 1) * 8);
  const unsigned ka = mb_smem(kh + (lane & 15) * LK + c0 + (lane >> 4) * 8);
  const unsigned kb = mb_smem(kl + (lane & 15) * LK + c0 + (lane >> 4) * 8);
  for (int j = 0; j < rows; j += 16) {
    unsigned a[4];
    mb_ldmatrix_trans(a, va + j * LV * 2);
#pragma unroll
    for (int q = 0; q < NT / 2; ++q) {
      unsigned bh[4], bl[4];
      mb_ldmatrix_trans(bh, ka + (j * LK + q * 16) * 2);
      mb_ldmatrix_trans(bl, kb + (j * LK + q * 16) * 2);
      mb_mma(acc[2 * q], a, bh[0], bh[1]);
      mb_mma(acc[2 * q + 1], a, bh[2], bh[3]);
      mb_mma(acc[2 * q], a, bl[0], bl[1]);
      mb_mma(acc[2 * q + 1], a, bl[2], bl[3]);
    }
  }
  const int g = lane >> 2, t4 = lane & 3;
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    const int c = c0 + j * 8 + t4 * 2;
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int v = v0 + vr + g + hf * 8;
      if (v >= p.V || c >= p.K) continue;
      float* o = out + (size_t)v * p.K + c;
      if (VEC) {
        *reinterpret_cast<float2*>(o) = make_float2(acc[j][2 * hf], acc[j][2 * hf + 1]);
      } else {
        o[0] = acc[j][2 * hf];
        if (c + 1 < p.K) o[1] = acc[j][2 * hf + 1];
      }
    }
  }
  if (v0 == 0)
    for (int c = threadIdx.x; c < p.K; c += blockDim.x) {
      float x0 = 0.f, x1 = 0.f;
#pragma unroll 8
      for (int j = 0; j < rows; j += 2) {
        x0 += __bfloat162float(kh[j * LK + c]) + __bfloat162float(kl[j * LK + c]);
        x1 += __bfloat162float(kh[(j + 1) * LK + c]) + __bfloat162float(kl[(j + 1) * LK + c]);
      }
      out[(size_t)p.V * p.K + c] = x0 + x1;
    }
}

// Along a run: scratch gets the state before each tile, the state what it is after the last.  A thread per VEC elements.
template <int VEC>
__global__ void mlstm_chunk_pass_kernel(float* scratch, float* state, const float4* coef, const int* __restrict__ slots,
                                        const int* __restrict__ token_req, const int* __restrict__ req_first_token, int H, int KV,
                                        int tile_rows) {
  const int r = blockIdx.z, h = blockIdx.y;
  const int t0 = req_first_token[r], t1 = req_first_token[r + 1];
  const int n = run_length(token_req, t0, t1, r);
  const int e = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (n < 2 || e >= KV) return;      // (runs of one row go through mlstm_scan)
  float S[VEC], U[VEC], N[VEC];
  float* sp = state + ((size_t)slots[r] * H + h) * KV + e;
  auto load = [](const float* q, float (&v)[VEC]) {
    if (VEC == 4) {
      const float4 f = *reinterpret_cast<const float4*>(q);
      v[0] = f.x; v[VEC > 1 ? 1 : 0] = f.y; v[VEC > 2 ? 2 : 0] = f.z; v[VEC > 3 ? 3 : 0] = f.w;
    } else {
      v[0] = *q;
    }
  };
  auto store = [](float* q, const float (&v)[VEC]) {
    if (VEC == 4) *reinterpret_cast<float4*>(q) = make_float4(v[0], v[VEC > 1 ? 1 : 0], v[VEC > 2 ? 2 : 0], v[VEC > 3 ? 3 : 0]);
    else *q = v[0];
  };
  load(sp, S);                       // written by an earlier step
  pdl_wait();
  pdl_trigger();
  scratch = after_wait(scratch);
  coef = after_wait(coef) + h;
  const int m = (n + tile_rows - 1) / tile_rows;
  const size_t step = (size_t)H * KV;
  float* up = scratch + ((size_t)(t0 / tile_rows + r) * H + h) * KV + e;
  auto kept = [&](int c) { return coef[(size_t)(t0 + min(n, (c + 1) * tile_rows) - 1) * H].z; };
  load(up, N);
  float gn = kept(0);
  for (int c = 0; c < m; ++c) {
    const float g = gn;
#pragma unroll
    for (int i = 0; i < VEC; ++i) U[i] = N[i];
    if (c + 1 < m) {
      load(up + step, N);
      gn = kept(c + 1);
    }
    store(up, S);
#pragma unroll
    for (int i = 0; i < VEC; ++i) S[i] = fmaf(g, S[i], U[i]);
    up += step;
  }
  store(sp, S);
}

// A tile's outputs, VS columns of one head from v0 on: warp w takes rows 16 w .. 16 w + 15.  With `gate` (VS covers the
// head's V columns) a row is divided, normed, weighted and gated, and the result is bfloat16; else o (undivided) and n . q are
// left in float32.
template <int KP, int VS, bool VEC>
__global__ void __launch_bounds__(256)
mlstm_chunk_out_kernel(const MlArgs p, float* __restrict__ o, int ldo, float* __restrict__ den, const __nv_bfloat16* gate, int ldg,
                       const float* __restrict__ norm_w, __nv_bfloat16* __restrict__ gated, int ldy, float eps) {
  extern __shared__ __align__(16) unsigned char mc_raw[];
  constexpr int LK = KP + 8, LV = VS + 8;
  constexpr int BROWS = VS + 16 > MC_KB ? VS + 16 : MC_KB;          // rows of the buffer that holds S^T and n, then blocks of k
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(mc_raw);     // [128][LK]
  __nv_bfloat16* bh = sq + MC_ROWS * LK;                            // [BROWS][LK]
  __nv_bfloat16* bl = bh + BROWS * LK;
  __nv_bfloat16* sv = bl + BROWS * LK;                              // [MC_KB][LV]
  __shared__ float4 sc[MC_ROWS];
  const int h = blockIdx.y, v0 = blockIdx.z * VS;
  const int t0 = p.tiles[blockIdx.x * 4], n = p.tiles[blockIdx.x * 4 + 1], r = p.tiles[blockIdx.x * 4 + 2],
            pos = p.tiles[blockIdx.x * 4 + 3];
  if (n <= 0) return;
  pdl_wait();
  pdl_trigger();
  const __nv_bfloat16* qkv = after_wait(p.qkv);
  gate = after_wait(gate);
  const float4* coef = after_wait(p.coef) + (size_t)t0 * p.H + h;
  const float* st = after_wait(p.scratch) + (ml_slot(p, r, pos) * p.H + h) * (size_t)(p.V + 1) * p.K;
  const int rows = (n + 15) & ~15;
  if (threadIdx.x < MC_ROWS)      // rows beyond the tile's weigh nothing
    sc[threadIdx.x] = threadIdx.x < n ? coef[(size_t)threadIdx.x * p.H] : make_float4(-INFINITY, 0.f, 0.f, 1.f);
  stage_values<VEC>(qkv + p.q_off + (size_t)h * p.K, p.ld, t0, n, rows, 0, p.K, KP, sq, LK);
  // S^T: rows v, columns k; row VS: n
  auto source = [&](int v) { return v < VS ? (v0 + v < p.V ? v0 + v : -1) : (v == VS ? p.V : -1); };
  if (VEC) {
#pragma unroll 8
    for (int e = threadIdx.x; e < (VS + 16) * (KP / 4); e += blockDim.x) {
      const int v = e / (KP / 4), c = (e - v * (KP / 4)) * 4, sr = source(v);
      float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
      if (sr >= 0 && c < p.K) f = *reinterpret_cast<const float4*>(st + (size_t)sr * p.K + c);
      uint2 hi, lo;
      mb_split2(f.x, f.y, hi.x, lo.x);
      mb_split2(f.z, f.w, hi.y, lo.y);
      *reinterpret_cast<uint2*>(bh + v * LK + c) = hi;
      *reinterpret_cast<uint2*>(bl + v * LK + c) = lo;
    }
  } else {
    for (int e = threadIdx.x; e < (VS + 16) * KP; e += blockDim.x) {
      const int v = e / KP, c = e - v * KP, sr = source(v);
      mb_split((sr >= 0 && c < p.K) ? st[(size_t)sr * p.K + c] : 0.f, bh[v * LK + c], bl[v * LK + c]);
    }
  }
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t4 = lane & 3;
  const int i0 = warp * 16;                     // this warp's rows of the tile
  const bool live = i0 < rows;
  constexpr int NT = VS / 8;
  float acc[NT][4], accn[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
  const unsigned qa = mb_smem(sq + (i0 + (lane & 15)) * LK + (lane >> 4) * 8);
  const unsigned ba = mb_smem(bh + ((lane & 7) + ((lane >> 4) & 1) * 8) * LK + ((lane >> 3) & 1) * 8);
  const unsigned bb = mb_smem(bl + ((lane & 7) + ((lane >> 4) & 1) * 8) * LK + ((lane >> 3) & 1) * 8);
  float A[2] = {0.f, 0.f}, rs[2] = {0.f, 0.f};
  if (live) {
    // c_i S^T q_i
#pragma unroll
    for (int ks = 0; ks < KP; ks += 16) {
      unsigned a[4], xh[4], xl[4];
      mb_ldmatrix(a, qa + ks * 2);
#pragma unroll
      for (int j = 0; j < NT / 2; ++j) {
        mb_ldmatrix(xh, ba + (j * 16 * LK + ks) * 2);
        mb_ldmatrix(xl, bb + (j * 16 * LK + ks) * 2);
        mb_mma(acc[2 * j], a, xh[0], xh[1]);
        mb_mma(acc[2 * j + 1], a, xh[2], xh[3]);
        mb_mma(acc[2 * j], a, xl[0], xl[1]);
        mb_mma(acc[2 * j + 1], a, xl[2], xl[3]);
      }
      mb_ldmatrix(xh, ba + (VS * LK + ks) * 2);
      mb_ldmatrix(xl, bb + (VS * LK + ks) * 2);
      mb_mma(accn, a, xh[0], xh[1]);
      mb_mma(accn, a, xl[0], xl[1]);
    }
    const float4 c0 = sc[i0 + g], c1 = sc[i0 + g + 8];
    A[0] = c0.y;
    A[1] = c1.y;
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      acc[j][0] *= c0.z;
      acc[j][1] *= c0.z;
      acc[j][2] *= c1.z;
      acc[j][3] *= c1.z;
    }
    if (t4 == 0) {          // column 0 of the extra tile
      rs[0] = accn[0] * c0.z;
      rs[1] = accn[2] * c1.z;
    }
  }
  for (int kb = 0; kb < n; kb += MC_KB) {
    const int nk = min(MC_KB, n - kb), krows = (nk + 15) & ~15;
    __syncthreads();
    stage_values<VEC>(qkv + p.k_off + (size_t)h * p.K, p.ld, t0 + kb, nk, krows, 0, p.K, KP, bh, LK);
    stage_values<VEC>(qkv + p.v_off + (size_t)h * p.V, p.ld, t0 + kb, nk, krows, v0, p.V, VS, sv, LV);
    __syncthreads();
    if (!live) continue;
    // sixteen keys at a time, up to the warp's last row
    for (int k0 = 0; k0 < krows && kb + k0 <= i0 + 15; k0 += 16) {
      float s[2][4];
#pragma unroll
      for (int e = 0; e < 4; ++e) s[0][e] = s[1][e] = 0.f;
#pragma unroll
      for (int ks = 0; ks < KP; ks += 16) {
        unsigned a[4], x[4];
        mb_ldmatrix(a, qa + ks * 2);
        mb_ldmatrix(x, ba + (k0 * LK + ks) * 2);
        mb_mma(s[0], a, x[0], x[1]);
        mb_mma(s[1], a, x[2], x[3]);
      }
      unsigned ph[4], pl[4];
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        const int j = kb + k0 + q * 8 + t4 * 2;              // this thread's two keys, counted in the tile
        const float a0 = sc[j].x, a1 = sc[j + 1].x;
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
          const int d = i0 + g + hf * 8 - j;                 // rows from the key to the query
          const float x = d >= 0 ? s[q][2 * hf] * expf(a0 - A[hf]) : 0.f, y = d >= 1 ? s[q][2 * hf + 1] * expf(a1 - A[hf]) : 0.f;
          rs[hf] += x + y;
          mb_split2(x, y, ph[q * 2 + hf], pl[q * 2 + hf]);
        }
      }
#pragma unroll
      for (int j = 0; j < NT / 2; ++j) {
        unsigned b[4];
        mb_ldmatrix_trans(b, mb_smem(sv + (k0 + (lane & 15)) * LV + j * 16 + (lane >> 4) * 8));
        mb_mma(acc[2 * j], ph, b[0], b[1]);
        mb_mma(acc[2 * j + 1], ph, b[2], b[3]);
        mb_mma(acc[2 * j], pl, b[0], b[1]);
        mb_mma(acc[2 * j + 1], pl, b[2], b[3]);
      }
    }
  }
  if (!live) return;
#pragma unroll
  for (int hf = 0; hf < 2; ++hf) {
    const int i = i0 + g + hf * 8;
    float nq = rs[hf], ss = 0.f;
    nq += __shfl_xor_sync(0xffffffffu, nq, 1);
    nq += __shfl_xor_sync(0xffffffffu, nq, 2);
    nq *= p.qscale;
    if (gate) {      // (columns beyond V are zeros)
#pragma unroll
      for (int j = 0; j < NT; ++j) ss = fmaf(acc[j][2 * hf], acc[j][2 * hf], fmaf(acc[j][2 * hf + 1], acc[j][2 * hf + 1], ss));
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
    }
    if (i >= n) continue;
    const size_t row = (size_t)(t0 + i);
    float f = p.qscale;
    if (gate) {
      f *= ml_divisor(nq, sc[i].w);
      f /= sqrtf(f * f * ss / (float)p.V + eps);
    } else if (v0 == 0 && t4 == 0) {
      den[row * p.H + h] = nq;
    }
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int v = v0 + j * 8 + t4 * 2;
      if (v >= p.V) continue;
      float x = acc[j][2 * hf] * f, y = acc[j][2 * hf + 1] * f;
      const size_t c = (size_t)h * p.V + v;
      if (gate) {
        const __nv_bfloat16* gp = gate + row * ldg + c;
        __nv_bfloat16* yp = gated + row * ldy + c;
        if (VEC) {
          const __nv_bfloat162 gv = *reinterpret_cast<const __nv_bfloat162*>(gp);
          const float2 wv = *reinterpret_cast<const float2*>(norm_w + c);
          x = x * wv.x / (1.f + expf(-__bfloat162float(gv.x)));
          y = y * wv.y / (1.f + expf(-__bfloat162float(gv.y)));
          *reinterpret_cast<__nv_bfloat162*>(yp) = __floats2bfloat162_rn(x, y);
        } else {
          yp[0] = from_f<__nv_bfloat16>(x * norm_w[c] / (1.f + expf(-to_f(gp[0]))));
          if (v + 1 < p.V) yp[1] = from_f<__nv_bfloat16>(y * norm_w[c + 1] / (1.f + expf(-to_f(gp[1]))));
        }
      } else {
        float* op = o + row * ldo + c;
        if (VEC) {
          *reinterpret_cast<float2*>(op) = make_float2(x, y);
        } else {
          op[0] = x;
          if (v + 1 < p.V) op[1] = y;
        }
      }
    }
  }
}

// Whether mlstm_chunks takes heads of K x V, and whether it can divide, norm and gate them itself.
MLXB_EXPORT int mlxb_mlstm_chunks_supported(int K, int V) { return K >= 1 && K <= 256 && V >= 1; }
MLXB_EXPORT int mlxb_mlstm_chunks_gated(int K, int V) { return V <= (K <= 128 ? 128 : 64); }

// The runs of two rows and more of a step, bfloat16.  qkv, offsets, qscale, coef (the tiled form), state: as in mlstm_scan; tiles:
// int32 [n_tiles, 4] = (first token row, rows up to tile_rows, request, first position); scratch: float32, (n_tokens / tile_rows +
// n_requests + 1) * H * (V + 1) * K; o, den: as in mlstm_scan, or, with gate, norm_w (float32 [H*V]) and gated (bfloat16), the
// finished rows in gated.
MLXB_EXPORT int mlxb_mlstm_chunks(const void* qkv, int ld, int q_off, int k_off, int v_off, float qscale, const float* coef,
                                  float* state, const int* slots, const int* token_req, const int* req_first_token,
                                  const int* req_first_position, const int* tiles, int n_tiles, int tile_rows, float* scratch,
                                  float* o, int ldo, float* den, const void* gate, int ldg, const float* norm_w, void* gated, int ldy,
                                  float eps, int H, int K, int V, int n_requests, cudaStream_t stream) {
  if (n_tiles <= 0 || n_requests <= 0) return 0;
  if (H <= 0 || H > 65535 || !mlxb_mlstm_chunks_supported(K, V) || n_requests > 65535 || tile_rows <= 0 || tile_rows > MC_ROWS ||
      (gate && (!gated || !norm_w || !mlxb_mlstm_chunks_gated(K, V) || ldg < H * V || ldy < H * V)) ||
      (!gate && (!o || !den || ldo < H * V)) || (((uintptr_t)coef) & 15))
    return mlxb_fail(MLXB_BAD_ARG, "mlstm_chunks: %d heads of %d x %d, tiles of %d rows", H, K, V, tile_rows);
  const MlArgs p = {(const __nv_bfloat16*)qkv, ld, q_off, k_off, v_off, qscale, (const float4*)coef, tiles, tile_rows,
                    req_first_token, req_first_position, scratch, H, K, V};
  const bool vec = K % 8 == 0 && V % 8 == 0 && ld % 8 == 0 && q_off % 8 == 0 && k_off % 8 == 0 && v_off % 8 == 0 &&
                   (((uintptr_t)qkv | (uintptr_t)scratch | (uintptr_t)state) & 15) == 0 && (!o || (ldo % 2 == 0 && ((uintptr_t)o & 7) == 0)) &&
                   (!gate || (ldg % 2 == 0 && ldy % 2 == 0 && (((uintptr_t)gate | (uintptr_t)gated) & 3) == 0 && ((uintptr_t)norm_w & 7) == 0));
  const int KP = K <= 32 ? 32 : (K <= 64 ? 64 : (K <= 128 ? 128 : 256));
  const int VS = V > 64 && KP <= 128 ? 128 : 64;
  cudaError_t e = cudaSuccess;
#define MC_BY_K(GO)                                                             \
  switch (KP) {                                                                 \
    case 32: if (vec) GO(32, true); else GO(32, false); break;                  \
    case 64: if (vec) GO(64, true); else GO(64, false); break;                  \
    case 128: if (vec) GO(128, true); else GO(128, false); break;               \
    default: if (vec) GO(256, true); else GO(256, false); break;                \
  }
  {
    const dim3 grid(n_tiles, H, (V + 63) / 64), block(256);
    const size_t smem = sizeof(__nv_bfloat16) * (2 * (size_t)MC_ROWS * (KP + 8) + (size_t)MC_ROWS * 72);
#define MC_STATES(KPV, VECV)                                                                                           \
  do {                                                                                                                 \
    e = cudaFuncSetAttribute(mlstm_chunk_states_kernel<KPV, VECV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    if (e == cudaSuccess) e = launch_pdl(mlstm_chunk_states_kernel<KPV, VECV>, grid, block, smem, stream, p);          \
  } while (0)
    MC_BY_K(MC_STATES)
#undef MC_STATES
    if (e != cudaSuccess) return mlxb_fail((int)e, "mlstm_chunk_states: %s", cudaGetErrorString(e));
  }
  {
    const int KV = K * (V + 1);
    const bool vec4 = K % 4 == 0 && (((uintptr_t)scratch | (uintptr_t)state) & 15) == 0;
    const int per = vec4 ? 4 : 1;
    const dim3 grid((KV + 256 * per - 1) / (256 * per), H, n_requests), block(256);
    if (vec4)
      launch_pdl(mlstm_chunk_pass_kernel<4>, grid, block, 0, stream, scratch, state, (const float4*)coef, slots, token_req,
                 req_first_token, H, KV, tile_rows);
    else
      launch_pdl(mlstm_chunk_pass_kernel<1>, grid, block, 0, stream, scratch, state, (const float4*)coef, slots, token_req,
                 req_first_token, H, KV, tile_rows);
    if (int c = mlxb_check_launch("mlstm_chunk_pass")) return c;
  }
  {
    const dim3 grid(n_tiles, H, (V + VS - 1) / VS), block(256);
    const int brows = VS + 16 > MC_KB ? VS + 16 : MC_KB;
    const size_t smem = sizeof(__nv_bfloat16) * ((size_t)MC_ROWS * (KP + 8) + 2 * (size_t)brows * (KP + 8) + (size_t)MC_KB * (VS + 8));
#define MC_OUT_VS(KPV, VSV, VECV)                                                                                      \
  do {                                                                                                                 \
    e = cudaFuncSetAttribute(mlstm_chunk_out_kernel<KPV, VSV, VECV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    if (e == cudaSuccess)                                                                                              \
      e = launch_pdl(mlstm_chunk_out_kernel<KPV, VSV, VECV>, grid, block, smem, stream, p, o, ldo, den,                \
                     (const __nv_bfloat16*)gate, ldg, norm_w, (__nv_bfloat16*)gated, ldy, eps);                        \
  } while (0)
#define MC_OUT(KPV, VECV)                                               \
  do {                                                                  \
    if (KPV <= 128 && VS == 128) MC_OUT_VS((KPV <= 128 ? KPV : 128), 128, VECV); \
    else MC_OUT_VS(KPV, 64, VECV);                                      \
  } while (0)
    MC_BY_K(MC_OUT)
#undef MC_OUT
#undef MC_OUT_VS
    if (e != cudaSuccess) return mlxb_fail((int)e, "mlstm_chunk_out: %s", cudaGetErrorString(e));
  }
#undef MC_BY_K
  return mlxb_check_launch("mlstm_chunks");
}
