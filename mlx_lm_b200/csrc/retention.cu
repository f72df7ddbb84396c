// Retention: linear attention with a fixed decay per head, behind a rotation of queries and keys.
//
//   q_t, k_t   the first 2 * half dimensions of a head turned by the token's position (pairs (i, i + half), angle
//              p * freq[i]), the rest as they are; k also times kscale, after the rotation;
//   S_t = decay_h S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,     S of K rows and V columns, float32.
//
// q, k and v arrive in the activation dtype (a fused projection); everything from there on is float32.  The state of a
// request lives in row slots[r] of a float32 pool ([slots, H, V, K]: a head's state column by column), is read at the
// start of the run of rows a step brings for it (req_first_token[r] .., as many as carry its index in token_req) and
// written back at its end.
//
// Two forms of the same recurrence:
//   retention_scan    token by token (float32 runs, single tokens, sizes the other form does not take).  A thread holds
//                     16 consecutive rows of a state column in registers; the NS threads of a column are neighbouring
//                     lanes and add their partial sums by shuffles; 16 tokens at a time are staged in shared memory.
//   retention_chunks  runs of rows in tiles of up to 128 tokens on tensor cores (bfloat16 runs), see below.
#include "common.cuh"

MLXB_DEFINE_LAST_ERROR()

// Rows t0 .. t1-1 that belong to request r (they come first in the range).  Every thread of the block calls it.
__device__ __forceinline__ int run_length(const int* __restrict__ token_req, int t0, int t1, int r) {
  int n = 0;
  for (int base = t0; base < t1; base += blockDim.x) {
    const int t = base + threadIdx.x;
    n += __syncthreads_count(t < t1 && token_req[t] == r);
  }
  return n;
}

constexpr int RT_NPT = 16;     // rows of a state column a thread holds
constexpr int RT_SEG = 20;     // floats between the staged runs of 16 rows (keeps 16-byte loads of neighbouring lanes apart)
constexpr int RT_CHUNK = 16;   // tokens staged at a time

// Runs longer than max_run rows are passed over (0: none are).
template <typename T, int NS>
__global__ void __launch_bounds__(256)
retention_scan_kernel(const T* qkv, int ld, int q_off, int k_off, int v_off, const float* __restrict__ freq, int half,
                      float kscale, const float* __restrict__ decay, float* state, const int* __restrict__ slots,
                      const int* __restrict__ positions, const int* __restrict__ token_req,
                      const int* __restrict__ req_first_token, float* __restrict__ o, int ldo, int H, int K, int V, int VB,
                      int max_run) {
  extern __shared__ __align__(16) float rt_sm[];
  constexpr int NP = NS * RT_SEG;
  float* sq = rt_sm;                       // [CHUNK][NP]
  float* sk = sq + RT_CHUNK * NP;          // [CHUNK][NP]
  float* sv = sk + RT_CHUNK * NP;          // [CHUNK][VB]
  const int h = blockIdx.x, r = blockIdx.y, vb = blockIdx.z;
  const int tid = threadIdx.x, nthreads = blockDim.x;
  const int s = tid % NS, vl = tid / NS, v = vb * VB + vl;
  const bool valid = v < V;
  const int t0 = req_first_token[r], t1 = req_first_token[r + 1];
  const int n = run_length(token_req, t0, t1, r);
  if (n == 0 || (max_run > 0 && n > max_run)) return;
  const float g = decay[h];
  // this thread's column; the kernel that wrote it ran in an earlier step, so it is asked for before the wait
  float* st = state + (((size_t)slots[r] * H + h) * V + (valid ? v : 0)) * K;
  float S[RT_NPT];
  const bool vec_state = K % 4 == 0;
  if (vec_state) {
#pragma unroll
    for (int i = 0; i < RT_NPT; i += 4) {
      const int kk = s * RT_NPT + i;
      float4 q = make_float4(0.f, 0.f, 0.f, 0.f);
      if (valid && kk < K) q = *reinterpret_cast<const float4*>(st + kk);
      S[i] = q.x; S[i + 1] = q.y; S[i + 2] = q.z; S[i + 3] = q.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < RT_NPT; ++i) {
      const int kk = s * RT_NPT + i;
      S[i] = (valid && kk < K) ? st[kk] : 0.f;
    }
  }
  for (int e = tid; e < 2 * RT_CHUNK * NP; e += nthreads) sq[e] = 0.f;     // rows beyond K stay zero
  const int items = K - half;      // a pair, or a dimension that does not turn
  pdl_wait();
  pdl_trigger();
  qkv = after_wait(qkv);
  auto place = [](int kk) { return (kk / RT_NPT) * RT_SEG + (kk % RT_NPT); };
  for (int c0 = 0; c0 < n; c0 += RT_CHUNK) {
    const int nc = min(RT_CHUNK, n - c0);
    __syncthreads();
    for (int e = tid; e < nc * items; e += nthreads) {
      const int tok = e / items, i = e - tok * items;
      const size_t row = (size_t)(t0 + c0 + tok);
      const T* qp = qkv + row * ld + q_off + (size_t)h * K;
      const T* kp = qkv + row * ld + k_off + (size_t)h * K;
      float* tq = sq + tok * NP;
      float* tk = sk + tok * NP;
      if (i < half) {
        float sn, cs;
        sincosf((float)positions[row] * freq[i], &sn, &cs);
        const float q0 = to_f(qp[i]), q1 = to_f(qp[i + half]), k0 = to_f(kp[i]), k1 = to_f(kp[i + half]);
        tq[place(i)] = q0 * cs - q1 * sn;
        tq[place(i + half)] = q1 * cs + q0 * sn;
        tk[place(i)] = (k0 * cs - k1 * sn) * kscale;
        tk[place(i + half)] = (k1 * cs + k0 * sn) * kscale;
      } else {
        tq[place(i + half)] = to_f(qp[i + half]);
        tk[place(i + half)] = to_f(kp[i + half]) * kscale;
      }
    }
    for (int e = tid; e < nc * VB; e += nthreads) {
      const int tok = e / VB, c = e - tok * VB;
      sv[e] = vb * VB + c < V ? to_f(qkv[(size_t)(t0 + c0 + tok) * ld + v_off + (size_t)h * V + vb * VB + c]) : 0.f;
    }
    __syncthreads();
#pragma unroll 4
    for (int tok = 0; tok < nc; ++tok) {
      const float* pq = sq + tok * NP + s * RT_SEG;
      const float* pk = sk + tok * NP + s * RT_SEG;
      const float vv = sv[tok * VB + vl];
      float a = 0.f;
#pragma unroll
      for (int i = 0; i < RT_NPT; i += 4) {
        const float4 q4 = *reinterpret_cast<const float4*>(pq + i);
        const float4 k4 = *reinterpret_cast<const float4*>(pk + i);
        S[i] = fmaf(g, S[i], k4.x * vv);
        S[i + 1] = fmaf(g, S[i + 1], k4.y * vv);
        S[i + 2] = fmaf(g, S[i + 2], k4.z * vv);
        S[i + 3] = fmaf(g, S[i + 3], k4.w * vv);
        a = fmaf(q4.x, S[i], a);
        a = fmaf(q4.y, S[i + 1], a);
        a = fmaf(q4.z, S[i + 2], a);
        a = fmaf(q4.w, S[i + 3], a);
      }
#pragma unroll
      for (int off = NS / 2; off > 0; off >>= 1) a += __shfl_xor_sync(0xffffffffu, a, off);
      if (s == 0 && valid) o[(size_t)(t0 + c0 + tok) * ldo + (size_t)h * V + v] = a;
    }
  }
  if (!valid) return;
  if (vec_state) {
#pragma unroll
    for (int i = 0; i < RT_NPT; i += 4) {
      const int kk = s * RT_NPT + i;
      if (kk < K) *reinterpret_cast<float4*>(st + kk) = make_float4(S[i], S[i + 1], S[i + 2], S[i + 3]);
    }
  } else {
#pragma unroll
    for (int i = 0; i < RT_NPT; ++i) {
      const int kk = s * RT_NPT + i;
      if (kk < K) st[kk] = S[i];
    }
  }
}

// qkv: [n_tokens, .] (activation dtype) holding q and k (H*K columns each from q_off / k_off) and v (H*V columns from
// v_off); freq: float32 [half] (2 * half <= K) or null; decay: float32 [H]; state: float32 [slots, H, V, K]; o: float32
// [n_tokens, H*V] at row stride ldo; max_run: runs of more rows are left to retention_chunks (0: all are taken here).
MLXB_EXPORT int mlxb_retention_scan(int dtype, const void* qkv, int ld, int q_off, int k_off, int v_off,
                                    const float* freq, int half, float kscale, const float* decay, float* state,
                                    const int* slots, const int* positions, const int* token_req,
                                    const int* req_first_token, float* o, int ldo, int H, int K, int V, int n_requests,
                                    int max_run, cudaStream_t stream) {
  if (n_requests <= 0) return 0;
  if (H <= 0 || K <= 0 || V <= 0 || K > 32 * RT_NPT || n_requests > 65535 || half < 0 || 2 * half > K || (half && !freq) ||
      ldo < H * V || (((uintptr_t)state) & 15))
    return mlxb_fail(MLXB_BAD_ARG, "retention_scan: %d heads with states of %d x %d (at most %d rows), %d pairs turned", H, K, V,
                     32 * RT_NPT, half);
  int NS = 1;
  while (NS * RT_NPT < K) NS *= 2;
  // few (request, head) pairs: the columns of a pair over several blocks, never below two warps a block
  const long long pairs = (long long)H * n_requests;
  const int sms = mlxb_sm_count();
  int threads = 2 * pairs >= sms ? 256 : (4 * pairs >= sms ? 128 : 64);
  if (threads < 2 * NS) threads = 2 * NS;
  const int unit = NS >= 32 ? 1 : 32 / NS;                 // columns that make a whole warp
  int VB = threads / NS;
  const int v_up = (V + unit - 1) / unit * unit;
  if (VB > v_up) VB = v_up;
  threads = VB * NS;
  const dim3 grid(H, n_requests, (V + VB - 1) / VB);
  const size_t smem = sizeof(float) * ((size_t)RT_CHUNK * (2 * NS * RT_SEG + VB));
#define RT_GO(T, N)                                                                                                  \
  if (smem > 48 * 1024) {                                                                                            \
    const cudaError_t e = cudaFuncSetAttribute(retention_scan_kernel<T, N>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    if (e != cudaSuccess) return mlxb_fail((int)e, "retention_scan: %zu bytes of shared memory: %s", smem, cudaGetErrorString(e)); \
  }                                                                                                                  \
  launch_pdl(retention_scan_kernel<T, N>, grid, dim3(threads), smem, stream, (const T*)qkv, ld, q_off, k_off, v_off, freq, \
             half, kscale, decay, state, slots, positions, token_req, req_first_token, o, ldo, H, K, V, VB, max_run)
#define RT_NS(T)                  \
  switch (NS) {                   \
    case 1: RT_GO(T, 1); break;   \
    case 2: RT_GO(T, 2); break;   \
    case 4: RT_GO(T, 4); break;   \
    case 8: RT_GO(T, 8); break;   \
    case 16: RT_GO(T, 16); break; \
    default: RT_GO(T, 32); break; \
  }
  if (dtype == MLXB_F32) { RT_NS(float) }
  else if (dtype == MLXB_BF16) { RT_NS(__nv_bfloat16) }
  else return mlxb_fail(MLXB_BAD_DTYPE, "retention_scan: dtype code %d", dtype);
#undef RT_NS
#undef RT_GO
  return mlxb_check_launch("retention_scan");
}
