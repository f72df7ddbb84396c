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
#include "mma_bf16.cuh"
#include "recurrent_tiles.cuh"

MLXB_DEFINE_LAST_ERROR()

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

// ---------------------------------------------------------------- runs of rows on tensor cores
//
// A run is cut into the tiles the attention kernels use (up to 128 rows: first token row, rows, request, first position).
// With i, j counted inside a tile of n rows and S the state before it:
//   o_i = decay^(i+1) S^T q_i + sum_(j <= i) decay^(i-j) (q_i . k_j) v_j
//   S'  = decay^n S + sum_j decay^(n-1-j) k_j v_j^T
// so three launches do the work of the recurrence, the tiles side by side in the first and the last:
//   chunk_states   every tile's own contribution sum_j decay^(n-1-j) k_j v_j^T, float32, to scratch memory;
//   chunk_pass     along each run: the contribution gives way to the state before the tile, the last state is stored;
//   chunk_out      every tile's outputs from the state before it and its own rows.
// A tile's scratch slot follows from where its run lies among the step's rows: req_first_token[r] / tile + r + number of
// the tile in its run (slots of different runs never meet: a run of m tiles spans more than (m - 1) * tile rows).
//
// The products run on bfloat16 tensor cores, but nothing that is float32 in the recurrence is rounded to bfloat16: the
// turned queries and keys, the states, the decayed keys and the decayed scores enter as two bfloat16 halves (hi + lo), and
// the three products hi hi + hi lo + lo hi (two where the other operand is v, which is bfloat16 as it comes) keep about
// sixteen bits of every factor; sums and the states themselves are float32.  Powers of the decays come from a table made
// in float64 when the weights are bound.

constexpr int RC_ROWS = 128;       // rows of a tile at most
constexpr int RC_KB = 64;          // rows of k and v staged at a time in chunk_out

// Rows row0 .. row0 + n - 1 of one head's q or k (K columns from src) turned by their positions pos0 + row, times `scale` and,
// with `fall`, times fall[n_tile - 1 - row] (the decay to the end of the tile), as hi / lo halves into [rows, lds]; rows
// from n on and columns from K on are zeros.
template <bool VEC>
__device__ __forceinline__ void stage_turned(const __nv_bfloat16* src, int ld, int row0, int n, int rows, int pos0,
                                             const float* __restrict__ freq, int half, int K, int KP, float scale,
                                             const float* fall, int fall_last, __nv_bfloat16* hi, __nv_bfloat16* lo, int lds) {
  const int tid = threadIdx.x, nt = blockDim.x;
  if (VEC) {
    const int per = (K - half) / 4;      // four neighbouring pairs, or four dimensions that do not turn
    constexpr int UN = 4;                // items whose loads are in flight together
    for (int e0 = tid; e0 < rows * per; e0 += UN * nt) {
      uint2 ua[UN], ub[UN];
#pragma unroll
      for (int x = 0; x < UN; ++x) {
        const int e = e0 + x * nt, tok = e / per, i = (e - tok * per) * 4;
        ua[x] = ub[x] = make_uint2(0u, 0u);
        if (tok < n) {                   // (an item beyond the last has a row beyond n)
          const __nv_bfloat16* rp = src + (size_t)(row0 + tok) * ld;
          ub[x] = *reinterpret_cast<const uint2*>(rp + i + half);
          if (i < half) ua[x] = *reinterpret_cast<const uint2*>(rp + i);
        }
      }
#pragma unroll
      for (int x = 0; x < UN; ++x) {
        const int e = e0 + x * nt;
        if (e >= rows * per) break;
        const int tok = e / per, i = (e - tok * per) * 4;
        __nv_bfloat16* ph = hi + tok * lds;
        __nv_bfloat16* pl = lo + tok * lds;
        const float f = fall ? (tok < n ? scale * fall[fall_last - tok] : 0.f) : scale;
        const float v1[4] = {__uint_as_float(ub[x].x << 16), __uint_as_float(ub[x].x & 0xffff0000u),
                             __uint_as_float(ub[x].y << 16), __uint_as_float(ub[x].y & 0xffff0000u)};
        float b[4];
        uint2 h, l;
        if (i < half) {
          const float v0[4] = {__uint_as_float(ua[x].x << 16), __uint_as_float(ua[x].x & 0xffff0000u),
                               __uint_as_float(ua[x].y << 16), __uint_as_float(ua[x].y & 0xffff0000u)};
          const float fp = (float)(pos0 + tok);
          float a[4];
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            float sn, cs;
            sincosf(fp * freq[i + q], &sn, &cs);
            a[q] = (v0[q] * cs - v1[q] * sn) * f;
            b[q] = (v1[q] * cs + v0[q] * sn) * f;
          }
          mb_split2(a[0], a[1], h.x, l.x);
          mb_split2(a[2], a[3], h.y, l.y);
          *reinterpret_cast<uint2*>(ph + i) = h;
          *reinterpret_cast<uint2*>(pl + i) = l;
        } else {
#pragma unroll
          for (int q = 0; q < 4; ++q) b[q] = v1[q] * f;
        }
        mb_split2(b[0], b[1], h.x, l.x);
        mb_split2(b[2], b[3], h.y, l.y);
        *reinterpret_cast<uint2*>(ph + i + half) = h;
        *reinterpret_cast<uint2*>(pl + i + half) = l;
      }
    }
  } else {
    const int per = K - half;
    for (int e = tid; e < rows * per; e += nt) {
      const int tok = e / per, i = e - tok * per;
      float a = 0.f, b = 0.f;
      if (tok < n) {
        const __nv_bfloat16* rp = src + (size_t)(row0 + tok) * ld;
        const float f = fall ? scale * fall[fall_last - tok] : scale;
        const float v1 = to_f(rp[i + half]);
        b = v1 * f;
        if (i < half) {
          const float v0 = to_f(rp[i]);
          float sn, cs;
          sincosf((float)(pos0 + tok) * freq[i], &sn, &cs);
          a = (v0 * cs - v1 * sn) * f;
          b = (v1 * cs + v0 * sn) * f;
        }
      }
      mb_split(b, hi[tok * lds + i + half], lo[tok * lds + i + half]);
      if (i < half) mb_split(a, hi[tok * lds + i], lo[tok * lds + i]);
    }
  }
  const int pad = KP - K;
  for (int e = tid; e < rows * pad; e += nt) {
    const int tok = e / pad, c = K + e - tok * pad;
    hi[tok * lds + c] = lo[tok * lds + c] = __float2bfloat16_rn(0.f);
  }
}

struct ChunkArgs {
  const __nv_bfloat16* qkv;
  int ld, q_off, k_off, v_off;
  const float* freq;
  int half;
  float kscale;
  const float* powers;      // [H, RC_ROWS + 1]: decay^0 .. decay^128
  const int* tiles;         // [n_tiles, 4]: first token row, rows, request, first position
  int tile_rows;
  const int* req_first_token;
  const int* req_first_position;
  float* scratch;           // [slots, H, V, K]
  int H, K, V;
};

__device__ __forceinline__ size_t chunk_slot(const ChunkArgs& p, int r, int pos) {
  return (size_t)(p.req_first_token[r] / p.tile_rows + r + (pos - p.req_first_position[r]) / p.tile_rows);
}

// A tile's contribution to the state, columns v0 .. v0 + 63 of one head: warp w takes v rows 16 (w % 4) .. and half of
// the K columns.
template <int KP, bool VEC>
__global__ void __launch_bounds__(256, KP <= 64 ? 3 : 1)
retention_chunk_states_kernel(const ChunkArgs p) {
  extern __shared__ __align__(16) unsigned char rc_raw[];
  constexpr int LK = KP + 8, LV = 64 + 8;
  __nv_bfloat16* kh = reinterpret_cast<__nv_bfloat16*>(rc_raw);     // [128][LK]
  __nv_bfloat16* kl = kh + RC_ROWS * LK;
  __nv_bfloat16* sv = kl + RC_ROWS * LK;                            // [128][LV]
  const int h = blockIdx.y, v0 = blockIdx.z * 64;
  const int t0 = p.tiles[blockIdx.x * 4], n = p.tiles[blockIdx.x * 4 + 1], r = p.tiles[blockIdx.x * 4 + 2],
            pos = p.tiles[blockIdx.x * 4 + 3];
  if (n <= 0) return;
  pdl_wait();
  pdl_trigger();
  const __nv_bfloat16* qkv = after_wait(p.qkv);
  const int rows = (n + 15) & ~15;
  stage_turned<VEC>(qkv + p.k_off + (size_t)h * p.K, p.ld, t0, n, rows, pos, p.freq, p.half, p.K, KP, p.kscale,
                    p.powers + (size_t)h * (RC_ROWS + 1), n - 1, kh, kl, LK);
  stage_values<VEC>(qkv + p.v_off + (size_t)h * p.V, p.ld, t0, n, rows, v0, p.V, 64, sv, LV);
  __syncthreads();
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
  float* out = p.scratch + (chunk_slot(p, r, pos) * p.H + h) * (size_t)p.V * p.K;
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
}

// Along a run: scratch gets the state before each tile, the state what it is after the last.  A thread per VEC elements.
template <int VEC>
__global__ void retention_chunk_pass_kernel(float* scratch, float* state, const float* __restrict__ powers,
                                            const int* __restrict__ slots, const int* __restrict__ token_req,
                                            const int* __restrict__ req_first_token, int H, int KV, int tile_rows) {
  const int r = blockIdx.z, h = blockIdx.y;
  const int t0 = req_first_token[r], t1 = req_first_token[r + 1];
  const int n = run_length(token_req, t0, t1, r);
  const int e = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (n < 2 || e >= KV) return;      // (runs of one row go through retention_scan)
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
  load(sp, S);
  const float full = powers[(size_t)h * (RC_ROWS + 1) + tile_rows];
  pdl_wait();
  pdl_trigger();
  scratch = after_wait(scratch);
  const int m = (n + tile_rows - 1) / tile_rows;
  const size_t step = (size_t)H * KV;
  float* up = scratch + ((size_t)(t0 / tile_rows + r) * H + h) * KV + e;
  load(up, N);
  for (int c = 0; c < m; ++c) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) U[i] = N[i];
    if (c + 1 < m) load(up + step, N);
    store(up, S);
    const int nc = n - c * tile_rows;
    const float g = nc >= tile_rows ? full : powers[(size_t)h * (RC_ROWS + 1) + nc];
#pragma unroll
    for (int i = 0; i < VEC; ++i) S[i] = fmaf(g, S[i], U[i]);
    up += step;
  }
  store(sp, S);
}

// A tile's outputs, VS columns of one head from v0 on: warp w takes rows 16 w .. 16 w + 15.  With `gate` (VS covers the
// head's V columns) every row of the head is divided by its root mean square and multiplied by silu(gate), and the
// result is bfloat16; else o is left in float32.
template <int KP, int VS, bool VEC>
__global__ void __launch_bounds__(256)
retention_chunk_out_kernel(const ChunkArgs p, float* __restrict__ o, int ldo, const __nv_bfloat16* gate, int ldg,
                           __nv_bfloat16* __restrict__ gated, int ldy, float eps) {
  extern __shared__ __align__(16) unsigned char rc_raw[];
  constexpr int LK = KP + 8, LV = VS + 8;
  constexpr int BROWS = VS > RC_KB ? VS : RC_KB;                     // rows of the buffer that holds S^T, then blocks of k
  __nv_bfloat16* qh = reinterpret_cast<__nv_bfloat16*>(rc_raw);     // [128][LK]
  __nv_bfloat16* ql = qh + RC_ROWS * LK;
  __nv_bfloat16* bh = ql + RC_ROWS * LK;                            // [BROWS][LK]
  __nv_bfloat16* bl = bh + BROWS * LK;
  __nv_bfloat16* sv = bl + BROWS * LK;                              // [RC_KB][LV]
  __shared__ float spow[RC_ROWS + 1];
  const int h = blockIdx.y, v0 = blockIdx.z * VS;
  const int t0 = p.tiles[blockIdx.x * 4], n = p.tiles[blockIdx.x * 4 + 1], r = p.tiles[blockIdx.x * 4 + 2],
            pos = p.tiles[blockIdx.x * 4 + 3];
  if (n <= 0) return;
  for (int e = threadIdx.x; e <= RC_ROWS; e += blockDim.x) spow[e] = p.powers[(size_t)h * (RC_ROWS + 1) + e];
  pdl_wait();
  pdl_trigger();
  const __nv_bfloat16* qkv = after_wait(p.qkv);
  const float* st = after_wait(p.scratch) + (chunk_slot(p, r, pos) * p.H + h) * (size_t)p.V * p.K;
  const int rows = (n + 15) & ~15;
  stage_turned<VEC>(qkv + p.q_off + (size_t)h * p.K, p.ld, t0, n, rows, pos, p.freq, p.half, p.K, KP, 1.f, nullptr, 0, qh, ql, LK);
  // S^T: rows v, columns k
  if (VEC) {
#pragma unroll 8
    for (int e = threadIdx.x; e < VS * (KP / 4); e += blockDim.x) {
      const int v = e / (KP / 4), c = (e - v * (KP / 4)) * 4;
      float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
      if (v0 + v < p.V && c < p.K) f = *reinterpret_cast<const float4*>(st + (size_t)(v0 + v) * p.K + c);
      uint2 hi, lo;
      mb_split2(f.x, f.y, hi.x, lo.x);
      mb_split2(f.z, f.w, hi.y, lo.y);
      *reinterpret_cast<uint2*>(bh + v * LK + c) = hi;
      *reinterpret_cast<uint2*>(bl + v * LK + c) = lo;
    }
  } else {
    for (int e = threadIdx.x; e < VS * KP; e += blockDim.x) {
      const int v = e / KP, c = e - v * KP;
      mb_split((v0 + v < p.V && c < p.K) ? st[(size_t)(v0 + v) * p.K + c] : 0.f, bh[v * LK + c], bl[v * LK + c]);
    }
  }
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t4 = lane & 3;
  const int i0 = warp * 16;                     // this warp's rows of the tile
  const bool live = i0 < rows;
  constexpr int NT = VS / 8;
  float acc[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
  const unsigned qa = mb_smem(qh + (i0 + (lane & 15)) * LK + (lane >> 4) * 8);
  const unsigned qb = mb_smem(ql + (i0 + (lane & 15)) * LK + (lane >> 4) * 8);
  const unsigned ba = mb_smem(bh + ((lane & 7) + ((lane >> 4) & 1) * 8) * LK + ((lane >> 3) & 1) * 8);
  const unsigned bb = mb_smem(bl + ((lane & 7) + ((lane >> 4) & 1) * 8) * LK + ((lane >> 3) & 1) * 8);
  if (live) {
    // decay^(i+1) S^T q_i
#pragma unroll
    for (int ks = 0; ks < KP; ks += 16) {
      unsigned ah[4], al[4];
      mb_ldmatrix(ah, qa + ks * 2);
      mb_ldmatrix(al, qb + ks * 2);
#pragma unroll
      for (int j = 0; j < NT / 2; ++j) {
        unsigned xh[4], xl[4];
        mb_ldmatrix(xh, ba + (j * 16 * LK + ks) * 2);
        mb_ldmatrix(xl, bb + (j * 16 * LK + ks) * 2);
        mb_mma(acc[2 * j], ah, xh[0], xh[1]);
        mb_mma(acc[2 * j + 1], ah, xh[2], xh[3]);
        mb_mma(acc[2 * j], ah, xl[0], xl[1]);
        mb_mma(acc[2 * j + 1], ah, xl[2], xl[3]);
        mb_mma(acc[2 * j], al, xh[0], xh[1]);
        mb_mma(acc[2 * j + 1], al, xh[2], xh[3]);
      }
    }
    const float f0 = spow[i0 + g + 1], f1 = spow[i0 + g + 9];
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      acc[j][0] *= f0;
      acc[j][1] *= f0;
      acc[j][2] *= f1;
      acc[j][3] *= f1;
    }
  }
  for (int kb = 0; kb < n; kb += RC_KB) {
    const int nk = min(RC_KB, n - kb), krows = (nk + 15) & ~15;
    __syncthreads();
    stage_turned<VEC>(qkv + p.k_off + (size_t)h * p.K, p.ld, t0 + kb, nk, krows, pos + kb, p.freq, p.half, p.K, KP, p.kscale,
                      nullptr, 0, bh, bl, LK);
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
        unsigned ah[4], al[4], xh[4], xl[4];
        mb_ldmatrix(ah, qa + ks * 2);
        mb_ldmatrix(al, qb + ks * 2);
        mb_ldmatrix(xh, ba + (k0 * LK + ks) * 2);
        mb_ldmatrix(xl, bb + (k0 * LK + ks) * 2);
        mb_mma(s[0], ah, xh[0], xh[1]);
        mb_mma(s[1], ah, xh[2], xh[3]);
        mb_mma(s[0], ah, xl[0], xl[1]);
        mb_mma(s[1], ah, xl[2], xl[3]);
        mb_mma(s[0], al, xh[0], xh[1]);
        mb_mma(s[1], al, xh[2], xh[3]);
      }
      unsigned ph[4], pl[4];
#pragma unroll
      for (int q = 0; q < 2; ++q)
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
          const int d = i0 + g + hf * 8 - (kb + k0 + q * 8 + t4 * 2);      // rows from the key to the query
          const float x = d >= 0 ? s[q][2 * hf] * spow[d] : 0.f, y = d >= 1 ? s[q][2 * hf + 1] * spow[d - 1] : 0.f;
          mb_split2(x, y, ph[q * 2 + hf], pl[q * 2 + hf]);
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
    float ss = 0.f;
    if (gate) {      // (columns beyond V are zeros)
#pragma unroll
      for (int j = 0; j < NT; ++j) ss = fmaf(acc[j][2 * hf], acc[j][2 * hf], fmaf(acc[j][2 * hf + 1], acc[j][2 * hf + 1], ss));
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
    }
    if (i >= n) continue;
    const float rinv = gate ? 1.f / sqrtf(ss / (float)p.V + eps) : 1.f;
    const size_t row = (size_t)(t0 + i);
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int v = v0 + j * 8 + t4 * 2;
      if (v >= p.V) continue;
      float x = acc[j][2 * hf], y = acc[j][2 * hf + 1];
      const size_t c = (size_t)h * p.V + v;
      if (gate) {
        const __nv_bfloat16* gp = gate + row * ldg + c;
        __nv_bfloat16* yp = gated + row * ldy + c;
        if (VEC) {
          const __nv_bfloat162 gv = *reinterpret_cast<const __nv_bfloat162*>(gp);
          const float g0 = __bfloat162float(gv.x), g1 = __bfloat162float(gv.y);
          x = x * rinv * (g0 / (1.f + expf(-g0)));
          y = y * rinv * (g1 / (1.f + expf(-g1)));
          *reinterpret_cast<__nv_bfloat162*>(yp) = __floats2bfloat162_rn(x, y);
        } else {
          const float g0 = to_f(gp[0]);
          yp[0] = from_f<__nv_bfloat16>(x * rinv * (g0 / (1.f + expf(-g0))));
          if (v + 1 < p.V) {
            const float g1 = to_f(gp[1]);
            yp[1] = from_f<__nv_bfloat16>(y * rinv * (g1 / (1.f + expf(-g1))));
          }
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

// Floats of scratch memory for a step of n_tokens rows and n_requests requests.
MLXB_EXPORT long long mlxb_retention_chunks_scratch(int n_tokens, int n_requests, int tile_rows, int H, int K, int V) {
  return (long long)(n_tokens / tile_rows + n_requests + 1) * H * K * V;
}

// Whether retention_chunks takes heads of K x V.
MLXB_EXPORT int mlxb_retention_chunks_supported(int K, int V) { return K >= 1 && K <= 256 && V >= 1; }

// The runs of two rows and more of a step, bfloat16.  qkv, offsets, freq, half, kscale, state: as in retention_scan;
// powers: float32 [H, 129]; tiles: int32 [n_tiles, 4] = (first token row, rows up to tile_rows, request, first position);
// scratch: mlxb_retention_chunks_scratch floats; o: float32 [n_tokens, H*V], or, with gate and gated (bfloat16; V up to 128, or 64 with K > 128), the
// heads' rows divided by their root mean square and multiplied by silu(gate) in gated.
MLXB_EXPORT int mlxb_retention_chunks(const void* qkv, int ld, int q_off, int k_off, int v_off, const float* freq, int half,
                                      float kscale, const float* powers, float* state, const int* slots, const int* token_req,
                                      const int* req_first_token, const int* req_first_position, const int* tiles,
                                      int n_tiles, int tile_rows, float* scratch, float* o, int ldo, const void* gate, int ldg,
                                      void* gated, int ldy, float eps, int H, int K, int V, int n_requests,
                                      cudaStream_t stream) {
  if (n_tiles <= 0 || n_requests <= 0) return 0;
  if (H <= 0 || H > 65535 || !mlxb_retention_chunks_supported(K, V) || n_requests > 65535 || half < 0 || 2 * half > K ||
      (half && !freq) || tile_rows <= 0 || tile_rows > RC_ROWS || (gate && (!gated || V > (K <= 128 ? 128 : 64) || ldg < H * V || ldy < H * V)) ||
      (!gate && (!o || ldo < H * V)))
    return mlxb_fail(MLXB_BAD_ARG, "retention_chunks: %d heads of %d x %d, %d pairs turned, tiles of %d rows", H, K, V, half, tile_rows);
  const ChunkArgs p = {(const __nv_bfloat16*)qkv, ld, q_off, k_off, v_off, freq, half, kscale, powers, tiles, tile_rows,
                       req_first_token, req_first_position, scratch, H, K, V};
  const bool vec = K % 8 == 0 && V % 8 == 0 && half % 4 == 0 && ld % 8 == 0 && q_off % 8 == 0 && k_off % 8 == 0 && v_off % 8 == 0 &&
                   (((uintptr_t)qkv | (uintptr_t)scratch | (uintptr_t)state) & 15) == 0 && (!o || (ldo % 2 == 0 && ((uintptr_t)o & 7) == 0)) &&
                   (!gate || (ldg % 2 == 0 && ldy % 2 == 0 && (((uintptr_t)gate | (uintptr_t)gated) & 3) == 0));
  const int KP = K <= 32 ? 32 : (K <= 64 ? 64 : (K <= 128 ? 128 : 256));
  const int VS = V > 64 && KP <= 128 ? 128 : 64;
  cudaError_t e = cudaSuccess;
  {
    const dim3 grid(n_tiles, H, (V + 63) / 64), block(256);
    const size_t smem = sizeof(__nv_bfloat16) * (2 * (size_t)RC_ROWS * (KP + 8) + (size_t)RC_ROWS * 72);
#define RC_STATES(KPV, VECV)                                                                                           \
  do {                                                                                                                 \
    e = cudaFuncSetAttribute(retention_chunk_states_kernel<KPV, VECV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    if (e == cudaSuccess) e = launch_pdl(retention_chunk_states_kernel<KPV, VECV>, grid, block, smem, stream, p);     \
  } while (0)
#define RC_BY_K(GO)                                                             \
  switch (KP) {                                                                 \
    case 32: if (vec) GO(32, true); else GO(32, false); break;                  \
    case 64: if (vec) GO(64, true); else GO(64, false); break;                  \
    case 128: if (vec) GO(128, true); else GO(128, false); break;               \
    default: if (vec) GO(256, true); else GO(256, false); break;                \
  }
    RC_BY_K(RC_STATES)
#undef RC_STATES
    if (e != cudaSuccess) return mlxb_fail((int)e, "retention_chunk_states: %s", cudaGetErrorString(e));
  }
  {
    const int KV = K * V;
    const bool vec4 = KV % 4 == 0 && (((uintptr_t)scratch | (uintptr_t)state) & 15) == 0;
    const int per = vec4 ? 4 : 1;
    const dim3 grid((KV + 256 * per - 1) / (256 * per), H, n_requests), block(256);
    if (vec4)
      launch_pdl(retention_chunk_pass_kernel<4>, grid, block, 0, stream, scratch, state, powers, slots, token_req, req_first_token,
                 H, KV, tile_rows);
    else
      launch_pdl(retention_chunk_pass_kernel<1>, grid, block, 0, stream, scratch, state, powers, slots, token_req, req_first_token,
                 H, KV, tile_rows);
    if (int c = mlxb_check_launch("retention_chunk_pass")) return c;
  }
  {
    const dim3 grid(n_tiles, H, (V + VS - 1) / VS), block(256);
    const int brows = VS > RC_KB ? VS : RC_KB;
    const size_t smem = sizeof(__nv_bfloat16) * (2 * (size_t)RC_ROWS * (KP + 8) + 2 * (size_t)brows * (KP + 8) + (size_t)RC_KB * (VS + 8));
#define RC_OUT_VS(KPV, VSV, VECV)                                                                                      \
  do {                                                                                                                 \
    e = cudaFuncSetAttribute(retention_chunk_out_kernel<KPV, VSV, VECV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    if (e == cudaSuccess)                                                                                              \
      e = launch_pdl(retention_chunk_out_kernel<KPV, VSV, VECV>, grid, block, smem, stream, p, o, ldo,                 \
                     (const __nv_bfloat16*)gate, ldg, (__nv_bfloat16*)gated, ldy, eps);                                \
  } while (0)
#define RC_OUT(KPV, VECV)                                               \
  do {                                                                  \
    if (KPV <= 128 && VS == 128) RC_OUT_VS((KPV <= 128 ? KPV : 128), 128, VECV); \
    else RC_OUT_VS(KPV, 64, VECV);                                      \
  } while (0)
    RC_BY_K(RC_OUT)
#undef RC_OUT
#undef RC_OUT_VS
    if (e != cudaSuccess) return mlxb_fail((int)e, "retention_chunk_out: %s", cudaGetErrorString(e));
  }
#undef RC_BY_K
  return mlxb_check_launch("retention_chunks");
}
