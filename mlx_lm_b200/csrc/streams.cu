// A residual of several streams (hyper-connections), float32 rows [x_1 | .. | x_S] of S * D columns per token.
//
// streams_read    h[r] = rmsnorm(u) * w, u = sum_s in[s] x_s[row(r)]: what a sublayer reads, in the activation dtype.
// streams_update  all streams at once from the old ones and a sublayer's float32 result y:
//                   x_t <- sum_s mix[s, t] x_s + out[t] y
//                 and, in the same pass, what the sublayer that runs next reads of them: h = rmsnorm(u) * w with
//                 u = sum_t in[t] x_t of the new streams.  With S = 1 and mix = in = 1 this is an ordinary residual sum.
//
// Everything is float32; sums run over the streams in order.  One block a row; u waits in shared memory for the root
// mean square.  Rows whose token_req is negative are left alone.
#include "common.cuh"

MLXB_DEFINE_LAST_ERROR()

constexpr int ST_MAX = 16;      // streams

// VEC neighbouring columns a thread: 4 (16-byte accesses) or 1.
template <int VEC>
struct Cols;
template <>
struct Cols<1> {
  float v[1];
  __device__ void load(const float* p) { v[0] = *p; }
  __device__ void store(float* p) const { *p = v[0]; }
};
template <>
struct Cols<4> {
  float v[4];
  __device__ void load(const float* p) {
    const float4 q = *reinterpret_cast<const float4*>(p);
    v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
  }
  __device__ void store(float* p) const { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
};

template <typename TO, int VEC>
__device__ __forceinline__ void store_row(TO* p, const float (&v)[VEC]);
template <>
__device__ __forceinline__ void store_row<float, 1>(float* p, const float (&v)[1]) { *p = v[0]; }
template <>
__device__ __forceinline__ void store_row<float, 4>(float* p, const float (&v)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
template <>
__device__ __forceinline__ void store_row<__nv_bfloat16, 1>(__nv_bfloat16* p, const float (&v)[1]) { *p = __float2bfloat16_rn(v[0]); }
template <>
__device__ __forceinline__ void store_row<__nv_bfloat16, 4>(__nv_bfloat16* p, const float (&v)[4]) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&a), *reinterpret_cast<const unsigned*>(&b));
}

// Row of u in shared memory -> h, given this thread's share of the sum of squares.
template <typename TO, int VEC>
__device__ __forceinline__ void norm_row(const float* u, float ss, const float* __restrict__ w, float eps, TO* h, int D,
                                         float* red) {
  const float rinv = 1.f / sqrtf(block_sum(ss, red) / (float)D + eps);
  for (int c = threadIdx.x * VEC; c < D; c += blockDim.x * VEC) {
    Cols<VEC> a, g;
    a.load(u + c);
    g.load(w + c);
#pragma unroll
    for (int e = 0; e < VEC; ++e) a.v[e] = a.v[e] * rinv * g.v[e];
    store_row<TO, VEC>(h + c, a.v);
  }
}

template <typename TO, int SM, int VEC>
__global__ void __launch_bounds__(512) streams_read_kernel(const float* x, int ldx, const int* __restrict__ rows, int n_src_rows, int S,
                                    const float* __restrict__ in, const float* __restrict__ w, float eps,
                                    TO* __restrict__ h, int ldh, int D) {
  extern __shared__ __align__(16) float u[];
  __shared__ float red[33];
  __shared__ float s_in[SM];
  if (threadIdx.x < S) s_in[threadIdx.x] = in[threadIdx.x];
  __syncthreads();
  pdl_wait();
  pdl_trigger();
  x = after_wait(x);
  const int r = blockIdx.x;
  const int src = rows ? rows[r] : r;
  TO* ho = h + (size_t)r * ldh;
  if (src < 0 || src >= n_src_rows) {
    for (int c = threadIdx.x; c < D; c += blockDim.x) ho[c] = from_f<TO>(0.f);
    return;
  }
  const float* xr = x + (size_t)src * ldx;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < D; c += blockDim.x * VEC) {
    Cols<VEC> a[SM], acc;
#pragma unroll
    for (int s = 0; s < SM; ++s)
      if (s < S) a[s].load(xr + (size_t)s * D + c);
#pragma unroll
    for (int e = 0; e < VEC; ++e) acc.v[e] = 0.f;
#pragma unroll
    for (int s = 0; s < SM; ++s)
      if (s < S)
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc.v[e] = fmaf(s_in[s], a[s].v[e], acc.v[e]);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss = fmaf(acc.v[e], acc.v[e], ss);
    acc.store(u + c);
  }
  norm_row<TO, VEC>(u, ss, w, eps, ho, D, red);
}

template <typename TO, int SM, int VEC>
__global__ void __launch_bounds__(512) streams_update_kernel(float* x, int ldx, const float* y, int ldy, int S, const float* __restrict__ mix,
                                      const float* __restrict__ out, const int* __restrict__ token_req,
                                      const float* __restrict__ in, const float* __restrict__ w, float eps,
                                      TO* __restrict__ h, int ldh, int D) {
  extern __shared__ __align__(16) float u[];
  __shared__ float red[33];
  __shared__ float s_mix[SM * SM], s_out[SM], s_in[SM];
  for (int e = threadIdx.x; e < S * S; e += blockDim.x) s_mix[(e / S) * SM + e % S] = mix[e];
  if (threadIdx.x < S) {
    s_out[threadIdx.x] = out[threadIdx.x];
    s_in[threadIdx.x] = h ? in[threadIdx.x] : 0.f;
  }
  __syncthreads();
  const int r = blockIdx.x;
  if (token_req && token_req[r] < 0) return;
  pdl_wait();
  pdl_trigger();
  x = after_wait(x);
  y = after_wait(y);
  float* xr = x + (size_t)r * ldx;
  const float* yr = y + (size_t)r * ldy;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < D; c += blockDim.x * VEC) {
    Cols<VEC> a[SM], b, acc;
    b.load(yr + c);
#pragma unroll
    for (int s = 0; s < SM; ++s)
      if (s < S) a[s].load(xr + (size_t)s * D + c);
#pragma unroll
    for (int e = 0; e < VEC; ++e) acc.v[e] = 0.f;
#pragma unroll
    for (int t = 0; t < SM; ++t) {
      if (t >= S) continue;
      Cols<VEC> n;
#pragma unroll
      for (int e = 0; e < VEC; ++e) n.v[e] = 0.f;
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (s < S)
#pragma unroll
          for (int e = 0; e < VEC; ++e) n.v[e] = fmaf(s_mix[s * SM + t], a[s].v[e], n.v[e]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        n.v[e] = fmaf(s_out[t], b.v[e], n.v[e]);
        acc.v[e] = fmaf(s_in[t], n.v[e], acc.v[e]);
      }
      n.store(xr + (size_t)t * D + c);
    }
    if (h) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss = fmaf(acc.v[e], acc.v[e], ss);
      acc.store(u + c);
    }
  }
  if (h) norm_row<TO, VEC>(u, ss, w, eps, h + (size_t)r * ldh, D, red);
}

static int streams_threads(int D, int vec) {
  const int n = (D + vec - 1) / vec;
  return n >= 512 ? 512 : (n >= 256 ? 256 : (n >= 128 ? 128 : 64));
}

#define ST_BY_COUNT(GO, TO, VEC)          \
  do {                                    \
    if (S <= 1) { GO(TO, 1, VEC); }       \
    else if (S <= 2) { GO(TO, 2, VEC); }  \
    else if (S <= 4) { GO(TO, 4, VEC); }  \
    else if (S <= 8) { GO(TO, 8, VEC); }  \
    else { GO(TO, ST_MAX, VEC); }         \
  } while (0)
#define ST_BY_TYPE(GO)                                               \
  do {                                                               \
    if (dtype == MLXB_F32) {                                         \
      if (vec) ST_BY_COUNT(GO, float, 4);                            \
      else ST_BY_COUNT(GO, float, 1);                                \
    } else {                                                         \
      if (vec) ST_BY_COUNT(GO, __nv_bfloat16, 4);                    \
      else ST_BY_COUNT(GO, __nv_bfloat16, 1);                        \
    }                                                                \
  } while (0)

// x: float32 [n_src_rows, S * D] at row stride ldx; rows: int32 [R] or null; in: float32 [S]; w: float32 [D];
// h: [R, D] of `dtype` at row stride ldh.
MLXB_EXPORT int mlxb_streams_read(int dtype, const float* x, int ldx, const int* rows, int n_src_rows, int S,
                                  const float* in, const float* w, float eps, void* h, int ldh, int R, int D,
                                  cudaStream_t stream) {
  if (R <= 0) return 0;
  if (S <= 0 || S > ST_MAX || D <= 0 || D > 12000 || ldx < S * D || ldh < D)
    return mlxb_fail(MLXB_BAD_ARG, "streams_read: %d streams (at most %d) of width %d, strides %d / %d", S, ST_MAX, D, ldx, ldh);
  if (dtype != MLXB_F32 && dtype != MLXB_BF16) return mlxb_fail(MLXB_BAD_DTYPE, "streams_read: dtype code %d", dtype);
  const bool vec = D % 4 == 0 && ldx % 4 == 0 && ldh % 4 == 0 && (((uintptr_t)x | (uintptr_t)w | (uintptr_t)h) & 15) == 0;
  const dim3 grid(R), block(streams_threads(D, vec ? 4 : 1));
  const size_t smem = sizeof(float) * (size_t)D;
#define ST_GO(TO, SM, VEC)                                                                                           \
  launch_pdl(streams_read_kernel<TO, SM, VEC>, grid, block, smem, stream, x, ldx, rows, n_src_rows, S, in, w, eps,  \
             (TO*)h, ldh, D)
  ST_BY_TYPE(ST_GO);
#undef ST_GO
  return mlxb_check_launch("streams_read");
}

// x: float32 [R, S * D] at row stride ldx, in place; y: float32 [R, D]; mix: float32 [S, S] (from, to); out: float32 [S];
// token_req: int32 [R] or null; h (or null): [R, D] of `dtype`, with in: float32 [S] and w: float32 [D].
MLXB_EXPORT int mlxb_streams_update(int dtype, float* x, int ldx, const float* y, int ldy, int S, const float* mix,
                                    const float* out, const int* token_req, const float* in, const float* w, float eps,
                                    void* h, int ldh, int R, int D, cudaStream_t stream) {
  if (R <= 0) return 0;
  if (S <= 0 || S > ST_MAX || D <= 0 || D > 12000 || ldx < S * D || ldy < D || (h && (ldh < D || !in || !w)))
    return mlxb_fail(MLXB_BAD_ARG, "streams_update: %d streams (at most %d) of width %d, strides %d / %d / %d", S, ST_MAX, D,
                     ldx, ldy, ldh);
  if (dtype != MLXB_F32 && dtype != MLXB_BF16) return mlxb_fail(MLXB_BAD_DTYPE, "streams_update: dtype code %d", dtype);
  const bool vec = D % 4 == 0 && ldx % 4 == 0 && ldy % 4 == 0 && (!h || ldh % 4 == 0) &&
                   (((uintptr_t)x | (uintptr_t)y | (uintptr_t)w | (uintptr_t)h) & 15) == 0;
  const dim3 grid(R), block(streams_threads(D, vec ? 4 : 1));
  const size_t smem = h ? sizeof(float) * (size_t)D : 0;
#define ST_GO(TO, SM, VEC)                                                                                           \
  launch_pdl(streams_update_kernel<TO, SM, VEC>, grid, block, smem, stream, x, ldx, y, ldy, S, mix, out, token_req, in, \
             w, eps, (TO*)h, ldh, D)
  ST_BY_TYPE(ST_GO);
#undef ST_GO
  return mlxb_check_launch("streams_update");
}
