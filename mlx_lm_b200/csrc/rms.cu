// Root-mean-square norms over float32 rows, and the update of a float32 residual stream.
//
// rmsnorm          out[r, c] = x[row(r), c] / sqrt(mean_g(x^2) + eps) * (offset + w[c % period])
//                  The row is cut into `groups` equal parts, each divided by its own root mean square.
//                  The weight repeats with `period` columns (the width: one weight per column; the width
//                  of a part: the parts share one weight), is stored as it is (offset 0) or as its distance
//                  from one (offset 1).  A gate g (activation dtype) may come in: mode 1 multiplies x by
//                  silu(g) BEFORE the statistics, mode 2 multiplies the normed value by silu(g).
//                  x is float32 or has the activation dtype, which the result has.  No weight: the normed value as it is
//                  (times the offset where there is one).  All arithmetic is float32.  Rows or parts of up to
//                  512 columns without a weight, or in the activation dtype, take a kernel with a warp each.
// rmsnorm_rows     the same for whole float32 rows with a weight per column, a row kept in registers.
// residual_update  x[r, :] += scale * (f1(y1[r, :]) + f2(y2[r, :])),  f_i = rmsnorm with weight w_i over the
//                  whole row, or the identity where w_i is null; y2 may be null.  Optionally a copy of the new
//                  row in the activation dtype is left in `cast_out` for the products that read it next.
// norm_update      y = scale * (sum of the row's `terms` rows of y1) + y2[r, :];  x[r, :] += y / sqrt(mean(y^2) + eps) * w: a sublayer
//                  whose result is normed before it joins the stream, with the sum over the experts a token used in the same
//                  pass, and a copy of the new row as above.
#include "common.cuh"

MLXB_DEFINE_LAST_ERROR()

__device__ __forceinline__ float silu_f(float v) { return v / (1.f + expf(-v)); }

template <typename TI, typename TO>
__global__ void rmsnorm_kernel(const TI* x, int ldx, const int* __restrict__ rows, int n_src_rows,
                               const float* __restrict__ w, float offset, int period, const TO* gate, int ldg,
                               int gate_mode, TO* __restrict__ out, int ldo, int D, int groups, float eps) {
  __shared__ float red[33];
  pdl_wait();
  pdl_trigger();
  x = after_wait(x);
  gate = after_wait(gate);
  const int r = blockIdx.x, g = blockIdx.y;
  const int src = rows ? rows[r] : r;
  const int Dg = D / groups;
  TO* o = out + (size_t)r * ldo + (size_t)g * Dg;
  if (src < 0 || src >= n_src_rows) {
    for (int c = threadIdx.x; c < Dg; c += blockDim.x) o[c] = from_f<TO>(0.f);
    return;
  }
  const TI* xr = x + (size_t)src * ldx + (size_t)g * Dg;
  const TO* gr = gate ? gate + (size_t)src * ldg + (size_t)g * Dg : nullptr;
  float s = 0.f;
  for (int c = threadIdx.x; c < Dg; c += blockDim.x) {
    float v = to_f(xr[c]);
    if (gate_mode == 1) v *= silu_f(to_f(gr[c]));
    s = fmaf(v, v, s);
  }
  const float rinv = 1.f / sqrtf(block_sum(s, red) / (float)Dg + eps);
  for (int c = threadIdx.x; c < Dg; c += blockDim.x) {
    float v = to_f(xr[c]);
    if (gate_mode == 1) v *= silu_f(to_f(gr[c]));
    v = v * rinv * (w ? offset + w[(g * Dg + c) % period] : offset);
    if (gate_mode == 2) v *= silu_f(to_f(gr[c]));
    o[c] = from_f<TO>(v);
  }
}

// Four neighbouring columns: 16 bytes of float32, 8 of bfloat16.
__device__ __forceinline__ void load4(const float* p, float (&v)[4]) {
  const float4 q = *reinterpret_cast<const float4*>(p);
  v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
}
__device__ __forceinline__ void load4(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 q = *reinterpret_cast<const uint2*>(p);
  v[0] = __uint_as_float(q.x << 16);
  v[1] = __uint_as_float(q.x & 0xffff0000u);
  v[2] = __uint_as_float(q.y << 16);
  v[3] = __uint_as_float(q.y & 0xffff0000u);
}
__device__ __forceinline__ void store4(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float (&v)[4]) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&a), *reinterpret_cast<const unsigned*>(&b));
}

// Parts (or whole rows) of at most 128 * RP_STEPS columns (a multiple of 4, accesses of four columns): a warp per part,
// the part in registers between the sum and the result.
constexpr int RP_STEPS = 4;
template <typename TI, typename TO>
__global__ void __launch_bounds__(256)
rmsnorm_parts_kernel(const TI* x, int ldx, const float* __restrict__ w, float offset, int period, const TO* gate, int ldg,
                     int gate_mode, TO* __restrict__ out, int ldo, int R, int Dg, int groups, float eps) {
  pdl_wait();
  pdl_trigger();
  x = after_wait(x);
  gate = after_wait(gate);
  const int lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (item >= (long long)R * groups) return;
  const int r = (int)(item / groups), g = (int)(item - (long long)r * groups);
  const TI* xr = x + (size_t)r * ldx + (size_t)g * Dg;
  const TO* gr = gate_mode ? gate + (size_t)r * ldg + (size_t)g * Dg : nullptr;
  float v[RP_STEPS][4], gv[RP_STEPS][4];
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < RP_STEPS; ++i) {
    const int c = (i * 32 + lane) * 4;
#pragma unroll
    for (int e = 0; e < 4; ++e) v[i][e] = gv[i][e] = 0.f;
    if (c < Dg) {
      load4(xr + c, v[i]);
      if (gate_mode) load4(gr + c, gv[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < RP_STEPS; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      if (gate_mode == 1) v[i][e] *= silu_f(gv[i][e]);
      s = fmaf(v[i][e], v[i][e], s);
    }
  const float rinv = 1.f / sqrtf(warp_sum(s) / (float)Dg + eps);
  TO* o = out + (size_t)r * ldo + (size_t)g * Dg;
#pragma unroll
  for (int i = 0; i < RP_STEPS; ++i) {
    const int c = (i * 32 + lane) * 4;
    if (c >= Dg) continue;
    float res[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      res[e] = v[i][e] * rinv * (w ? offset + w[(g * Dg + c + e) % period] : offset);
      if (gate_mode == 2) res[e] *= silu_f(gv[i][e]);
    }
    store4(o + c, res);
  }
}

// Whole float32 rows with a weight per column, four columns a thread and step: the row stays in registers between the sum and
// the result, the weights are asked for before the wait.  NV * 4 * blockDim.x columns at most.
template <typename TO, int NV>
__global__ void __launch_bounds__(512)
rmsnorm_rows_kernel(const float* x, int ldx, const int* __restrict__ rows, int n_src_rows, const float* __restrict__ w, float offset,
                    TO* __restrict__ out, int ldo, int D, float eps) {
  __shared__ float red[33];
  const int r = blockIdx.x;
  const int src = rows ? rows[r] : r;
  const bool there = src >= 0 && src < n_src_rows;
  float wv[NV][4], v[NV][4];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 4;
    if (c < D) load4(w + c, wv[i]);
  }
  pdl_wait();
  pdl_trigger();
  x = after_wait(x);
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 4;
#pragma unroll
    for (int e = 0; e < 4; ++e) v[i][e] = 0.f;
    if (c < D && there) load4(x + (size_t)src * ldx + c, v[i]);
  }
#pragma unroll
  for (int i = 0; i < NV; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) s = fmaf(v[i][e], v[i][e], s);
  const float rinv = 1.f / sqrtf(block_sum(s, red) / (float)D + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 4;
    if (c >= D) continue;
#pragma unroll
    for (int e = 0; e < 4; ++e) v[i][e] = v[i][e] * rinv * (offset + wv[i][e]);
    store4(out + (size_t)r * ldo + c, v[i]);
  }
}

// x_f32: x is float32 (else it has out_dtype); w may be null (the offset is then the factor).
MLXB_EXPORT int mlxb_rmsnorm(int out_dtype, int x_f32, const void* x, int ldx, const int* rows, int n_src_rows, const float* w,
                             float offset, int period, const void* gate, int ldg, int gate_mode, void* out, int ldo,
                             int R, int D, int groups, float eps, cudaStream_t stream) {
  if (R <= 0) return 0;
  if (D <= 0 || groups <= 0 || D % groups || period <= 0 || ldx < D || ldo < D)
    return mlxb_fail(MLXB_BAD_ARG, "rmsnorm: width %d in %d parts, weight period %d, strides %d / %d", D, groups, period,
                     ldx, ldo);
  if (gate_mode < 0 || gate_mode > 2 || ((gate_mode != 0) != (gate != nullptr)))
    return mlxb_fail(MLXB_BAD_ARG, "rmsnorm: gate mode %d %s a gate", gate_mode, gate ? "with" : "without");
  if (groups > 65535) return mlxb_fail(MLXB_BAD_ARG, "rmsnorm: %d parts", groups);
  if (out_dtype != MLXB_F32 && out_dtype != MLXB_BF16) return mlxb_fail(MLXB_BAD_DTYPE, "rmsnorm: dtype code %d", out_dtype);
  const int Dg = D / groups;
  const int xb = (x_f32 || out_dtype == MLXB_F32) ? 16 : 8, ob = out_dtype == MLXB_F32 ? 16 : 8;   // bytes of four columns
  // (weighted norms of float32 rows keep the block per row or part and its order of additions)
  const bool parts = (w == nullptr || (!x_f32 && out_dtype == MLXB_BF16)) && rows == nullptr && Dg % 4 == 0 && Dg <= 128 * RP_STEPS && ldx % 4 == 0 && ldo % 4 == 0 &&
                     (!gate || ldg % 4 == 0) && (uintptr_t)x % xb == 0 && ((uintptr_t)out | (uintptr_t)gate) % ob == 0;
  const int threads = parts ? 256 : (Dg >= 2048 ? 256 : (Dg >= 512 ? 128 : (Dg >= 128 ? 64 : 32)));
  const dim3 grid = parts ? dim3((unsigned)(((long long)R * groups + 7) / 8)) : dim3(R, groups);
#define RMS_GO(TI, TO)                                                                                                  if (parts)                                                                                                              launch_pdl(rmsnorm_parts_kernel<TI, TO>, grid, dim3(threads), 0, stream, (const TI*)x, ldx, w, offset, period,                   (const TO*)gate, ldg, gate_mode, (TO*)out, ldo, R, Dg, groups, eps);                                     else                                                                                                                    launch_pdl(rmsnorm_kernel<TI, TO>, grid, dim3(threads), 0, stream, (const TI*)x, ldx, rows, n_src_rows, w, offset,                period, (const TO*)gate, ldg, gate_mode, (TO*)out, ldo, D, groups, eps)
  if (out_dtype == MLXB_F32) { RMS_GO(float, float); }
  else if (x_f32) { RMS_GO(float, __nv_bfloat16); }
  else { RMS_GO(__nv_bfloat16, __nv_bfloat16); }
#undef RMS_GO
  return mlxb_check_launch("rmsnorm");
}

// x: float32 rows at stride ldx, whole groups of four columns, 16-byte aligned, at most 8192 wide; rows: int32 [R] or null; w:
// float32 [D]; out: [R, D] of out_dtype.
MLXB_EXPORT int mlxb_rmsnorm_rows(int out_dtype, const float* x, int ldx, const int* rows, int n_src_rows, const float* w,
                                  float offset, void* out, int ldo, int R, int D, float eps, cudaStream_t stream) {
  if (R <= 0) return 0;
  const int ob = out_dtype == MLXB_F32 ? 16 : 8;
  if (D <= 0 || D % 4 || D > 4 * 512 * 4 || ldx % 4 || ldo % 4 || ldx < D || ldo < D || !w || (((uintptr_t)x | (uintptr_t)w) & 15) ||
      (uintptr_t)out % ob)
    return mlxb_fail(MLXB_BAD_ARG, "rmsnorm_rows: width %d, strides %d / %d", D, ldx, ldo);
  int threads = 64;
  while (threads < 512 && D / 4 > threads * 2) threads *= 2;
  const int nv = (D / 4 + threads - 1) / threads;
#define RMS_ROWS(TO, NV)                                                                                                \
  launch_pdl(rmsnorm_rows_kernel<TO, NV>, dim3(R), dim3(threads), 0, stream, x, ldx, rows, n_src_rows, w, offset, (TO*)out, ldo, \
             D, eps)
#define RMS_ROWS_NV(TO)                \
  do {                                 \
    if (nv <= 1) RMS_ROWS(TO, 1);      \
    else if (nv <= 2) RMS_ROWS(TO, 2); \
    else RMS_ROWS(TO, 4);              \
  } while (0)
  if (out_dtype == MLXB_F32) RMS_ROWS_NV(float);
  else if (out_dtype == MLXB_BF16) RMS_ROWS_NV(__nv_bfloat16);
  else return mlxb_fail(MLXB_BAD_DTYPE, "rmsnorm_rows: dtype code %d", out_dtype);
#undef RMS_ROWS_NV
#undef RMS_ROWS
  return mlxb_check_launch("rmsnorm_rows");
}

template <typename TO>
__global__ void residual_update_kernel(float* x, int ldx, const float* y1, const float* __restrict__ w1,
                                       const float* y2, const float* __restrict__ w2, int ldy, float scale, float eps,
                                       TO* __restrict__ cast_out, int ldc, int D) {
  __shared__ float red[33];
  pdl_wait();
  pdl_trigger();
  x = after_wait(x);
  y1 = after_wait(y1);
  y2 = after_wait(y2);
  const int r = blockIdx.x;
  float* xr = x + (size_t)r * ldx;
  const float* a = y1 + (size_t)r * ldy;
  const float* b = y2 ? y2 + (size_t)r * ldy : nullptr;
  float ra = 1.f, rb = 1.f;
  if (w1) {
    float s = 0.f;
    for (int c = threadIdx.x; c < D; c += blockDim.x) s = fmaf(a[c], a[c], s);
    ra = 1.f / sqrtf(block_sum(s, red) / (float)D + eps);
  }
  if (b && w2) {
    float s = 0.f;
    for (int c = threadIdx.x; c < D; c += blockDim.x) s = fmaf(b[c], b[c], s);
    rb = 1.f / sqrtf(block_sum(s, red) / (float)D + eps);
  }
  for (int c = threadIdx.x; c < D; c += blockDim.x) {
    float v = w1 ? a[c] * ra * w1[c] : a[c];
    if (b) v += w2 ? b[c] * rb * w2[c] : b[c];
    const float nx = xr[c] + scale * v;
    xr[c] = nx;
    if (cast_out) cast_out[(size_t)r * ldc + c] = from_f<TO>(nx);
  }
}

MLXB_EXPORT int mlxb_residual_update(int cast_dtype, float* x, int ldx, const float* y1, const float* w1,
                                     const float* y2, const float* w2, int ldy, float scale, float eps, void* cast_out,
                                     int ldc, int R, int D, cudaStream_t stream) {
  if (R <= 0) return 0;
  if (D <= 0 || ldx < D || ldy < D || y1 == nullptr || (cast_out && ldc < D))
    return mlxb_fail(MLXB_BAD_ARG, "residual_update: width %d, strides %d / %d / %d", D, ldx, ldy, ldc);
  const int threads = D >= 2048 ? 256 : (D >= 512 ? 128 : 64);
  if (cast_dtype == MLXB_F32)
    launch_pdl(residual_update_kernel<float>, dim3(R), dim3(threads), 0, stream, x, ldx, y1, w1, y2, w2, ldy, scale,
               eps, (float*)cast_out, ldc, D);
  else if (cast_dtype == MLXB_BF16)
    launch_pdl(residual_update_kernel<__nv_bfloat16>, dim3(R), dim3(threads), 0, stream, x, ldx, y1, w1, y2, w2, ldy,
               scale, eps, (__nv_bfloat16*)cast_out, ldc, D);
  else
    return mlxb_fail(MLXB_BAD_DTYPE, "residual_update: dtype code %d", cast_dtype);
  return mlxb_check_launch("residual_update");
}

// Two score maps over the same values, combined per head: with a1 and a2 the two maps' outputs of head h,
// o = a1 - lambda * a2, divided by its root mean square over the head's Dv columns (eps inside the root, no weight),
// times `post`.  a: float32 [T, lda] in which the heads of key/value group g lie as [map 1: rep heads | map 2: rep heads]
// (head h = g * rep + r has its first map at column ((2 g) rep + r) Dv and its second at ((2 g + 1) rep + r) Dv).
// One warp per (token, head).
template <typename TO>
__global__ void head_difference_kernel(const float* a, int lda, const int* __restrict__ token_req, int H, int rep, int Dv,
                                       float lambda, float eps, float post, TO* __restrict__ out, int ldo, int T) {
  pdl_wait();
  pdl_trigger();
  a = after_wait(a);
  const int lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (item >= (long long)T * H) return;
  const int t = (int)(item / H), h = (int)(item - (long long)t * H);
  if (token_req && token_req[t] < 0) return;
  const int g = h / rep, r = h - g * rep;
  const float* a1 = a + (size_t)t * lda + (size_t)((2 * g) * rep + r) * Dv;
  const float* a2 = a1 + (size_t)rep * Dv;
  float ss = 0.f;
  for (int d = lane; d < Dv; d += 32) { const float o = a1[d] - lambda * a2[d]; ss = fmaf(o, o, ss); }
  const float f = post / sqrtf(warp_sum(ss) / (float)Dv + eps);
  TO* op = out + (size_t)t * ldo + (size_t)h * Dv;
  for (int d = lane; d < Dv; d += 32) op[d] = from_f<TO>((a1[d] - lambda * a2[d]) * f);
}

MLXB_EXPORT int mlxb_head_difference(int out_dtype, const float* a, int lda, const int* token_req, int H, int rep, int Dv,
                                     float lambda, float eps, float post, void* out, int ldo, int T, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H <= 0 || rep <= 0 || H % rep || Dv <= 0 || lda < 2 * H * Dv || ldo < H * Dv)
    return mlxb_fail(MLXB_BAD_ARG, "head_difference: %d heads in groups of %d, %d columns, strides %d / %d", H, rep, Dv, lda, ldo);
  const int warps = 4;
  const dim3 grid((unsigned)(((long long)T * H + warps - 1) / warps));
  if (out_dtype == MLXB_F32)
    launch_pdl(head_difference_kernel<float>, grid, dim3(32 * warps), 0, stream, a, lda, token_req, H, rep, Dv, lambda, eps,
               post, (float*)out, ldo, T);
  else if (out_dtype == MLXB_BF16)
    launch_pdl(head_difference_kernel<__nv_bfloat16>, grid, dim3(32 * warps), 0, stream, a, lda, token_req, H, rep, Dv,
               lambda, eps, post, (__nv_bfloat16*)out, ldo, T);
  else
    return mlxb_fail(MLXB_BAD_DTYPE, "head_difference: dtype code %d", out_dtype);
  return mlxb_check_launch("head_difference");
}

// VEC: four columns a thread and step (16-byte accesses), or one.  A row's y and x stay in registers: NV * VEC * blockDim.x
// columns at most.
template <typename TO, int VEC, int NV>
__global__ void __launch_bounds__(512)
norm_update_kernel(float* x, int ldx, const float* y1, int ld1, int terms, float scale, const float* y2, int ld2,
                   const float* __restrict__ w, float eps, const int* __restrict__ token_req, TO* __restrict__ cast_out, int ldc,
                   int D) {
  __shared__ float red[33];
  const int r = blockIdx.x;
  if (token_req && token_req[r] < 0) return;
  auto get = [](const float* p, float (&v)[VEC]) {
    if (VEC == 4) {
      const float4 q = *reinterpret_cast<const float4*>(p);
      v[0] = q.x; v[VEC > 1 ? 1 : 0] = q.y; v[VEC > 2 ? 2 : 0] = q.z; v[VEC > 3 ? 3 : 0] = q.w;
    } else {
      v[0] = *p;
    }
  };
  float wv[NV][VEC], xv[NV][VEC], y[NV][VEC];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * VEC;
    if (c < D) get(w + c, wv[i]);
  }
  pdl_wait();
  pdl_trigger();
  x = after_wait(x);
  y1 = after_wait(y1);
  y2 = after_wait(y2);
  float* xr = x + (size_t)r * ldx;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * VEC;
    if (c < D) {
      get(xr + c, xv[i]);
      get(y1 + (size_t)r * terms * ld1 + c, y[i]);
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[i][e] = 0.f;
    }
  }
  for (int k = 1; k < terms; ++k)
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * VEC;
      if (c < D) {
        float a[VEC];
        get(y1 + ((size_t)r * terms + k) * ld1 + c, a);
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[i][e] += a[e];
      }
    }
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * VEC;
    float b[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) b[e] = 0.f;
    if (y2 && c < D) get(y2 + (size_t)r * ld2 + c, b);
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      y[i][e] = fmaf(scale, y[i][e], b[e]);
      s = fmaf(y[i][e], y[i][e], s);
    }
  }
  const float rinv = 1.f / sqrtf(block_sum(s, red) / (float)D + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * VEC;
    if (c >= D) continue;
    float n[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int e = 0; e < VEC; ++e) n[e] = xv[i][e] + y[i][e] * rinv * wv[i][e];
    if (VEC == 4) {
      store4(xr + c, n);
      if (cast_out) store4(cast_out + (size_t)r * ldc + c, n);
    } else {
      xr[c] = n[0];
      if (cast_out) cast_out[(size_t)r * ldc + c] = from_f<TO>(n[0]);
    }
  }
}

// x: float32 [R, D] at row stride ldx, in place; y1: float32 [R * terms, D]; y2: float32 [R, D] or null; w: float32 [D];
// token_req: int32 [R] or null (negative: the row is left alone); cast_out: [R, D] of cast_dtype, or null.
MLXB_EXPORT int mlxb_norm_update(int cast_dtype, float* x, int ldx, const float* y1, int ld1, int terms, float scale,
                                 const float* y2, int ld2, const float* w, float eps, const int* token_req, void* cast_out,
                                 int ldc, int R, int D, cudaStream_t stream) {
  if (R <= 0) return 0;
  if (cast_dtype != MLXB_F32 && cast_dtype != MLXB_BF16) return mlxb_fail(MLXB_BAD_DTYPE, "norm_update: dtype code %d", cast_dtype);
  const int cb = cast_dtype == MLXB_F32 ? 16 : 8;
  const bool vec = D % 4 == 0 && ldx % 4 == 0 && ld1 % 4 == 0 && (!y2 || ld2 % 4 == 0) && (!cast_out || ldc % 4 == 0) &&
                   (((uintptr_t)x | (uintptr_t)y1 | (uintptr_t)y2 | (uintptr_t)w) & 15) == 0 && (uintptr_t)cast_out % cb == 0;
  const int n = vec ? D / 4 : D;               // steps of one thread over a row, all together
  if (D <= 0 || terms <= 0 || ldx < D || ld1 < D || (y2 && ld2 < D) || (cast_out && ldc < D) || n > 512 * 8)
    return mlxb_fail(MLXB_BAD_ARG, "norm_update: width %d, %d terms, strides %d / %d / %d / %d", D, terms, ldx, ld1, ld2, ldc);
  int threads = 64;
  while (threads < 512 && n > threads * 2) threads *= 2;
  const int nv = (n + threads - 1) / threads;
#define NU_GO(TO, VEC, NV)                                                                                                \
  launch_pdl(norm_update_kernel<TO, VEC, NV>, dim3(R), dim3(threads), 0, stream, x, ldx, y1, ld1, terms, scale, y2, ld2, w, \
             eps, token_req, (TO*)cast_out, ldc, D)
#define NU_BY(TO, VEC)                    \
  do {                                    \
    if (nv <= 1) NU_GO(TO, VEC, 1);       \
    else if (nv <= 2) NU_GO(TO, VEC, 2);  \
    else if (nv <= 4) NU_GO(TO, VEC, 4);  \
    else NU_GO(TO, VEC, 8);               \
  } while (0)
  if (cast_dtype == MLXB_F32) { if (vec) NU_BY(float, 4); else NU_BY(float, 1); }
  else { if (vec) NU_BY(__nv_bfloat16, 4); else NU_BY(__nv_bfloat16, 1); }
#undef NU_BY
#undef NU_GO
  return mlxb_check_launch("norm_update");
}
