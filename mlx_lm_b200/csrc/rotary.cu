// Queries, keys and values on their way from the projection into the attention kernels:
//   q, k   optional RMS norm over the WHOLE projection of a token (all heads at once, one weight per
//          column, eps inside the root), then a rotation by position of the first 2*half dimensions of
//          every head: dimension i is paired with i + half, the pair (u, v) at position p becomes
//          (u cos a - v sin a, v cos a + u sin a) with a = p * freq[i]; the other dimensions pass.
//   q      goes to a buffer [tokens, Hq*Dh]; k and v go into the token's page.  Heads are laid out Dh
//          wide there (values: Dvr wide), Dh >= dk, Dvr >= dv, the columns beyond a head's own size are written as zeros, so
//          that attention kernels built for one head size serve keys and values of different sizes
//          (zeros add nothing to a score, and the value columns they produce are never read).
//   Options: the pairs of a rotation may be neighbours instead ((2i, 2i+1), `interleaved`); cosine and sine may both
//   carry a factor (`mscale`, what a stretched rotation multiplies them with); every head of q and of k may be divided
//   by its root mean square over its dk columns after the rotation (no weight, `head_eps` >= 0); the values may have
//   fewer heads than the keys (Hv of them, [n_pages, Hv, page, Dvr]: several key heads then read one value head); every value head may be
//   divided by its root mean square over its dv columns (no weight, `v_eps` >= 0) before it enters the page; q may
//   leave in float32 whatever the activation dtype is (for attention kernels that take float32 queries), with a rounded
//   copy beside it (`q16`).  The values may be mixed with those of an earlier layer (rows of Hv*dv columns in a buffer):
//   (1 - lambda) v + lambda v_first goes into the page; the layer they come from leaves its own there (`v_keep`).
// Norm, angle, sine and cosine are float32 (the angle is the float32 product of the position and a
// float32 frequency, reduced accurately by sincosf).
#include "common.cuh"

MLXB_DEFINE_LAST_ERROR()

template <typename T, typename TQ>
__global__ void qkv_prepare_kernel(const T* proj, int ld, int q_off, int k_off, int v_off, int Hq, int Hkv, int dk,
                                   int dv, int Dh, const float* __restrict__ wq, const float* __restrict__ wk,
                                   float eps, const float* __restrict__ freq, int half,
                                   const int* __restrict__ positions, const int* __restrict__ token_req,
                                   const int* __restrict__ block_table, int max_pages, int n_pages, int page,
                                   TQ* __restrict__ q_out, int ldq, T* __restrict__ k_pool, T* __restrict__ v_pool,
                                   int write, int* __restrict__ status, int interleaved, float v_eps, int Dvr, int Hv,
                                   float mscale, float head_eps, __nv_bfloat16* __restrict__ q16, int ldq16,
                                   const T* v_first, T* v_keep, int ldvf, float lambda) {
  __shared__ float red[33];
  const int t = blockIdx.x;
  const int r = token_req[t];
  if (r < 0) return;
  const int p = positions[t];
  long long slot = -1;      // the token's row in head 0 of its page, counted in rows
  long long vslot = -1;     // the same among the value heads (Hv of them)
  if (write) {
    const int lp = p / page;
    if (p < 0 || lp >= max_pages) {
      if (threadIdx.x == 0) atomicOr(status, MLXB_ST_POSITION_RANGE);
    } else {
      const int pg = block_table[(size_t)r * max_pages + lp];
      if (pg >= n_pages) {
        if (threadIdx.x == 0) atomicOr(status, MLXB_ST_PAGE_RANGE);
      } else if (pg >= 0) {
        slot = (long long)pg * Hkv * page + (p % page);
        vslot = (long long)pg * Hv * page + (p % page);
      }
    }
  }
  pdl_wait();
  pdl_trigger();
  proj = after_wait(proj);
  v_first = after_wait(v_first);
  const T* row = proj + (size_t)t * ld;
  float rq = 1.f, rk = 1.f;
  if (wq) {
    float s = 0.f;
    for (int e = threadIdx.x; e < Hq * dk; e += blockDim.x) { const float v = to_f(row[q_off + e]); s = fmaf(v, v, s); }
    rq = 1.f / sqrtf(block_sum(s, red) / (float)(Hq * dk) + eps);
  }
  if (wk) {
    float s = 0.f;
    for (int e = threadIdx.x; e < Hkv * dk; e += blockDim.x) { const float v = to_f(row[k_off + e]); s = fmaf(v, v, s); }
    rk = 1.f / sqrtf(block_sum(s, red) / (float)(Hkv * dk) + eps);
  }
  const float fp = (float)p;
  if (head_eps >= 0.f) {
    // every head of q and of k divided by its root mean square AFTER the rotation: a warp a head, which forms the
    // head's values twice (for the sum of squares, then to write them)
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    for (int hh = warp; hh < Hq + Hkv; hh += nw) {
      const bool is_q = hh < Hq;
      const int h = is_q ? hh : hh - Hq;
      if (!is_q && slot < 0) continue;
      const T* src = row + (is_q ? q_off : k_off) + (size_t)h * dk;
      const float* w = is_q ? wq : wk;
      const float rn = is_q ? rq : rk;
      auto value = [&](int i) {
        float x = to_f(src[i]) * rn;
        if (w) x *= w[h * dk + i];
        if (i >= 2 * half) return x;
        const bool lower = interleaved ? !(i & 1) : i < half;
        const int partner = interleaved ? (i ^ 1) : (lower ? i + half : i - half);
        float y = to_f(src[partner]) * rn;
        if (w) y *= w[h * dk + partner];
        float sn, cs;
        sincosf(fp * freq[interleaved ? i >> 1 : (lower ? i : i - half)], &sn, &cs);
        cs *= mscale;
        sn *= mscale;
        return lower ? x * cs - y * sn : x * cs + y * sn;
      };
      float ss = 0.f;
      for (int i = lane; i < dk; i += 32) { const float a = value(i); ss = fmaf(a, a, ss); }
      const float rinv = 1.f / sqrtf(warp_sum(ss) / (float)dk + head_eps);
      for (int i = lane; i < Dh; i += 32) {
        const float a = i < dk ? value(i) * rinv : 0.f;
        if (is_q) {
          q_out[(size_t)t * ldq + (size_t)h * Dh + i] = from_f<TQ>(a);
          if (q16) q16[(size_t)t * ldq16 + (size_t)h * Dh + i] = __float2bfloat16_rn(a);
        } else k_pool[(size_t)(slot + (long long)h * page) * Dh + i] = from_f<T>(a);
      }
    }
  }
  // one thread per (head, dimension below Dh) of q and of k; the lower partner of a pair computes both
  for (int e = threadIdx.x; e < (head_eps >= 0.f ? 0 : (Hq + Hkv) * Dh); e += blockDim.x) {
    const int hh = e / Dh, i = e - hh * Dh;
    const bool is_q = hh < Hq;
    const int h = is_q ? hh : hh - Hq;
    const int off = is_q ? q_off : k_off;
    const float* w = is_q ? wq : wk;
    const float rn = is_q ? rq : rk;
    TQ* dq = nullptr;
    T* dk_ = nullptr;
    if (is_q) dq = q_out + (size_t)t * ldq + (size_t)h * Dh;
    else if (slot >= 0) dk_ = k_pool + (size_t)(slot + (long long)h * page) * Dh;
    else continue;
    float a = 0.f, b = 0.f;     // what goes to column i and, for the lower partner of a pair, to column j
    int j = -1;
    if (i < dk) {
      const bool rotated = i < 2 * half;
      if (rotated && (interleaved ? (i & 1) : i >= half)) continue;      // written by its partner
      const int c = h * dk + i;
      float u = to_f(row[off + c]) * rn;
      if (w) u *= w[c];
      if (rotated) {
        const int step = interleaved ? 1 : half;
        float v = to_f(row[off + c + step]) * rn;
        if (w) v *= w[c + step];
        float sn, cs;
        sincosf(fp * freq[interleaved ? i >> 1 : i], &sn, &cs);
        cs *= mscale;
        sn *= mscale;
        a = u * cs - v * sn;
        b = v * cs + u * sn;
        j = i + step;
      } else {
        a = u;
      }
    }
    if (is_q) {
      dq[i] = from_f<TQ>(a);
      if (j >= 0) dq[j] = from_f<TQ>(b);
      if (q16) {
        __nv_bfloat16* dr = q16 + (size_t)t * ldq16 + (size_t)h * Dh;
        dr[i] = __float2bfloat16_rn(a);
        if (j >= 0) dr[j] = __float2bfloat16_rn(b);
      }
    } else {
      dk_[i] = from_f<T>(a);
      if (j >= 0) dk_[j] = from_f<T>(b);
    }
  }
  if (v_keep)
    for (int e = threadIdx.x; e < Hv * dv; e += blockDim.x) v_keep[(size_t)t * ldvf + e] = row[v_off + e];
  if (slot >= 0 && v_eps >= 0.f) {
    // every value head divided by its root mean square: a warp a head
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    for (int h = warp; h < Hv; h += nw) {
      float s = 0.f;
      for (int i = lane; i < dv; i += 32) { const float v = to_f(row[v_off + h * dv + i]); s = fmaf(v, v, s); }
      const float rv = 1.f / sqrtf(warp_sum(s) / (float)dv + v_eps);
      for (int i = lane; i < Dvr; i += 32)
        v_pool[(size_t)(vslot + (long long)h * page) * Dvr + i] = from_f<T>(i < dv ? to_f(row[v_off + h * dv + i]) * rv : 0.f);
    }
  } else if (slot >= 0) {
    for (int e = threadIdx.x; e < Hv * Dvr; e += blockDim.x) {
      const int h = e / Dvr, i = e - h * Dvr;
      T v = i < dv ? row[v_off + h * dv + i] : from_f<T>(0.f);
      if (v_first && i < dv) v = from_f<T>((1.f - lambda) * to_f(v) + lambda * to_f(v_first[(size_t)t * ldvf + h * dv + i]));
      v_pool[(size_t)(vslot + (long long)h * page) * Dvr + i] = v;
    }
  }
}

// Four neighbouring elements as float32, and back.
__device__ __forceinline__ void qp_load4(const float* p, float (&v)[4]) {
  const float4 q = *reinterpret_cast<const float4*>(p);
  v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
}
__device__ __forceinline__ void qp_load4(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 q = *reinterpret_cast<const uint2*>(p);
  v[0] = __uint_as_float(q.x << 16);
  v[1] = __uint_as_float(q.x & 0xffff0000u);
  v[2] = __uint_as_float(q.y << 16);
  v[3] = __uint_as_float(q.y & 0xffff0000u);
}
__device__ __forceinline__ void qp_store4(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void qp_store4(__nv_bfloat16* p, const float (&v)[4]) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&a), *reinterpret_cast<const unsigned*>(&b));
}

// The same for heads whose sizes are multiples of 8 and fill their rows of the pages, pairs (i, i + half) with half a multiple
// of 4, no norm of single heads.  A thread takes four pairs of a head (eight columns where nothing turns), loads them once and
// keeps them in registers between the norm's sum and the result; sine and cosine are formed once per row and pair, and with
// the weights' and the page's lookups before the wait for the projection.  NI: pieces of q and k a thread takes.
constexpr int QF_HALF = 128;      // pairs at most

template <typename T, typename TQ, int NI>
__global__ void __launch_bounds__(256)
qkv_prepare_fast_kernel(const T* proj, int ld, int q_off, int k_off, int v_off, int Hq, int Hkv, int dk, int dv,
                        const float* __restrict__ wq, const float* __restrict__ wk, float eps, const float* __restrict__ freq,
                        int half, const int* __restrict__ positions, const int* __restrict__ token_req,
                        const int* __restrict__ block_table, int max_pages, int n_pages, int page, TQ* __restrict__ q_out, int ldq,
                        T* __restrict__ k_pool, T* __restrict__ v_pool, int write, int* __restrict__ status, int Hv, float mscale,
                        __nv_bfloat16* __restrict__ q16, int ldq16, const T* v_first, T* v_keep, int ldvf, float lambda) {
  __shared__ float s_cos[QF_HALF], s_sin[QF_HALF], s_red[2][8];
  const int t = blockIdx.x, tid = threadIdx.x;
  const int r = token_req[t];
  if (r < 0) return;
  const int p = positions[t];
  long long slot = -1, vslot = -1;      // the token's row in head 0 of its page, among the key heads and the value heads
  if (write) {
    const int lp = p / page;
    if (p < 0 || lp >= max_pages) {
      if (tid == 0) atomicOr(status, MLXB_ST_POSITION_RANGE);
    } else {
      const int pg = block_table[(size_t)r * max_pages + lp];
      if (pg >= n_pages) {
        if (tid == 0) atomicOr(status, MLXB_ST_PAGE_RANGE);
      } else if (pg >= 0) {
        slot = (long long)pg * Hkv * page + (p % page);
        vslot = (long long)pg * Hv * page + (p % page);
      }
    }
  }
  for (int i = tid; i < half; i += blockDim.x) {
    float sn, cs;
    sincosf((float)p * freq[i], &sn, &cs);
    s_cos[i] = cs * mscale;
    s_sin[i] = sn * mscale;
  }
  const int per = dk / 8, items = (Hq + Hkv) * per, turning = half / 4;
  // piece j of this thread: head, its first column and that of the partners
  auto place = [&](int e, int& hh, int& c0, int& c1) {
    hh = e / per;
    const int i = e - hh * per;
    if (i < turning) {
      c0 = 4 * i;
      c1 = c0 + half;
    } else {
      c0 = 8 * i;            // (the pieces that turn cover the first 2 * half = 8 * turning columns)
      c1 = c0 + 4;
    }
  };
  float w0[NI][4], w1[NI][4];
#pragma unroll
  for (int j = 0; j < NI; ++j) {
    const int e = tid + j * blockDim.x;
#pragma unroll
    for (int x = 0; x < 4; ++x) w0[j][x] = w1[j][x] = 1.f;
    if (e < items) {
      int hh, c0, c1;
      place(e, hh, c0, c1);
      const float* w = hh < Hq ? wq : wk;
      if (w) {
        w += (size_t)(hh < Hq ? hh : hh - Hq) * dk;
        qp_load4(w + c0, w0[j]);
        qp_load4(w + c1, w1[j]);
      }
    }
  }
  pdl_wait();
  pdl_trigger();
  proj = after_wait(proj);
  v_first = after_wait(v_first);
  const T* row = proj + (size_t)t * ld;
  float a[NI][4], b[NI][4], sq = 0.f, sk = 0.f;
#pragma unroll
  for (int j = 0; j < NI; ++j) {
    const int e = tid + j * blockDim.x;
    if (e < items) {
      int hh, c0, c1;
      place(e, hh, c0, c1);
      const T* src = row + (hh < Hq ? q_off + hh * dk : k_off + (hh - Hq) * dk);
      qp_load4(src + c0, a[j]);
      qp_load4(src + c1, b[j]);
      float s = 0.f;
#pragma unroll
      for (int x = 0; x < 4; ++x) s = fmaf(a[j][x], a[j][x], fmaf(b[j][x], b[j][x], s));
      if (hh < Hq) sq += s;
      else sk += s;
    }
  }
  // the values meanwhile: eight columns a piece
  const int vper = dv / 8;
  for (int e = tid; e < Hv * vper; e += blockDim.x) {
    const int h = e / vper, c = (e - h * vper) * 8, col = h * dv + c;
    float v0[4], v1[4];
    qp_load4(row + v_off + col, v0);
    qp_load4(row + v_off + col + 4, v1);
    if (v_keep) {
      qp_store4(v_keep + (size_t)t * ldvf + col, v0);
      qp_store4(v_keep + (size_t)t * ldvf + col + 4, v1);
    }
    if (slot < 0) continue;
    if (v_first) {
      float f0[4], f1[4];
      qp_load4(v_first + (size_t)t * ldvf + col, f0);
      qp_load4(v_first + (size_t)t * ldvf + col + 4, f1);
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        v0[x] = (1.f - lambda) * v0[x] + lambda * f0[x];
        v1[x] = (1.f - lambda) * v1[x] + lambda * f1[x];
      }
    }
    T* dst = v_pool + (size_t)(vslot + (long long)h * page) * dv + c;
    qp_store4(dst, v0);
    qp_store4(dst + 4, v1);
  }
  float rq = 1.f, rk = 1.f;
  {
    const int lane = tid & 31, warp = tid >> 5, nw = blockDim.x >> 5;
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0) {
      s_red[0][warp] = sq;
      s_red[1][warp] = sk;
    }
    __syncthreads();
    float tq = 0.f, tk = 0.f;
    for (int w = 0; w < nw; ++w) {
      tq += s_red[0][w];
      tk += s_red[1][w];
    }
    if (wq) rq = 1.f / sqrtf(tq / (float)(Hq * dk) + eps);
    if (wk) rk = 1.f / sqrtf(tk / (float)(Hkv * dk) + eps);
  }
#pragma unroll
  for (int j = 0; j < NI; ++j) {
    const int e = tid + j * blockDim.x;
    if (e >= items) continue;
    int hh, c0, c1;
    place(e, hh, c0, c1);
    const bool is_q = hh < Hq;
    const float rn = is_q ? rq : rk;
    float u[4], v[4];
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      u[x] = a[j][x] * rn * w0[j][x];
      v[x] = b[j][x] * rn * w1[j][x];
    }
    if (c1 - c0 == half && c0 < half) {
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const float cs = s_cos[c0 + x], sn = s_sin[c0 + x], y = u[x];
        u[x] = y * cs - v[x] * sn;
        v[x] = v[x] * cs + y * sn;
      }
    }
    if (is_q) {
      TQ* dst = q_out + (size_t)t * ldq + (size_t)hh * dk;
      qp_store4(dst + c0, u);
      qp_store4(dst + c1, v);
      if (q16) {
        __nv_bfloat16* d16 = q16 + (size_t)t * ldq16 + (size_t)hh * dk;
        qp_store4(d16 + c0, u);
        qp_store4(d16 + c1, v);
      }
    } else if (slot >= 0) {
      T* dst = k_pool + (size_t)(slot + (long long)(hh - Hq) * page) * dk;
      qp_store4(dst + c0, u);
      qp_store4(dst + c1, v);
    }
  }
}

// proj: [n_tokens, ...] at row stride ld holding q (Hq*dk columns from q_off), k (Hkv*dk from k_off) and v (Hkv*dv
// from v_off); interleaved: pairs (2i, 2i+1) instead of (i, i+half); v_eps >= 0: value heads divided by their root mean
// square with this eps; Hv: value heads (0: as many as key heads); mscale: factor on cosine and sine; head_eps >= 0: q and k
// heads divided by their root mean square after the rotation; q16: bfloat16 copy of q_out at row stride ldq16, or null; v_first
// (or null): [n_tokens, Hv*dv] at row stride ldvf, mixed into the values with weight lambda; v_keep (or null): the same rows
// written from this projection's values; q_f32: q_out is float32 whatever dtype says; wq / wk: float32 norm weights over the whole q / k projection, or null for no norm; freq: float32
// [half] rotation frequencies (half may be 0); k_pool [n_pages, Hkv, page, Dh], v_pool [n_pages, Hkv, page, Dvr]; q_out [n_tokens, Hq*Dh] at row stride ldq.
MLXB_EXPORT int mlxb_qkv_prepare(int dtype, const void* proj, int ld, int q_off, int k_off, int v_off, int Hq, int Hkv,
                                 int dk, int dv, int Dh, const float* wq, const float* wk, float eps, const float* freq,
                                 int half, const int* positions, const int* token_req, const int* block_table,
                                 int max_pages, int n_pages, int page, void* q_out, int ldq, void* k_pool, void* v_pool,
                                 int write, int n_tokens, int* status, int interleaved, float v_eps, int q_f32, int Dvr,
                                 int Hv, float mscale, float head_eps, void* q16, int ldq16, const void* v_first,
                                 void* v_keep, int ldvf, float lambda, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (Hv <= 0) Hv = Hkv;
  if (Hq <= 0 || Hkv <= 0 || dk <= 0 || dv <= 0 || Dh < dk || Dvr < dv || 2 * half > dk || half < 0 || page <= 0 ||
      (half > 0 && freq == nullptr) || ldq < Hq * Dh || (q16 && ldq16 < Hq * Dh) || ((v_first || v_keep) && ldvf < Hv * dv) ||
      (v_first && v_eps >= 0.f))
    return mlxb_fail(MLXB_BAD_ARG, "qkv_prepare: %d/%d heads, sizes %d/%d in %d, %d rotated pairs, page %d", Hq, Hkv, dk,
                     dv, Dh, half, page);
  {
    const size_t es = dtype == MLXB_F32 ? 4 : 2, qs = (dtype == MLXB_F32 || q_f32) ? 4 : 2;
    const int items = (Hq + Hkv) * (dk / 8);
    auto whole = [](const void* p, long long stride, size_t size) {      // rows of whole groups of four elements, aligned
      return p == nullptr || ((uintptr_t)p % (4 * size) == 0 && stride % 4 == 0);
    };
    const bool fast = head_eps < 0.f && v_eps < 0.f && !(interleaved && half) && dk % 8 == 0 && dv % 8 == 0 && Dh == dk && Dvr == dv &&
                      half % 4 == 0 && half <= QF_HALF && items <= 4 * 256 && q_off % 4 == 0 && k_off % 4 == 0 && v_off % 4 == 0 &&
                      whole(proj, ld, es) && whole(q_out, ldq, qs) && whole(k_pool, 0, es) && whole(v_pool, 0, es) && whole(q16, ldq16, 2) &&
                      whole(v_first, ldvf, es) && whole(v_keep, ldvf, es) && whole(wq, 0, 4) && whole(wk, 0, 4) &&
                      (dtype == MLXB_F32 || dtype == MLXB_BF16);
    if (fast) {
      const int threads = items <= 64 ? 64 : (items <= 128 ? 128 : 256), ni = (items + threads - 1) / threads;
#define QKVP_FAST(T, TQ, NI)                                                                                            \
  launch_pdl(qkv_prepare_fast_kernel<T, TQ, NI>, dim3(n_tokens), dim3(threads), 0, stream, (const T*)proj, ld, q_off, k_off, \
             v_off, Hq, Hkv, dk, dv, wq, wk, eps, freq, half, positions, token_req, block_table, max_pages, n_pages, page, \
             (TQ*)q_out, ldq, (T*)k_pool, (T*)v_pool, write, status, Hv, mscale, (__nv_bfloat16*)q16, ldq16,            \
             (const T*)v_first, (T*)v_keep, ldvf, lambda)
#define QKVP_FAST_NI(T, TQ)                                                                                             \
  do {                                                                                                                  \
    if (ni <= 1) QKVP_FAST(T, TQ, 1);                                                                                   \
    else if (ni <= 2) QKVP_FAST(T, TQ, 2);                                                                              \
    else QKVP_FAST(T, TQ, 4);                                                                                           \
  } while (0)
      if (dtype == MLXB_F32) QKVP_FAST_NI(float, float);
      else if (q_f32) QKVP_FAST_NI(__nv_bfloat16, float);
      else QKVP_FAST_NI(__nv_bfloat16, __nv_bfloat16);
#undef QKVP_FAST_NI
#undef QKVP_FAST
      return mlxb_check_launch("qkv_prepare");
    }
  }
  const int work = (Hq + Hkv) * Dh;
  const int threads = work >= 2048 ? 256 : (work >= 512 ? 128 : 64);
#define QKVP_GO(T, TQ)                                                                                                  \
  launch_pdl(qkv_prepare_kernel<T, TQ>, dim3(n_tokens), dim3(threads), 0, stream, (const T*)proj, ld, q_off, k_off, v_off, \
             Hq, Hkv, dk, dv, Dh, wq, wk, eps, freq, half, positions, token_req, block_table, max_pages, n_pages, page,  \
             (TQ*)q_out, ldq, (T*)k_pool, (T*)v_pool, write, status, interleaved, v_eps, Dvr, Hv, mscale, head_eps, \
             (__nv_bfloat16*)q16, ldq16, (const T*)v_first, (T*)v_keep, ldvf, lambda)
  if (dtype == MLXB_F32) QKVP_GO(float, float);
  else if (dtype == MLXB_BF16 && q_f32) QKVP_GO(__nv_bfloat16, float);
  else if (dtype == MLXB_BF16) QKVP_GO(__nv_bfloat16, __nv_bfloat16);
  else return mlxb_fail(MLXB_BAD_DTYPE, "qkv_prepare: dtype code %d", dtype);
#undef QKVP_GO
  return mlxb_check_launch("qkv_prepare");
}
