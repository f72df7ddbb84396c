// Token embedding gather plus learned absolute position add:
//   h[t, :] = round(float(wte[tok[t], :]) + float(wpe[pos[t], :]))
// The sum is formed in 32-bit and rounded once.  `wpe` may be null (a model
// without a position table): then it is a plain gather.
// Instead of a table the positions may add a sinusoid: column 2i gets sin(p * freq[i]), column 2i+1 the cosine
// of the same angle (`freq` float32 [ceil(D/2)], the angle a float32 product, sincosf).
// embed_pairs is the embedding of a model that also looks up the pair (token before, token): the sum of the scaled
// token row and the pair's row, RMS-normed with a weight, written once per stream of the residual.
// Ids outside the tables set a status bit and produce zeros instead of
// reading out of bounds.
#include "common.cuh"

MLXB_DEFINE_LAST_ERROR()

template <typename T, typename TO = T>
__global__ void embed_pos_kernel(const int* __restrict__ tok, const int* __restrict__ pos,
                                 const T* __restrict__ wte, const T* __restrict__ wpe,
                                 TO* __restrict__ out, int D, int V, int P, float scale,
                                 int* __restrict__ status, const float* __restrict__ freq) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const int id = tok[t];
  const int p = (wpe || freq) ? pos[t] : 0;
  bool ok = true;
  if (id < 0 || id >= V) { ok = false; if (threadIdx.x == 0) atomicOr(status, MLXB_ST_TOKEN_RANGE); }
  if (wpe && (p < 0 || p >= P)) { ok = false; if (threadIdx.x == 0) atomicOr(status, MLXB_ST_POSITION_RANGE); }
  TO* o = out + (size_t)t * D;
  if (!ok) {
    for (int d = threadIdx.x; d < D; d += blockDim.x) o[d] = from_f<TO>(0.f);
    return;
  }
  const T* e = wte + (size_t)id * D;
  const T* q = wpe ? wpe + (size_t)p * D : nullptr;
  for (int d = threadIdx.x; d < D; d += blockDim.x) {
    float v = to_f(e[d]) * scale;
    if (q) v += to_f(q[d]);
    if (freq) {
      float sn, cs;
      sincosf((float)p * freq[d >> 1], &sn, &cs);
      v += (d & 1) ? cs : sn;
    }
    o[d] = from_f<TO>(v);
  }
}

// dtype: MLXB_F32 / MLXB_BF16 for the tables; the output has that dtype too, or is float32 with out_f32 (a model
// whose residual stream is float32 whatever its weights are).
MLXB_EXPORT int mlxb_embed_pos(int dtype, const int* tok, const int* pos, const void* wte, const void* wpe,
                               void* out, int T_, int D, int V, int P, float scale, int* status,
                               int out_f32, const float* freq, cudaStream_t stream) {
  if (T_ <= 0) return 0;
  if (D <= 0 || V <= 0) return mlxb_fail(MLXB_BAD_ARG, "embed_pos: width %d, vocabulary %d", D, V);
  const int threads = D >= 1024 ? 256 : (D >= 256 ? 128 : 64);
  if (dtype == MLXB_BF16 && out_f32)
    embed_pos_kernel<__nv_bfloat16, float><<<T_, threads, 0, stream>>>(tok, pos, (const __nv_bfloat16*)wte,
                                                                       (const __nv_bfloat16*)wpe, (float*)out, D, V, P,
                                                                       scale, status, freq);
  else if (dtype == MLXB_F32)
    embed_pos_kernel<float><<<T_, threads, 0, stream>>>(tok, pos, (const float*)wte, (const float*)wpe,
                                                        (float*)out, D, V, P, scale, status, freq);
  else if (dtype == MLXB_BF16)
    embed_pos_kernel<__nv_bfloat16><<<T_, threads, 0, stream>>>(tok, pos, (const __nv_bfloat16*)wte,
                                                                (const __nv_bfloat16*)wpe, (__nv_bfloat16*)out,
                                                                D, V, P, scale, status, freq);
  else
    return mlxb_fail(MLXB_BAD_DTYPE, "embed_pos: dtype code %d", dtype);
  return mlxb_check_launch("embed_pos");
}

// Tokens that are still on the device: dst[i] = src[index[i]] where index[i] >= 0 (dst[i] stays as it is where
// index[i] < 0).  Used to feed the tokens a step has just sampled into the next step without a round trip
// through the host; src has n_src words, an index outside it sets MLXB_ST_TOKEN_RANGE and leaves dst[i] alone.
__global__ void gather_tokens_kernel(const int* __restrict__ src, int n_src, const int* __restrict__ index,
                                     int* __restrict__ dst, int n, int* __restrict__ status) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const int j = index[i];
  if (j < 0) return;
  if (j >= n_src) { atomicOr(status, MLXB_ST_TOKEN_RANGE); return; }
  dst[i] = src[j];
}

MLXB_EXPORT int mlxb_gather_tokens(const int* src, int n_src, const int* index, int* dst, int n, int* status,
                                   cudaStream_t stream) {
  if (n <= 0) return 0;
  if (n_src <= 0) return mlxb_fail(MLXB_BAD_ARG, "gather_tokens: %d source words", n_src);
  gather_tokens_kernel<<<(n + 127) / 128, 128, 0, stream>>>(src, n_src, index, dst, n, status);
  return mlxb_check_launch("gather_tokens");
}

// out[t, n*D + d] = rmsnorm(wte[tok[t]] * scale + pairs[row(t)])[d] * w[d] for each of the S streams n, with
// row(t) = (prev * mul_prev + tok * mul_cur) mod buckets (64-bit arithmetic), or the table's last row (`buckets`) at
// position 0.  `prev` is the token of the row before, or, for the first row a request brings, the last token of the step
// before, kept in `last` (float32 [slots]: token ids are exact there up to 2^24).  The block of that first row is the
// only one that touches the request's slot: it reads it and then leaves the run's last token in it.  Without a pair
// table (pairs null) only the scaled rows are normed; without a weight (w null) nothing is normed.
template <typename T>
__global__ void embed_pairs_kernel(const int* __restrict__ tok, const int* __restrict__ pos,
                                   const int* __restrict__ token_req, const int* __restrict__ req_first_token,
                                   const int* __restrict__ slots, const T* __restrict__ wte,
                                   const T* __restrict__ pairs, float* last, const float* __restrict__ w,
                                   float* __restrict__ out, int D, int V, int S, float scale, long long buckets,
                                   long long mul_prev, long long mul_cur, float eps, int* __restrict__ status) {
  extern __shared__ float row[];      // the sum before the norm
  __shared__ float red[33];
  const int t = blockIdx.x;
  const int r = token_req[t], p = pos[t];
  int t0 = 0, t1 = 0, slot = 0;
  if (r >= 0) { t0 = req_first_token[r]; t1 = req_first_token[r + 1]; slot = slots[r]; }
  const bool first = r >= 0 && t == t0;
  pdl_wait();
  pdl_trigger();
  float* o = out + (size_t)t * S * D;
  const int id = tok[t];
  long long prev = 0;
  if (pairs && r >= 0 && p > 0) prev = first ? (long long)after_wait(last)[slot] : (long long)tok[t - 1];
  bool ok = r >= 0;
  if (ok && (id < 0 || id >= V)) { ok = false; if (threadIdx.x == 0) atomicOr(status, MLXB_ST_TOKEN_RANGE); }
  if (!ok) {
    for (int d = threadIdx.x; d < S * D; d += blockDim.x) o[d] = 0.f;
  } else {
    const T* e = wte + (size_t)id * D;
    const T* b = nullptr;
    if (pairs) {
      long long at = buckets;
      if (p > 0) {
        at = (prev * mul_prev + (long long)id * mul_cur) % buckets;
        if (at < 0) at += buckets;
      }
      b = pairs + (size_t)at * D;
    }
    float ss = 0.f;
    for (int d = threadIdx.x; d < D; d += blockDim.x) {
      float v = to_f(e[d]) * scale;
      if (b) v += to_f(b[d]);
      row[d] = v;
      ss = fmaf(v, v, ss);
    }
    const float rinv = w ? 1.f / sqrtf(block_sum(ss, red) / (float)D + eps) : 1.f;
    for (int d = threadIdx.x; d < D; d += blockDim.x) {
      const float v = w ? row[d] * rinv * w[d] : row[d];
      for (int n = 0; n < S; ++n) o[(size_t)n * D + d] = v;
    }
  }
  if (pairs && first) {
    // the run's last row (a request's rows come first in its range); every thread has read the slot by the first barrier
    int n = 0;
    for (int base = t; base < t1; base += blockDim.x) {
      const int tt = base + threadIdx.x;
      n += __syncthreads_count(tt < t1 && token_req[tt] == r);
    }
    if (threadIdx.x == 0) last[slot] = (float)tok[t + n - 1];
  }
}

// wte [V, D], pairs [buckets + 1, D]: dtype MLXB_F32 / MLXB_BF16; out: float32 [n_tokens, S * D].
MLXB_EXPORT int mlxb_embed_pairs(int dtype, const int* tok, const int* pos, const int* token_req,
                                 const int* req_first_token, const int* slots, const void* wte, const void* pairs,
                                 float* last, const float* w, float* out, int n_tokens, int D, int V, int S, float scale,
                                 long long buckets, long long mul_prev, long long mul_cur, float eps, int* status,
                                 cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (D <= 0 || V <= 0 || S <= 0 || (pairs && (buckets <= 0 || !last)) || D > 12000)
    return mlxb_fail(MLXB_BAD_ARG, "embed_pairs: width %d, vocabulary %d, %d streams, %lld buckets", D, V, S, buckets);
  const int threads = D >= 1024 ? 256 : (D >= 256 ? 128 : 64);
  const size_t smem = sizeof(float) * (size_t)D;
  if (dtype == MLXB_F32)
    launch_pdl(embed_pairs_kernel<float>, dim3(n_tokens), dim3(threads), smem, stream, tok, pos, token_req,
               req_first_token, slots, (const float*)wte, (const float*)pairs, last, w, out, D, V, S, scale, buckets,
               mul_prev, mul_cur, eps, status);
  else if (dtype == MLXB_BF16)
    launch_pdl(embed_pairs_kernel<__nv_bfloat16>, dim3(n_tokens), dim3(threads), smem, stream, tok, pos, token_req,
               req_first_token, slots, (const __nv_bfloat16*)wte, (const __nv_bfloat16*)pairs, last, w, out, D, V, S, scale,
               buckets, mul_prev, mul_cur, eps, status);
  else
    return mlxb_fail(MLXB_BAD_DTYPE, "embed_pairs: dtype code %d", dtype);
  return mlxb_check_launch("embed_pairs");
}
