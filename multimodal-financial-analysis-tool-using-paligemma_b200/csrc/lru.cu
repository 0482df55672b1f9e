// Real-gated linear recurrent unit (a diagonal recurrence with input-dependent decays) for ragged token batches.
//
//   u  = causal convolution over time of (x + x_bias) per channel, plus a bias; zeros before the sequence's start
//   r, i = sigmoid of the block-diagonal products of u (fp32 pre-activations z from the per-head GEMM) + their biases
//   log a = -c r softplus(lam),  S_t = a S_(t-1) + sqrt(1 - a^2) i u,  S zero at the start       (c: a constant of the design)
//   out = S * gelu_tanh(y + y_bias)
// Gates, decays and state are fp32; 1 - a^2 is -expm1(2 log a), exact for slow decays.
//
// lru_conv_kernel    : u in the model dtype (the operand of the gates' products), a tile of rows per CTA.  Inputs of earlier
//                      positions are rows of this step where the sequence has them, else its state, which holds projected
//                      values WITHOUT the bias (the bias must not reach positions before the sequence).
// lru_scan_kernel    : a thread owns one, two or four channels and walks tokens; the loads of four tokens are in flight at once.
//   SEQ    (decode steps and short portions) one CTA column per segment, state read and written in place
//   FOLD   each chunk of LC tokens of a segment as an affine map of its incoming state: product of decays, final state from 0;
//          decays and inputs of the recurrence take the place of the gates' pre-activations
//   OUT    the chunk again from its incoming state, with the outputs: S = a S + x and the product with y are left to do
// lru_carry_kernel   : between FOLD and OUT, per (segment, channel): runs the chunks' maps in order, leaves every chunk's
//                      incoming state in the place of its product, writes the segment's final state to the slot.
// Chunks are cut inside segments; chunk k of segment s has number row0 / LC + s + k (unique, at most tokens / LC + segments),
// so the launch size depends on counts only.  Only lru_carry_kernel touches the slots, and a segment of 0 tokens has no chunk.
#include "common.cuh"

namespace pg {

constexpr int LRU_LC = 32;
__device__ __forceinline__ float lru_sigmoid(float v) { return 1.f / (1.f + expf(-v)); }

// VEC consecutive elements as floats, one vector access
template <typename T, int VEC>
__device__ __forceinline__ void lru_load(const T* q, float* f) {
  if constexpr (VEC == 1) {
    f[0] = to_f<T>(q[0]);
  } else if constexpr (sizeof(T) == 4) {
    if constexpr (VEC == 4) { const float4 v = *reinterpret_cast<const float4*>(q); f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w; }
    else { const float2 v = *reinterpret_cast<const float2*>(q); f[0] = v.x; f[1] = v.y; }
  } else {
    typename std::conditional<VEC == 4, uint2, uint32_t>::type v = *reinterpret_cast<const decltype(v)*>(q);
    const T* e = reinterpret_cast<const T*>(&v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) f[i] = to_f<T>(e[i]);
  }
}
template <typename T, int VEC>
__device__ __forceinline__ void lru_store(T* q, const float* f) {
  if constexpr (VEC == 1) {
    q[0] = from_f<T>(f[0]);
  } else if constexpr (sizeof(T) == 4) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(q) = make_float4(f[0], f[1], f[2], f[3]);
    else *reinterpret_cast<float2*>(q) = make_float2(f[0], f[1]);
  } else {
    T e[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) e[i] = from_f<T>(f[i]);
    typedef typename std::conditional<VEC == 4, uint2, uint32_t>::type U;
    *reinterpret_cast<U*>(q) = *reinterpret_cast<const U*>(e);
  }
}

// TOK consecutive rows per CTA; a thread walks them with the last KM inputs of its VEC channels in registers, refilled where
// the tile or a sequence starts.
template <typename T, int TOK, int VEC, int KM>
__global__ void __launch_bounds__(256)
lru_conv_kernel(T* __restrict__ u, const T* __restrict__ proj, int ld, int x_col0, const T* __restrict__ x_bias,
                const T* __restrict__ conv, const T* __restrict__ conv_b, int taps, const float* __restrict__ state,
                int state_len, int state_cols, const int32_t* __restrict__ tok_slot, const int32_t* __restrict__ tok_pos,
                int n_tokens, int width) {
  __shared__ int bef[TOK], reach_of[TOK], slot_of[TOK];
  pdl_launch_dependents();
  pdl_wait();
  const int K = taps - 1, t0 = blockIdx.x * TOK, nt = min(TOK, n_tokens - t0);
  if (threadIdx.x < nt) {
    const int t = t0 + threadIdx.x, slot = tok_slot[t], reach = min(K, tok_pos[t]);   // rows back that lie inside the sequence
    int b = 0;                                     // ... of which this many are rows of the step
    while (b < reach && t - b - 1 >= 0 && tok_slot[t - b - 1] == slot) ++b;
    bef[threadIdx.x] = b;
    reach_of[threadIdx.x] = reach;
    slot_of[threadIdx.x] = slot;
  }
  __syncthreads();
  for (int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC; c < width; c += gridDim.y * blockDim.x * VEC) {
    float bx[VEC], cb[VEC], w[KM + 1][VEC], prev[KM][VEC];   // w[j], prev[j - 1]: the tap and the (biased) input j rows back
    lru_load<T, VEC>(x_bias + c, bx);
    lru_load<T, VEC>(conv_b + c, cb);
#pragma unroll
    for (int j = 0; j <= KM; ++j)
      if (j <= K) lru_load<T, VEC>(conv + (size_t)(K - j) * width + c, w[j]);
    const T* row = proj + (size_t)t0 * ld + x_col0 + c;
    constexpr int UN = TOK < 8 ? TOK : 8;          // rows requested together
    float rows[UN][VEC];
    for (int r0 = 0; r0 < nt; r0 += UN) {
#pragma unroll
      for (int q = 0; q < UN; ++q) lru_load<T, VEC>(row + (size_t)min(r0 + q, nt - 1) * ld, rows[q]);
#pragma unroll
      for (int q = 0; q < UN; ++q) {
        const int r = r0 + q;
        if (r >= nt) break;
        const int b = bef[r];
        if (r == 0 || b < K) {
#pragma unroll
          for (int j = 1; j <= KM; ++j)
            if (j <= K) {
              float* v = prev[j - 1];
              if (j > reach_of[r]) {               // before the sequence: nothing, not even the bias
#pragma unroll
                for (int i = 0; i < VEC; ++i) v[i] = 0.f;
              } else if (j > b || r == 0) {
                if (j <= b) lru_load<T, VEC>(row - (long long)j * ld, v);
                else lru_load<float, VEC>(state + ((size_t)slot_of[r] * state_len + (state_len - (j - b))) * state_cols + c, v);
#pragma unroll
                for (int i = 0; i < VEC; ++i) v[i] += bx[i];
              }
            }
        }
        float o[VEC];
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          rows[q][i] += bx[i];
          o[i] = fmaf(rows[q][i], w[0][i], cb[i]);
#pragma unroll
          for (int j = 1; j <= KM; ++j)
            if (j <= K) o[i] = fmaf(prev[j - 1][i], w[j][i], o[i]);
        }
        lru_store<T, VEC>(u + (size_t)(t0 + r) * width + c, o);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
#pragma unroll
          for (int j = KM; j >= 2; --j)
            if (j <= K) prev[j - 1][i] = prev[j - 2][i];
          if (K >= 1) prev[0][i] = rows[q][i];
        }
      }
    }
  }
}

// Any number of taps: a token per CTA row, every input read where it lies.
template <typename T>
__global__ void __launch_bounds__(256)
lru_conv_any_kernel(T* __restrict__ u, const T* __restrict__ proj, int ld, int x_col0, const T* __restrict__ x_bias,
                    const T* __restrict__ conv, const T* __restrict__ conv_b, int taps, const float* __restrict__ state,
                    int state_len, int state_cols, const int32_t* __restrict__ tok_slot, const int32_t* __restrict__ tok_pos,
                    int n_tokens, int width) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, K = taps - 1, slot = tok_slot[t], reach = min(K, tok_pos[t]);
  int before = 0;
  while (before < reach && t - before - 1 >= 0 && tok_slot[t - before - 1] == slot) ++before;
  const T* row = proj + (size_t)t * ld + x_col0;
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < width; c += gridDim.y * blockDim.x) {
    const float bx = to_f<T>(x_bias[c]);
    float acc = to_f<T>(conv_b[c]);
    for (int j = 0; j <= reach; ++j) {
      const float v = j <= before ? to_f<T>(row[c - (long long)j * ld])
                                  : state[((size_t)slot * state_len + (state_len - (j - before))) * state_cols + c];
      acc = fmaf(v + bx, to_f<T>(conv[(size_t)(K - j) * width + c]), acc);
    }
    u[(size_t)t * width + c] = from_f<T>(acc);
  }
}

template <typename T>
struct LruP {
  T* out; int ld_out;
  float* state;                                    // [slots][width]
  float* z;                                        // [tokens][2 * width]: per block [r: bs | i: bs]; after FOLD [a | x]
  const T* u; const T* y; int ld_y; const T* y_b; const T* r_b; const T* i_b;
  const float* lam; float c;
  const int32_t* segs; int n_segs, width, bs;
  float* sum_a; float* sum_s;                      // [chunks][width]
};

// The segment that owns chunk `c` and the chunk's place in it; false when there is none.
__device__ __forceinline__ bool lru_chunk(const int32_t* segs, int n_segs, int c, int& row0, int& n) {
  auto base = [&](int s) { return segs[3 * s + 2] > 0 ? segs[3 * s + 1] / LRU_LC + s : 0x7fffffff; };   // empty ones come last
  int lo = 0, hi = n_segs;                         // the last segment with base <= c
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (base(mid) <= c) lo = mid; else hi = mid;
  }
  const int b = base(lo);
  if (b > c) return false;
  const int first = (c - b) * LRU_LC, len = segs[3 * lo + 2];
  if (first >= len) return false;
  row0 = segs[3 * lo + 1] + first;
  n = min(LRU_LC, len - first);
  return true;
}

enum { LRU_SEQ = 0, LRU_FOLD = 1, LRU_OUT = 2 };

// The decay a = exp(la) and 1 - a^2 (la <= 0).  Close to 0 the Taylor series of -expm1(2 la) to the sixth power (relative
// error below 1e-7 for 2 la > -1/4), elsewhere 1 - a a, which loses at most two bits there.
__device__ __forceinline__ void lru_decay(float la, float& a, float& gain2) {
  a = expf(la);
  const float x = 2.f * la;
  float s = fmaf(x, 1.f / 720.f, 1.f / 120.f);
  s = fmaf(x, s, 1.f / 24.f);
  s = fmaf(x, s, 1.f / 6.f);
  s = fmaf(x, s, 0.5f);
  s = fmaf(x, s, 1.f);
  gain2 = x > -0.25f ? -x * s : fmaf(-a, a, 1.f);
}

template <typename T, int VEC, int MODE>
__global__ void __launch_bounds__(128) lru_scan_kernel(LruP<T> p) {
  constexpr bool FAST = sizeof(T) == 2;            // 16-bit u, y and outputs: the fast exponential in the gates' sigmoids
  __shared__ int where[3];
  pdl_launch_dependents();
  pdl_wait();
  int row0, n, slot = 0;
  if (MODE == LRU_SEQ) {
    const int32_t* sg = p.segs + 3 * (size_t)blockIdx.x;
    slot = sg[0]; row0 = sg[1]; n = sg[2];
  } else {
    if (threadIdx.x == 0) {
      int a = 0, b = 0;
      where[2] = lru_chunk(p.segs, p.n_segs, blockIdx.x, a, b) ? 1 : 0;
      where[0] = a;
      where[1] = b;
    }
    __syncthreads();
    row0 = where[0];
    n = where[2] ? where[1] : 0;
  }
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  if (n <= 0 || c >= p.width) return;
  const int blk = c / p.bs, zc = blk * 2 * p.bs + (c - blk * p.bs);
  float k[VEC], rb[VEC], ib[VEC], yb[VEC], S[VEC], A[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) {
    if (MODE != LRU_OUT) {
      const float l = p.lam[c + e];
      k[e] = -p.c * (fmaxf(l, 0.f) + log1pf(expf(-fabsf(l))));
      rb[e] = to_f<T>(p.r_b[c + e]);
      ib[e] = to_f<T>(p.i_b[c + e]);
    }
    if (MODE != LRU_FOLD) yb[e] = to_f<T>(p.y_b[c + e]);
    A[e] = 1.f;
    S[e] = MODE == LRU_SEQ ? p.state[(size_t)slot * p.width + c + e]
                           : (MODE == LRU_OUT ? p.sum_a[(size_t)blockIdx.x * p.width + c + e] : 0.f);
  }
  float* zp = p.z + (size_t)row0 * 2 * p.width + zc;
  const T* up = p.u + (size_t)row0 * p.width + c;
  const T* yp = p.y + (size_t)row0 * p.ld_y + c;
  T* op = p.out + (size_t)row0 * p.ld_out + c;
  constexpr int UN = 4;
  for (int t0 = 0; t0 < n; t0 += UN) {
    float zr[UN][VEC], zi[UN][VEC], uu[UN][VEC], yy[UN][VEC];
#pragma unroll
    for (int q = 0; q < UN; ++q) {
      const int t = min(t0 + q, n - 1);
      lru_load<float, VEC>(zp + (size_t)t * 2 * p.width, zr[q]);
      lru_load<float, VEC>(zp + (size_t)t * 2 * p.width + p.bs, zi[q]);
      if (MODE != LRU_OUT) lru_load<T, VEC>(up + (size_t)t * p.width, uu[q]);
      if (MODE != LRU_FOLD) lru_load<T, VEC>(yp + (size_t)t * p.ld_y, yy[q]);
    }
#pragma unroll
    for (int q = 0; q < UN; ++q) {
      if (t0 + q >= n) break;
      float o[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        if (MODE != LRU_OUT) {                     // pre-activations to decay and input
          float a, g2;
          const float r = FAST ? __fdividef(1.f, 1.f + __expf(-(zr[q][e] + rb[e]))) : lru_sigmoid(zr[q][e] + rb[e]);
          const float i = FAST ? __fdividef(1.f, 1.f + __expf(-(zi[q][e] + ib[e]))) : lru_sigmoid(zi[q][e] + ib[e]);
          lru_decay(k[e] * r, a, g2);
          zr[q][e] = a;
          zi[q][e] = sqrtf(g2) * i * uu[q][e];
        }
        S[e] = fmaf(zr[q][e], S[e], zi[q][e]);
        if (MODE == LRU_FOLD) A[e] *= zr[q][e];
        else o[e] = S[e] * (FAST ? gelu_tanh_fast(yy[q][e] + yb[e]) : gelu_tanh(yy[q][e] + yb[e]));
      }
      if (MODE == LRU_FOLD) {
        float* d = zp + (size_t)(t0 + q) * 2 * p.width;
        lru_store<float, VEC>(d, zr[q]);
        lru_store<float, VEC>(d + p.bs, zi[q]);
      } else {
        lru_store<T, VEC>(op + (size_t)(t0 + q) * p.ld_out, o);
      }
    }
  }
#pragma unroll
  for (int e = 0; e < VEC; ++e) {
    if (MODE == LRU_SEQ) p.state[(size_t)slot * p.width + c + e] = S[e];
    if (MODE == LRU_FOLD) {
      p.sum_a[(size_t)blockIdx.x * p.width + c + e] = A[e];
      p.sum_s[(size_t)blockIdx.x * p.width + c + e] = S[e];
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(128) lru_carry_kernel(LruP<T> p) {
  pdl_launch_dependents();
  pdl_wait();
  const int s = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
  const int slot = p.segs[3 * s], row0 = p.segs[3 * s + 1], n = p.segs[3 * s + 2];
  if (n <= 0 || c >= p.width) return;
  const int chunks = (n + LRU_LC - 1) / LRU_LC;
  float* a = p.sum_a + (size_t)(row0 / LRU_LC + s) * p.width + c;
  const float* f = p.sum_s + (size_t)(row0 / LRU_LC + s) * p.width + c;
  float S = p.state[(size_t)slot * p.width + c];
  constexpr int UN = 8;
  for (int k0 = 0; k0 < chunks; k0 += UN) {
    float av[UN], fv[UN];
#pragma unroll
    for (int q = 0; q < UN; ++q) {
      const int k = min(k0 + q, chunks - 1);
      av[q] = a[(size_t)k * p.width];
      fv[q] = f[(size_t)k * p.width];
    }
#pragma unroll
    for (int q = 0; q < UN; ++q) {
      if (k0 + q >= chunks) break;
      a[(size_t)(k0 + q) * p.width] = S;           // the chunk's incoming state, in the place of its product
      S = fmaf(av[q], S, fv[q]);
    }
  }
  p.state[(size_t)slot * p.width + c] = S;
}

template <typename T, int VEC>
static int launch_lru(const LruP<T>& p, int n_tokens, bool chunked, cudaStream_t st) {
  const int gy = cdiv(p.width, 128 * VEC);
  if (!chunked) return launch_pdl("lru_scan", lru_scan_kernel<T, VEC, LRU_SEQ>, dim3(p.n_segs, gy), dim3(128), 0, st, p);
  const int chunks = n_tokens / LRU_LC + p.n_segs;
  int rc = launch_pdl("lru_fold", lru_scan_kernel<T, VEC, LRU_FOLD>, dim3(chunks, gy), dim3(128), 0, st, p);
  if (rc == PG_OK) rc = launch_pdl("lru_carry", lru_carry_kernel<T>, dim3(p.n_segs, cdiv(p.width, 128)), dim3(128), 0, st, p);
  if (rc == PG_OK) rc = launch_pdl("lru_out", lru_scan_kernel<T, VEC, LRU_OUT>, dim3(chunks, gy), dim3(128), 0, st, p);
  return rc;
}

}  // namespace pg

using namespace pg;

extern "C" int pg_lru_conv(void* u, const void* proj, int ld, int x_col0, const void* x_bias, const void* conv,
                           const void* conv_b, int taps, const float* state, int state_len, int state_cols,
                           const int32_t* tok_slot, const int32_t* tok_pos, int n_tokens, int width, int dtype, void* stream) {
  if (n_tokens <= 0) return PG_OK;
  PG_REQUIRE(u && proj && x_bias && conv && conv_b && tok_slot && tok_pos && width > 0, "lru_conv: bad arguments");
  PG_REQUIRE(taps >= 1 && (taps == 1 || (state && state_len >= taps - 1 && state_cols >= width)),
             "lru_conv: %d taps over a state of %d rows of %d columns", taps, state_len, state_cols);
  PG_DISPATCH_DTYPE(dtype, T, {
    const size_t a4 = 4 * sizeof(T);
    const bool quad = width % 4 == 0 && ld % 4 == 0 && x_col0 % 4 == 0 && ((uintptr_t)proj % a4) == 0 && ((uintptr_t)u % a4) == 0 &&
                      ((uintptr_t)x_bias % a4) == 0 && ((uintptr_t)conv_b % a4) == 0 && ((uintptr_t)conv % a4) == 0 &&
                      (taps == 1 || (((uintptr_t)state % 16) == 0 && state_cols % 4 == 0));
    auto kern = lru_conv_any_kernel<T>;
    int tok = 1;
    if (taps <= 8) {
      tok = n_tokens <= 296 ? 1 : 16;
      if (tok == 1) kern = quad ? lru_conv_kernel<T, 1, 4, 7> : lru_conv_kernel<T, 1, 1, 7>;
      else if (taps <= 4) kern = quad ? lru_conv_kernel<T, 16, 4, 3> : lru_conv_kernel<T, 16, 1, 3>;
      else kern = quad ? lru_conv_kernel<T, 16, 4, 7> : lru_conv_kernel<T, 16, 1, 7>;
    }
    const int cols = (taps <= 8 && quad) ? width / 4 : width, threads = cols <= 128 ? 128 : 256;
    return launch_pdl("lru_conv", kern, dim3(cdiv(n_tokens, tok), cdiv(cols, threads)), dim3(threads), 0, (cudaStream_t)stream, (T*)u,
                      (const T*)proj, ld, x_col0, (const T*)x_bias, (const T*)conv, (const T*)conv_b, taps, state, state_len, state_cols, tok_slot,
                      tok_pos, n_tokens, width);
  });
  return PG_OK;
}

extern "C" long long pg_lru_ws_floats(int n_tokens, int n_segs, int width) {
  return 2ll * (n_tokens / LRU_LC + n_segs) * width;
}

extern "C" int pg_lru_scan(void* out, int ld_out, float* state, float* z, const void* u, const void* y, int ld_y,
                           const void* y_bias, const void* r_bias, const void* i_bias, const float* lam, float c,
                           const int32_t* segs, int n_segs, int n_tokens, int width, int blocks, float* ws, int impl, int dtype,
                           void* stream) {
  if (n_segs <= 0 || n_tokens <= 0) return PG_OK;
  PG_REQUIRE(out && state && z && u && y && y_bias && r_bias && i_bias && lam && segs, "lru_scan: bad arguments");
  PG_REQUIRE(blocks >= 1 && width % blocks == 0, "lru_scan: %d channels in %d blocks", width, blocks);
  PG_REQUIRE(impl >= 0 && impl <= 2 && (impl != 2 || ws), "lru_scan: impl %d", impl);
  // impl 0: chunked where some segment is long enough to gain from it, 1: token by token, 2: chunked
  const bool chunked = impl == 2 || (impl == 0 && ws && n_tokens - n_segs >= 2 * LRU_LC);
  const int bs = width / blocks;
  PG_DISPATCH_DTYPE(dtype, T, {
    const LruP<T> p = {(T*)out, ld_out, state, z, (const T*)u, (const T*)y, ld_y, (const T*)y_bias, (const T*)r_bias,
                       (const T*)i_bias, lam, c, segs, n_segs, width, bs, ws,
                       ws ? ws + (size_t)(n_tokens / LRU_LC + n_segs) * width : nullptr};
    auto fits = [&](int v) {
      const size_t av = v * sizeof(T);
      return bs % v == 0 && ld_y % v == 0 && ld_out % v == 0 && ((uintptr_t)u % av) == 0 && ((uintptr_t)y % av) == 0 &&
             ((uintptr_t)out % av) == 0 && ((uintptr_t)z % (4 * v)) == 0;
    };
    static const int wide = env_int("PG_LRU_WIDE", 1);
    if (wide && chunked && width >= 2048 && fits(4)) return launch_lru<T, 4>(p, n_tokens, chunked, (cudaStream_t)stream);
    return fits(2) ? launch_lru<T, 2>(p, n_tokens, chunked, (cudaStream_t)stream) : launch_lru<T, 1>(p, n_tokens, chunked, (cudaStream_t)stream);
  });
  return PG_OK;
}
