// Hyper-connections for ragged token batches: the residual stream of a token is S copies x_1 .. x_S (fp32), and one row
// kernel does everything between the output y of a sublayer and the operand of the next one, in ONE pass over the row:
//
//   x_t <- sum_s mix[s, t] x_s + w_out[t] * y        (all streams at once from the old ones; mix is [from][to])
//   u    = sum_s w_in[s] x_s                         (what the next sublayer reads; all ones: the model's output)
//   out  = tanh(alpha * u) * w + b                   (dynamic tanh: a norm without statistics), rounded once
//
// The sublayer's output is one of
//   dense rows            y[r]
//   expert rows           sum_k y_w[r, k] * y[y_pos[r, k]]    (rows in expert-grouped order)
//   a pair of branches    pair_scale * (RMS(y[r]) * w1 + RMS(y2[r]) * w2)     (each normed over the whole row)
// With ids given the old streams are all the token's embedding row, read from the table: the streams of a token need not
// exist in memory before the first sublayer has written them.  x is written only when there is a y and no rows_idx;
// rows_idx picks input rows (output packed).
//
// Nothing but the pair's two statistics looks across columns, so a thread owns four columns of all streams; a CTA serves
// one row, or (a handful of tokens) a slice of its columns.
#include "common.cuh"

namespace pg {

constexpr int HYPER_MAX_STREAMS = 32;

template <typename T>
struct HyperP {
  T* out; int ld_out;
  float* x;                                     // [rows][S][D]
  const T* y; int ldy;
  const int32_t* y_pos; const float* y_w; int y_top;
  const T* y2; int ldy2; const T* n1; const T* n2; float eps, pair_scale;
  const int64_t* ids; const T* table; long long vocab;
  const float* mix; const float* w_out;         // [S][S], [S]
  const float* w_in;                            // [S] stream weights of the next reader, then alpha
  const T* w; const T* b;
  const int32_t* rows_idx;
  int rows, D, S;
  int* err_flag;
};

template <typename T> __device__ __forceinline__ void hy_load4(const T* p, float* f) {
  if constexpr (sizeof(T) == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
  } else {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const T* t = reinterpret_cast<const T*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) f[i] = to_f<T>(t[i]);
  }
}
template <typename T> __device__ __forceinline__ void hy_store4(T* p, const float* f) {
  if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  } else {
    T t[4] = {from_f<T>(f[0]), from_f<T>(f[1]), from_f<T>(f[2]), from_f<T>(f[3])};
    *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(t);
  }
}

// 1 / rms of the two rows of a pair, every thread of the CTA
template <typename T, int VEC>
__device__ __forceinline__ void pair_inverse(const HyperP<T>& p, int src, float* red, float& i1, float& i2) {
  const T* a = p.y + (size_t)src * p.ldy;
  const T* b = p.y2 + (size_t)src * p.ldy2;
  float s1 = 0.f, s2 = 0.f;
  for (int c = threadIdx.x * VEC; c < p.D; c += blockDim.x * VEC) {
    float f[VEC], g[VEC];
    if constexpr (VEC == 4) { hy_load4<T>(a + c, f); hy_load4<T>(b + c, g); }
    else { f[0] = to_f<T>(a[c]); g[0] = to_f<T>(b[c]); }
#pragma unroll
    for (int i = 0; i < VEC; ++i) { s1 = fmaf(f[i], f[i], s1); s2 = fmaf(g[i], g[i], s2); }
  }
  s1 = block_sum(s1, red);
  s2 = block_sum(s2, red);
  i1 = p.pair_scale / sqrtf(s1 / (float)p.D + p.eps);
  i2 = p.pair_scale / sqrtf(s2 / (float)p.D + p.eps);
}

template <typename T>
__device__ __forceinline__ const T* embedding_row(const HyperP<T>& p, int src) {
  if (!p.ids) return nullptr;
  const int64_t id = p.ids[src];
  if (id >= 0 && id < p.vocab) return p.table + (size_t)id * p.D;
  if (threadIdx.x == 0 && p.err_flag) *p.err_flag = 1;
  return nullptr;
}

template <typename T, int S>
__global__ void __launch_bounds__(256) hyper_kernel(HyperP<T> p) {
  __shared__ float red[32];
  __shared__ float co[S * S + 2 * S + 1];          // mix | w_out | w_in | alpha
  pdl_launch_dependents();
  for (int i = threadIdx.x; i < S * S + 2 * S + 1; i += blockDim.x) {   // weights: not written by the preceding kernel
    float v = 0.f;
    if (i < S * S) { if (p.y) v = p.mix[i]; }
    else if (i < S * S + S) { if (p.y) v = p.w_out[i - S * S]; }
    else if (p.out) v = p.w_in[i - S * S - S];
    co[i] = v;
  }
  pdl_wait();
  __syncthreads();
  const int r = blockIdx.x, src = p.rows_idx ? p.rows_idx[r] : r;
  float* xr = p.x + (size_t)src * S * p.D;
  const T* er = embedding_row(p, src);
  float i1 = 0.f, i2 = 0.f;
  if (p.y2) pair_inverse<T, 4>(p, src, red, i1, i2);
  const float alpha = co[S * S + 2 * S];
  for (int c = (blockIdx.y * blockDim.x + threadIdx.x) * 4; c < p.D; c += gridDim.y * blockDim.x * 4) {
    float v[S][4], y[4] = {0.f, 0.f, 0.f, 0.f};
    if (p.ids) {
#pragma unroll
      for (int k = 0; k < 4; ++k) v[0][k] = 0.f;
      if (er) hy_load4<T>(er + c, v[0]);
#pragma unroll
      for (int s = 1; s < S; ++s)
#pragma unroll
        for (int k = 0; k < 4; ++k) v[s][k] = v[0][k];
    } else {
#pragma unroll
      for (int s = 0; s < S; ++s) hy_load4<float>(xr + (size_t)s * p.D + c, v[s]);
    }
    if (p.y) {
      if (p.y_pos) {
        for (int k = 0; k < p.y_top; ++k) {
          const int pos = p.y_pos[(size_t)src * p.y_top + k];
          if (pos < 0) continue;
          float f[4];
          hy_load4<T>(p.y + (size_t)pos * p.ldy + c, f);
          const float wk = p.y_w[(size_t)src * p.y_top + k];
#pragma unroll
          for (int i = 0; i < 4; ++i) y[i] = fmaf(wk, f[i], y[i]);
        }
      } else {
        hy_load4<T>(p.y + (size_t)src * p.ldy + c, y);
        if (p.y2) {
          float f[4], g1[4], g2[4];
          hy_load4<T>(p.y2 + (size_t)src * p.ldy2 + c, f);
          hy_load4<T>(p.n1 + c, g1);
          hy_load4<T>(p.n2 + c, g2);
#pragma unroll
          for (int i = 0; i < 4; ++i) y[i] = y[i] * i1 * g1[i] + f[i] * i2 * g2[i];
        }
      }
      float n[S][4];
#pragma unroll
      for (int t = 0; t < S; ++t) {
        const float wo = co[S * S + t];
#pragma unroll
        for (int i = 0; i < 4; ++i) n[t][i] = wo * y[i];
#pragma unroll
        for (int s = 0; s < S; ++s) {
          const float m = co[s * S + t];
#pragma unroll
          for (int i = 0; i < 4; ++i) n[t][i] = fmaf(m, v[s][i], n[t][i]);
        }
      }
#pragma unroll
      for (int t = 0; t < S; ++t) {
        if (!p.rows_idx) hy_store4<float>(xr + (size_t)t * p.D + c, n[t]);
#pragma unroll
        for (int i = 0; i < 4; ++i) v[t][i] = n[t][i];
      }
    }
    if (p.out) {
      float u[4] = {0.f, 0.f, 0.f, 0.f}, w[4], b[4];
#pragma unroll
      for (int s = 0; s < S; ++s) {
        const float wi = co[S * S + S + s];
#pragma unroll
        for (int i = 0; i < 4; ++i) u[i] = fmaf(wi, v[s][i], u[i]);
      }
      hy_load4<T>(p.w + c, w);
      hy_load4<T>(p.b + c, b);
#pragma unroll
      for (int i = 0; i < 4; ++i) u[i] = fmaf(tanhf(alpha * u[i]), w[i], b[i]);
      hy_store4<T>(p.out + (size_t)r * p.ld_out + c, u);
    }
  }
}

// Any number of streams, width and alignment: one column per thread.
template <typename T>
__global__ void __launch_bounds__(256) hyper_any_kernel(HyperP<T> p) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int S = p.S, r = blockIdx.x, src = p.rows_idx ? p.rows_idx[r] : r;
  float* xr = p.x + (size_t)src * S * p.D;
  const T* er = embedding_row(p, src);
  float i1 = 0.f, i2 = 0.f;
  if (p.y2) pair_inverse<T, 1>(p, src, red, i1, i2);
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < p.D; c += gridDim.y * blockDim.x) {
    float v[HYPER_MAX_STREAMS], y = 0.f, u = 0.f;
    for (int s = 0; s < S; ++s) v[s] = p.ids ? (er ? to_f<T>(er[c]) : 0.f) : xr[(size_t)s * p.D + c];
    if (p.y && p.y_pos) {
      for (int k = 0; k < p.y_top; ++k) {
        const int pos = p.y_pos[(size_t)src * p.y_top + k];
        if (pos >= 0) y = fmaf(p.y_w[(size_t)src * p.y_top + k], to_f<T>(p.y[(size_t)pos * p.ldy + c]), y);
      }
    } else if (p.y) {
      y = to_f<T>(p.y[(size_t)src * p.ldy + c]);
      if (p.y2) y = y * i1 * to_f<T>(p.n1[c]) + to_f<T>(p.y2[(size_t)src * p.ldy2 + c]) * i2 * to_f<T>(p.n2[c]);
    }
    for (int t = 0; t < S; ++t) {
      float n = v[t];
      if (p.y) {
        n = p.w_out[t] * y;
        for (int s = 0; s < S; ++s) n = fmaf(p.mix[s * S + t], v[s], n);
        if (!p.rows_idx) xr[(size_t)t * p.D + c] = n;
      }
      if (p.out) u = fmaf(p.w_in[t], n, u);
    }
    if (p.out) p.out[(size_t)r * p.ld_out + c] = from_f<T>(fmaf(tanhf(p.w_in[S] * u), to_f<T>(p.w[c]), to_f<T>(p.b[c])));
  }
}

template <typename T>
static int launch_hyper(const HyperP<T>& p, cudaStream_t st) {
  auto aligned = [](const void* q, size_t n) { return ((uintptr_t)q % n) == 0; };
  const size_t a4 = 4 * sizeof(T);
  const bool vec = p.S <= 8 && p.D % 4 == 0 && aligned(p.x, 16) && (!p.y || (p.ldy % 4 == 0 && aligned(p.y, a4))) &&
                   (!p.y2 || (p.ldy2 % 4 == 0 && aligned(p.y2, a4) && aligned(p.n1, a4) && aligned(p.n2, a4))) &&
                   (!p.ids || aligned(p.table, a4)) &&
                   (!p.out || (p.ld_out % 4 == 0 && aligned(p.out, a4) && aligned(p.w, a4) && aligned(p.b, a4)));
  const int cols = vec ? p.D / 4 : p.D, threads = cols <= 128 ? 128 : 256;
  // a handful of rows: a row's columns over several CTAs (a pair's statistics are then taken by each of them)
  const dim3 grid(p.rows, p.rows < 148 ? cdiv(cols, threads) : 1), block(threads);
  void (*kern)(HyperP<T>) = hyper_any_kernel<T>;
  if (vec) {
    switch (p.S) {
      case 1: kern = hyper_kernel<T, 1>; break;
      case 2: kern = hyper_kernel<T, 2>; break;
      case 3: kern = hyper_kernel<T, 3>; break;
      case 4: kern = hyper_kernel<T, 4>; break;
      case 5: kern = hyper_kernel<T, 5>; break;
      case 6: kern = hyper_kernel<T, 6>; break;
      case 7: kern = hyper_kernel<T, 7>; break;
      default: kern = hyper_kernel<T, 8>; break;
    }
  }
  return launch_pdl("hyper_connect", kern, grid, block, 0, st, p);
}

}  // namespace pg

using namespace pg;

extern "C" int pg_hyper_connect(void* out, int ld_out, float* x, int streams, const void* y, int ldy, const int32_t* y_pos,
                                const float* y_w, int y_top, const void* y2, int ldy2, const void* pair_w1, const void* pair_w2,
                                float eps, float pair_scale, const int64_t* ids, const void* table, long long vocab,
                                const float* mix, const float* w_out, const float* w_in, const void* w, const void* b,
                                const int32_t* rows_idx, int rows, int D, int* err_flag, int dtype, void* stream) {
  if (rows <= 0) return PG_OK;
  PG_REQUIRE(x && D > 0 && streams >= 1 && streams <= HYPER_MAX_STREAMS, "hyper_connect: %d streams (1..%d) of %d columns", streams,
             HYPER_MAX_STREAMS, D);
  PG_REQUIRE(!y || (mix && w_out), "hyper_connect: a sublayer's output needs the mixing weights");
  PG_REQUIRE(!y_pos || (y && y_w && y_top >= 1 && !y2), "hyper_connect: expert rows need places and weights");
  PG_REQUIRE(!y2 || (y && pair_w1 && pair_w2 && ldy2 >= D), "hyper_connect: a pair of branches needs both rows and both weights");
  PG_REQUIRE(!y || ldy >= D, "hyper_connect: sublayer rows of %d columns", ldy);
  PG_REQUIRE(!out || (w_in && w && b && ld_out >= D), "hyper_connect: an operand needs stream weights, weight and bias");
  PG_REQUIRE(!ids || table, "hyper_connect: embedding rows need a table");
  PG_DISPATCH_DTYPE(dtype, T, {
    const HyperP<T> p = {(T*)out, ld_out, x, (const T*)y, ldy, y_pos, y_w, y_top, (const T*)y2, ldy2, (const T*)pair_w1,
                         (const T*)pair_w2, eps, pair_scale, ids, (const T*)table, vocab, mix, w_out, w_in, (const T*)w,
                         (const T*)b, rows_idx, rows, D, streams, err_flag};
    return launch_hyper<T>(p, (cudaStream_t)stream);
  });
  return PG_OK;
}
