// The row kernel between two sublayers of a pre-norm model with layer norms: everything that happens to a row of the
// fp32 residual stream from the end of one sublayer to the operand of the next one, in ONE pass over the row.
//
//   x[r]  = table[ids[r]]                       (emb_mode PG_EMB_INIT: the first sublayer of the model)
//   x[r] += sum of the sublayer's output rows   (a dense output row, or the `y_top` expert outputs of the token, found
//                                                through y_pos in expert-grouped order, each times y_w)
//   x[r] += table[ids[r]]                       (emb_mode PG_EMB_ADD: the embedding output once more, before a repeated
//                                                pass of a looped block: read again from the table, never kept)
//   x[r] += vec                                 (one vector for all rows: a pass's step vector)
//   out   = ((x - mean) / sqrt(mean((x - mean)^2) + eps) * w + b) * out_scale
//
// The result is rounded once, to the model dtype.  With out_pos the row is written to the `out_top` places of the
// token's experts in expert-grouped order: where the routing is known before the row is (experts picked by token id),
// the norm gathers the grouped GEMM's operand itself.  rows_idx picks input rows (output packed); x is then read but not
// written, so a row may be picked twice.
//
// One warp per row while a row is short enough for a warp's registers and there are enough rows to fill the machine,
// otherwise one CTA per row; either way the row stays in registers between the sum, the two statistics and the write.
#include "common.cuh"

namespace pg {

template <typename T>
struct ResLn {
  T* out; int ld_out;
  float* x;
  const T* y; int ldy; const int32_t* y_pos; int y_top; float y_w;
  const int64_t* ids; const T* table; long long vocab; int emb_mode;
  const T* vec;
  const T* w; const T* b; float eps, out_scale;
  const int32_t* rows_idx; const int32_t* out_pos; int out_top;
  int rows, D;
  int* err_flag;
};

template <typename T> __device__ __forceinline__ void load4(const T* p, float* f);
template <> __device__ __forceinline__ void load4<float>(const float* p, float* f) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
}
template <> __device__ __forceinline__ void load4<bf16>(const bf16* p, float* f) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  f[0] = __uint_as_float(u.x << 16); f[1] = __uint_as_float(u.x & 0xffff0000u);
  f[2] = __uint_as_float(u.y << 16); f[3] = __uint_as_float(u.y & 0xffff0000u);
}
template <> __device__ __forceinline__ void load4<f16>(const f16* p, float* f) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const __half2* h = reinterpret_cast<const __half2*>(&u);
  const float2 a = __half22float2(h[0]), b = __half22float2(h[1]);
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
}
template <typename T> __device__ __forceinline__ void store4(T* p, const float* f) {
  if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  } else {
    T t[4] = {from_f<T>(f[0]), from_f<T>(f[1]), from_f<T>(f[2]), from_f<T>(f[3])};
    *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(t);
  }
}

// TPR threads per row (32: a warp, several rows per CTA; otherwise the whole CTA), NV groups of four columns per thread.
template <typename T, int TPR, int NV>
__global__ void __launch_bounds__(256) residual_layernorm_kernel(ResLn<T> p) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int per_cta = blockDim.x / TPR, tid = threadIdx.x % TPR;
  const int r = blockIdx.x * per_cta + threadIdx.x / TPR;
  if (r >= p.rows) return;                          // whole warps (or no thread of a CTA) leave
  const int src = p.rows_idx ? p.rows_idx[r] : r;
  float* xr = p.x + (size_t)src * p.D;
  const T* er = nullptr;
  if (p.emb_mode) {
    const int64_t id = p.ids[src];
    if (id >= 0 && id < p.vocab) er = p.table + (size_t)id * p.D;
    else if (tid == 0 && p.err_flag) *p.err_flag = 1;
  }
  float v[NV][4];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (tid + i * TPR) * 4;
#pragma unroll
    for (int k = 0; k < 4; ++k) v[i][k] = 0.f;
    if (c < p.D && p.emb_mode != PG_EMB_INIT) load4<float>(xr + c, v[i]);
  }
  auto add_row = [&](const T* row, float wgt) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (tid + i * TPR) * 4;
      if (c < p.D) {
        float f[4];
        load4<T>(row + c, f);
#pragma unroll
        for (int k = 0; k < 4; ++k) v[i][k] = fmaf(wgt, f[k], v[i][k]);
      }
    }
  };
  if (p.y && !p.y_pos) add_row(p.y + (size_t)src * p.ldy, 1.f);
  if (p.y && p.y_pos)
    for (int k = 0; k < p.y_top; ++k) {
      const int pos = p.y_pos[(size_t)src * p.y_top + k];
      if (pos >= 0) add_row(p.y + (size_t)pos * p.ldy, p.y_w);
    }
  if (er) add_row(er, 1.f);
  if (p.vec) add_row(p.vec, 1.f);
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (tid + i * TPR) * 4;
    if (c >= p.D) continue;
    if (!p.rows_idx && (p.y || p.emb_mode || p.vec)) store4<float>(xr + c, v[i]);
    s += (v[i][0] + v[i][1]) + (v[i][2] + v[i][3]);
  }
  if (!p.out) return;
  s = TPR == 32 ? warp_sum(s) : block_sum(s, red);
  const float mean = s / (float)p.D;
  float q = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    if ((tid + i * TPR) * 4 >= p.D) continue;
#pragma unroll
    for (int k = 0; k < 4; ++k) { const float d = v[i][k] - mean; q = fmaf(d, d, q); }
  }
  q = TPR == 32 ? warp_sum(q) : block_sum(q, red);
  const float inv = 1.f / sqrtf(q / (float)p.D + p.eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (tid + i * TPR) * 4;
    if (c >= p.D) continue;
    float w[4], b[4], o[4];
    load4<T>(p.w + c, w);
    load4<T>(p.b + c, b);
#pragma unroll
    for (int k = 0; k < 4; ++k) o[k] = ((v[i][k] - mean) * inv * w[k] + b[k]) * p.out_scale;
    if (!p.out_pos) {
      store4<T>(p.out + (size_t)r * p.ld_out + c, o);
    } else {
      for (int k = 0; k < p.out_top; ++k) {
        const int pos = p.out_pos[(size_t)src * p.out_top + k];
        if (pos >= 0) store4<T>(p.out + (size_t)pos * p.ld_out + c, o);
      }
    }
  }
}

// Any width and alignment: the row in shared memory, one CTA per row.
template <typename T>
__global__ void __launch_bounds__(256) residual_layernorm_any_kernel(ResLn<T> p) {
  extern __shared__ float row[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x, src = p.rows_idx ? p.rows_idx[r] : r;
  float* xr = p.x + (size_t)src * p.D;
  const T* er = nullptr;
  if (p.emb_mode) {
    const int64_t id = p.ids[src];
    if (id >= 0 && id < p.vocab) er = p.table + (size_t)id * p.D;
    else if (threadIdx.x == 0 && p.err_flag) *p.err_flag = 1;
  }
  float s = 0.f;
  for (int c = threadIdx.x; c < p.D; c += blockDim.x) {
    float v = p.emb_mode != PG_EMB_INIT ? xr[c] : 0.f;
    if (p.y && !p.y_pos) v += to_f<T>(p.y[(size_t)src * p.ldy + c]);
    if (p.y && p.y_pos)
      for (int k = 0; k < p.y_top; ++k) {
        const int pos = p.y_pos[(size_t)src * p.y_top + k];
        if (pos >= 0) v = fmaf(p.y_w, to_f<T>(p.y[(size_t)pos * p.ldy + c]), v);
      }
    if (er) v += to_f<T>(er[c]);
    if (p.vec) v += to_f<T>(p.vec[c]);
    if (!p.rows_idx && (p.y || p.emb_mode || p.vec)) xr[c] = v;
    row[c] = v;
    s += v;
  }
  if (!p.out) return;
  const float mean = block_sum(s, red) / (float)p.D;
  float q = 0.f;
  for (int c = threadIdx.x; c < p.D; c += blockDim.x) { const float d = row[c] - mean; q = fmaf(d, d, q); }
  const float inv = 1.f / sqrtf(block_sum(q, red) / (float)p.D + p.eps);
  for (int c = threadIdx.x; c < p.D; c += blockDim.x) {
    const T o = from_f<T>(((row[c] - mean) * inv * to_f<T>(p.w[c]) + to_f<T>(p.b[c])) * p.out_scale);
    if (!p.out_pos) {
      p.out[(size_t)r * p.ld_out + c] = o;
    } else {
      for (int k = 0; k < p.out_top; ++k) {
        const int pos = p.out_pos[(size_t)src * p.out_top + k];
        if (pos >= 0) p.out[(size_t)pos * p.ld_out + c] = o;
      }
    }
  }
}

template <typename T>
static int launch_res_ln(const ResLn<T>& p, cudaStream_t st) {
  auto aligned = [](const void* q, size_t n) { return ((uintptr_t)q % n) == 0; };
  const size_t a4 = 4 * sizeof(T);
  const bool vec = p.D % 4 == 0 && aligned(p.x, 16) && (!p.y || (p.ldy % 4 == 0 && aligned(p.y, a4))) &&
                   (!p.emb_mode || aligned(p.table, a4)) && (!p.vec || aligned(p.vec, a4)) &&
                   (!p.out || (p.ld_out % 4 == 0 && aligned(p.out, a4) && aligned(p.w, a4) && aligned(p.b, a4)));
  const char* what = "residual_layernorm";
  if (vec && p.D <= 1024 && p.rows > 296) {          // measured at 8192 rows: a warp per row up to 1024 columns, ...
    const dim3 grid(cdiv(p.rows, 4)), block(128);
    if (p.D <= 512) return launch_pdl(what, residual_layernorm_kernel<T, 32, 4>, grid, block, 0, st, p);
    return launch_pdl(what, residual_layernorm_kernel<T, 32, 8>, grid, block, 0, st, p);
  }
  if (vec && p.D <= 256 * 4 * 16) {
    const dim3 grid(p.rows), block(256);
    // ... 128 threads per row up to 2048 (0.34 against 0.55 ms with a warp per row of 2048)
    if (p.rows > 296 && p.D <= 2048) return launch_pdl(what, residual_layernorm_kernel<T, 128, 4>, grid, dim3(128), 0, st, p);
    if (p.D <= 1024) return launch_pdl(what, residual_layernorm_kernel<T, 256, 1>, grid, block, 0, st, p);
    if (p.D <= 2048) return launch_pdl(what, residual_layernorm_kernel<T, 256, 2>, grid, block, 0, st, p);
    if (p.D <= 4096) return launch_pdl(what, residual_layernorm_kernel<T, 256, 4>, grid, block, 0, st, p);
    return launch_pdl(what, residual_layernorm_kernel<T, 256, 16>, grid, block, 0, st, p);
  }
  const size_t smem = sizeof(float) * (size_t)p.D;
  PG_REQUIRE(smem <= 200 * 1024, "residual_layernorm: rows of %d columns do not fit shared memory", p.D);
  return launch_pdl(what, residual_layernorm_any_kernel<T>, dim3(p.rows), dim3(256), smem, st, p);
}

// ------------------------------------------------------------------ key rows into the paged pool
// Columns [k_col0, k_col0 + cols) of token t's projection row -> the pool row of (tok_slot, tok_pos), unchanged.
template <typename T, int V>
__global__ void cache_append_kernel(T* __restrict__ pool, int ld_pool, const T* __restrict__ proj, int ld, int k_col0, int cols,
                                    const int32_t* __restrict__ page_table, int pt_stride, int page_size,
                                    const int32_t* __restrict__ tok_slot, const int32_t* __restrict__ tok_pos, long long n) {
  pdl_launch_dependents();
  pdl_wait();
  const int per = cols / V;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < n * per; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / per;
    const int c = (int)(i - t * per) * V, pos = tok_pos[t];
    const size_t row = (size_t)page_table[(size_t)tok_slot[t] * pt_stride + pos / page_size] * page_size + pos % page_size;
    const T* s = proj + t * ld + k_col0 + c;
    T* d = pool + row * ld_pool + c;
    if constexpr (V * sizeof(T) == 16) *reinterpret_cast<uint4*>(d) = *reinterpret_cast<const uint4*>(s);
    else *d = *s;
  }
}

}  // namespace pg

using namespace pg;

extern "C" int pg_residual_layernorm(void* out, int ld_out, float* x, const void* y, int ldy, const int32_t* y_pos, int y_top,
                                     float y_w, const int64_t* ids, const void* table, long long vocab, int emb_mode,
                                     const void* vec, const void* w, const void* b, float eps, float out_scale,
                                     const int32_t* rows_idx, const int32_t* out_pos, int out_top, int rows, int D,
                                     int* err_flag, int dtype, void* stream) {
  if (rows <= 0) return PG_OK;
  PG_REQUIRE(x && D > 0, "residual_layernorm: a residual stream is needed");
  PG_REQUIRE(!out || (w && b && ld_out >= D), "residual_layernorm: a normed output needs weight, bias and rows of %d columns", D);
  PG_REQUIRE(emb_mode == PG_EMB_NONE || ((emb_mode == PG_EMB_INIT || emb_mode == PG_EMB_ADD) && ids && table),
             "residual_layernorm: embedding mode %d", emb_mode);
  PG_REQUIRE(!y || ldy >= D, "residual_layernorm: sublayer rows of %d columns", ldy);
  PG_REQUIRE(!y_pos || (y && y_top >= 1), "residual_layernorm: expert rows without an output");
  PG_REQUIRE(!out_pos || (out && out_top >= 1 && !rows_idx), "residual_layernorm: expert places take all rows");
  PG_DISPATCH_DTYPE(dtype, T, {
    const ResLn<T> p = {(T*)out, ld_out, x, (const T*)y, ldy, y_pos, y_top, y_w, ids, (const T*)table, vocab, emb_mode,
                        (const T*)vec, (const T*)w, (const T*)b, eps, out_scale, rows_idx, out_pos, out_top, rows, D, err_flag};
    return launch_res_ln<T>(p, (cudaStream_t)stream);
  });
  return PG_OK;
}

extern "C" int pg_cache_append(void* pool, int ld_pool, const void* proj, int ld, int k_col0, int cols, const int32_t* page_table,
                               int pt_stride, int page_size, const int32_t* tok_slot, const int32_t* tok_pos, int n_tokens,
                               int dtype, void* stream) {
  if (n_tokens <= 0) return PG_OK;
  PG_REQUIRE(pool && proj && page_table && tok_slot && tok_pos && page_size > 0 && cols > 0 && ld_pool >= cols,
             "cache_append: pool and token map");
  PG_DISPATCH_DTYPE(dtype, T, {
    constexpr int V = Vec<T>::N;
    const bool vec = cols % V == 0 && ld % V == 0 && ld_pool % V == 0 && k_col0 % V == 0 && ((uintptr_t)pool % 16) == 0 &&
                     ((uintptr_t)proj % 16) == 0;
    const long long work = (long long)n_tokens * (vec ? cols / V : cols);
    const int blocks = (int)((work + 255) / 256 < 148 * 16 ? (work + 255) / 256 : 148 * 16);
    if (vec)
      return launch_pdl("cache_append", cache_append_kernel<T, V>, dim3(blocks), dim3(256), 0, (cudaStream_t)stream, (T*)pool,
                        ld_pool, (const T*)proj, ld, k_col0, cols, page_table, pt_stride, page_size, tok_slot, tok_pos,
                        (long long)n_tokens);
    return launch_pdl("cache_append", cache_append_kernel<T, 1>, dim3(blocks), dim3(256), 0, (cudaStream_t)stream, (T*)pool,
                      ld_pool, (const T*)proj, ld, k_col0, cols, page_table, pt_stride, page_size, tok_slot, tok_pos,
                      (long long)n_tokens);
  });
  return PG_OK;
}
