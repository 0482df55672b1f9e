// Short causal convolutions over the projected queries and keys of an attention layer, for ragged token batches.
//
// Per token, from one fused projection row [.. q (H heads x dim) .. k (G x dim) ..] (the key columns behind the query columns):
//   q, k <- causal convolution over time per channel (the sequence's earlier rows: rows of this step, beyond that its state)
//   v    =  k as it leaves the convolution              (the values are the keys before norm and rotation)
//   q, k <- divided by the root mean square over ALL query (key) columns of the token, times a weight per column
//   q, k <- rotated by position over the first rot_dims columns of every head (pairs (i, i + rot_dims / 2))
// Queries go to q_out (packed), keys and values to the paged pools at (tok_slot, tok_pos).  Everything between the projection
// and the stores is fp32, one rounding.
//
// conv_qk_reg_kernel : up to 8 taps and 4096 columns, head sizes in groups of eight.  A CTA owns TOK consecutive rows; a thread
//                      owns two groups of four columns that the rotation pairs with one another (or eight unrotated ones) and
//                      walks the rows with the last taps - 1 inputs in registers, so that the convolved values never leave them:
//                      only the row statistics cross threads.  Sines and cosines once per row and pair, in shared memory.
// conv_qk_kernel     : any sizes.  The convolved rows stay in shared memory between the three steps, the rows that the taps
//                      share are served by L1.
//  The convolution's weights are [taps][columns] in the model dtype (last row: the current token), so
// that a thread's columns are one vector load per tap.  The state ([slots][state_len][state_cols] fp32, entry state_len - 1 the most
// recent) is kept by time_conv_state_kernel over a range of projection columns that starts where the queries do.
#include "common.cuh"

namespace pg {

template <typename T>
struct ConvQk {
  T* q_out;
  const T* proj; int ld, q_col0, k_off;            // the keys start k_off columns behind the queries
  int H, G, dim;
  const T* conv; int taps;                         // [taps][k_off + G * dim]
  const float* state; int state_len, state_cols;
  const T* q_w; const T* k_w; float eps;
  const float2* freq; int rot_dims;
  T* k_pool; T* v_pool;
  const int32_t* page_table; int pt_stride, page_size;
  const int32_t* tok_slot; const int32_t* tok_pos;
  int n_tokens;
};

template <typename T, int TOK, bool QUAD>
__global__ void __launch_bounds__(256) conv_qk_kernel(ConvQk<T> p) {
  extern __shared__ __align__(16) float sm[];      // [TOK][cols] convolved rows | [TOK][rot_dims / 2] (cos, sin)
  __shared__ float part[8][2 * TOK];
  __shared__ int bef[TOK], slot_of[TOK];
  pdl_launch_dependents();
  pdl_wait();
  const int K = p.taps - 1, t0 = blockIdx.x * TOK, nt = min(TOK, p.n_tokens - t0);
  const int nq = p.H * p.dim, nk = p.G * p.dim, cols = p.k_off + nk, half = p.rot_dims >> 1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  float2* cs = reinterpret_cast<float2*>(sm + TOK * ((cols + 3) & ~3));
  const int row_f = (cols + 3) & ~3;
  if (threadIdx.x < nt) {
    const int t = t0 + threadIdx.x, slot = p.tok_slot[t];
    int b = 0;                                     // rows of the same sequence right before this one, up to K
    while (b < K && t - b - 1 >= 0 && p.tok_slot[t - b - 1] == slot) ++b;
    bef[threadIdx.x] = b;
    slot_of[threadIdx.x] = slot;
  }
  for (int i = threadIdx.x; i < nt * half; i += blockDim.x) {
    const int tt = i / half, m = i - tt * half;
    const float2 f = p.freq[m];
    float s, c;
    rotary_sincos((float)p.tok_pos[t0 + tt], f.x, f.y, &s, &c);
    cs[tt * half + m] = make_float2(c, s);
  }
  __syncthreads();
  float sq[TOK], sk[TOK];
#pragma unroll
  for (int tt = 0; tt < TOK; ++tt) { sq[tt] = 0.f; sk[tt] = 0.f; }
  if constexpr (QUAD) {                            // four columns per thread
    for (int c = threadIdx.x * 4; c < cols; c += blockDim.x * 4) {
      if (c >= nq && c < p.k_off) continue;
      const bool is_k = c >= p.k_off;
      const T* src = p.proj + (size_t)t0 * p.ld + p.q_col0 + c;
      auto ld4 = [&](const T* q, float* f) {
        if constexpr (sizeof(T) == 4) {
          const float4 v = *reinterpret_cast<const float4*>(q);
          f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
        } else {
          const uint2 v = *reinterpret_cast<const uint2*>(q);
          const T* e = reinterpret_cast<const T*>(&v);
#pragma unroll
          for (int k = 0; k < 4; ++k) f[k] = to_f<T>(e[k]);
        }
      };
#pragma unroll
      for (int tt = 0; tt < TOK; ++tt) {
        if (tt >= nt) break;
        const T* w = p.conv + (size_t)K * cols + c;
        float acc[4], u[4], wf[4];
        ld4(src + (size_t)tt * p.ld, u);
        ld4(w, wf);
#pragma unroll
        for (int k = 0; k < 4; ++k) acc[k] = u[k] * wf[k];
        const int b = bef[tt];
        for (int j = 1; j <= K; ++j) {
          w -= cols;
          if (j <= b) {
            ld4(src + ((long long)tt - j) * p.ld, u);
          } else {
            const float* s = p.state + ((size_t)slot_of[tt] * p.state_len + (p.state_len - (j - b))) * p.state_cols + c;
#pragma unroll
            for (int k = 0; k < 4; ++k) u[k] = s[k];
          }
          ld4(w, wf);
#pragma unroll
          for (int k = 0; k < 4; ++k) acc[k] = fmaf(u[k], wf[k], acc[k]);
        }
        *reinterpret_cast<float4*>(sm + tt * row_f + c) = make_float4(acc[0], acc[1], acc[2], acc[3]);
        const float ss = (acc[0] * acc[0] + acc[1] * acc[1]) + (acc[2] * acc[2] + acc[3] * acc[3]);
        if (is_k) sk[tt] += ss; else sq[tt] += ss;
      }
    }
  } else {
    for (int c = threadIdx.x; c < cols; c += blockDim.x) {
      if (c >= nq && c < p.k_off) continue;
      const T* src = p.proj + (size_t)t0 * p.ld + p.q_col0 + c;
#pragma unroll
      for (int tt = 0; tt < TOK; ++tt) {
        if (tt >= nt) break;
        float acc = to_f<T>(src[(size_t)tt * p.ld]) * to_f<T>(p.conv[(size_t)K * cols + c]);
        const int b = bef[tt];
        for (int j = 1; j <= K; ++j) {
          const float u = j <= b ? to_f<T>(src[((long long)tt - j) * p.ld])
                                 : p.state[((size_t)slot_of[tt] * p.state_len + (p.state_len - (j - b))) * p.state_cols + c];
          acc = fmaf(u, to_f<T>(p.conv[(size_t)(K - j) * cols + c]), acc);
        }
        sm[tt * row_f + c] = acc;
        if (c >= p.k_off) sk[tt] += acc * acc; else sq[tt] += acc * acc;
      }
    }
  }
#pragma unroll
  for (int tt = 0; tt < TOK; ++tt) {
    const float a = warp_sum(sq[tt]), b = warp_sum(sk[tt]);
    if (lane == 0) { part[warp][2 * tt] = a; part[warp][2 * tt + 1] = b; }
  }
  __syncthreads();
#pragma unroll 1
  for (int tt = 0; tt < nt; ++tt) {
    float a = 0.f, b = 0.f;
    for (int w = 0; w < warps; ++w) { a += part[w][2 * tt]; b += part[w][2 * tt + 1]; }
    const float iq = p.q_w ? 1.f / sqrtf(a / (float)nq + p.eps) : 1.f, ik = p.k_w ? 1.f / sqrtf(b / (float)nk + p.eps) : 1.f;
    const int t = t0 + tt, pos = p.tok_pos[t];
    const size_t row = (size_t)p.page_table[(size_t)p.tok_slot[t] * p.pt_stride + pos / p.page_size] * p.page_size + pos % p.page_size;
    T* qd = p.q_out + (size_t)t * nq;
    T* kd = p.k_pool + row * nk;
    T* vd = p.v_pool + row * nk;
    const float* x = sm + tt * row_f;
    const float2* e = cs + tt * half;
    if constexpr (QUAD) {                          // dim and rot_dims / 2 in whole groups of four: a group never straddles a boundary
      for (int i = threadIdx.x * 4; i < nq + nk; i += blockDim.x * 4) {
        const bool is_k = i >= nq;
        const int li = is_k ? i - nq : i, c = li % p.dim;
        const float* xh = x + (is_k ? p.k_off : 0) + (li - c);
        const T* wv = is_k ? p.k_w : p.q_w;
        const T* wh = wv ? wv + (li - c) : nullptr;
        const float iv = is_k ? ik : iq;
        float o[4], u[4], w[4];
        const int pc = c < half ? c + half : c - half;   // the partner group, where c is rotated at all
#pragma unroll
        for (int k = 0; k < 4; ++k) u[k] = xh[c + k] * iv * (wh ? to_f<T>(wh[c + k]) : 1.f);
        if (c < p.rot_dims) {
#pragma unroll
          for (int k = 0; k < 4; ++k) w[k] = xh[pc + k] * iv * (wh ? to_f<T>(wh[pc + k]) : 1.f);
          const float2* ee = e + (c < half ? c : pc);
          const float sg = c < half ? -1.f : 1.f;
#pragma unroll
          for (int k = 0; k < 4; ++k) o[k] = u[k] * ee[k].x + sg * w[k] * ee[k].y;
        } else {
#pragma unroll
          for (int k = 0; k < 4; ++k) o[k] = u[k];
        }
        auto st4 = [&](T* d, const float* f) {
          if constexpr (sizeof(T) == 4) {
            *reinterpret_cast<float4*>(d) = make_float4(f[0], f[1], f[2], f[3]);
          } else {
            T v[4] = {from_f<T>(f[0]), from_f<T>(f[1]), from_f<T>(f[2]), from_f<T>(f[3])};
            *reinterpret_cast<uint2*>(d) = *reinterpret_cast<const uint2*>(v);
          }
        };
        st4((is_k ? kd : qd) + li, o);
        if (is_k) st4(vd + li, xh + c);
      }
    } else {
      for (int i = threadIdx.x; i < nq + nk; i += blockDim.x) {
        const bool is_k = i >= nq;
        const int li = is_k ? i - nq : i, c = li % p.dim;
        const float* xh = x + (is_k ? p.k_off : 0) + (li - c);
        const T* wv = is_k ? p.k_w : p.q_w;
        const T* wh = wv ? wv + (li - c) : nullptr;
        const float iv = is_k ? ik : iq;
        float o = xh[c] * iv * (wh ? to_f<T>(wh[c]) : 1.f);
        if (c < p.rot_dims) {
          const int pc = c < half ? c + half : c - half;
          const float w = xh[pc] * iv * (wh ? to_f<T>(wh[pc]) : 1.f);
          const float2 f = e[c < half ? c : pc];
          o = c < half ? o * f.x - w * f.y : o * f.x + w * f.y;
        }
        (is_k ? kd : qd)[li] = from_f<T>(o);
        if (is_k) vd[li] = from_f<T>(xh[c]);
      }
    }
  }
}

// Four consecutive elements as they lie in memory, and as floats.
template <typename T> struct Quad { typedef uint2 type; };
template <> struct Quad<float> { typedef float4 type; };
template <typename T> __device__ __forceinline__ typename Quad<T>::type cq_raw4(const T* q) {
  return *reinterpret_cast<const typename Quad<T>::type*>(q);
}
template <typename T> __device__ __forceinline__ void cq_unpack4(const typename Quad<T>::type& v, float* f) {
  const T* e = reinterpret_cast<const T*>(&v);
#pragma unroll
  for (int k = 0; k < 4; ++k) f[k] = to_f<T>(e[k]);
}
template <typename T> __device__ __forceinline__ void cq_load4(const T* q, float* f) { cq_unpack4<T>(cq_raw4<T>(q), f); }
template <typename T> __device__ __forceinline__ void cq_store4(T* d, const float* f) {
  if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(d) = make_float4(f[0], f[1], f[2], f[3]);
  } else {
    T v[4] = {from_f<T>(f[0]), from_f<T>(f[1]), from_f<T>(f[2]), from_f<T>(f[3])};
    *reinterpret_cast<uint2*>(d) = *reinterpret_cast<const uint2*>(v);
  }
}

// KM: the most rows back this instance keeps in registers (taps - 1 <= KM); THREADS: the most threads, MINB CTAs per SM
template <typename T, int TOK, int KM, int THREADS, int MINB>
__global__ void __launch_bounds__(THREADS, MINB) conv_qk_reg_kernel(ConvQk<T> p) {
  typedef typename Quad<T>::type R4;
  extern __shared__ __align__(16) float2 cs[];       // [TOK][rot_dims / 2] (cos, sin)
  __shared__ float part[16][2 * TOK];
  __shared__ int bef[TOK], slot_of[TOK];
  __shared__ size_t row_of[TOK];
  pdl_launch_dependents();
  pdl_wait();
  const int K = p.taps - 1, t0 = blockIdx.x * TOK, nt = min(TOK, p.n_tokens - t0);
  const int nq = p.H * p.dim, nk = p.G * p.dim, cols = p.k_off + nk, half = p.rot_dims >> 1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  if (threadIdx.x < nt) {
    const int t = t0 + threadIdx.x, slot = p.tok_slot[t], pos = p.tok_pos[t];
    int b = 0;                                       // rows of the same sequence right before this one, up to K
    while (b < K && t - b - 1 >= 0 && p.tok_slot[t - b - 1] == slot) ++b;
    bef[threadIdx.x] = b;
    slot_of[threadIdx.x] = slot;
    row_of[threadIdx.x] = (size_t)p.page_table[(size_t)slot * p.pt_stride + pos / p.page_size] * p.page_size + pos % p.page_size;
  }
  for (int i = threadIdx.x; i < nt * half; i += blockDim.x) {
    const int tt = i / half, m = i - tt * half;
    const float2 f = p.freq[m];
    float s, c;
    rotary_sincos((float)p.tok_pos[t0 + tt], f.x, f.y, &s, &c);
    cs[i] = make_float2(c, s);
  }
  __syncthreads();
  // the thread's two groups of columns: (c, c + half) of a head's rotated part, or (c, c + 4) behind it
  const int per_head = p.dim / 8, head = threadIdx.x / per_head, it = threadIdx.x - head * per_head, rot_items = half / 4;
  const bool live = head < p.H + p.G, is_k = head >= p.H, turned = it < rot_items;
  const int ca = turned ? it * 4 : p.rot_dims + (it - rot_items) * 8, cb = turned ? ca + half : ca + 4;
  const int hb = is_k ? (head - p.H) * p.dim : head * p.dim;         // the head's first column among the query (key) columns
  const int c0 = (is_k ? p.k_off : 0) + hb;
  float v[TOK][8], sq[TOK], sk[TOK];
#pragma unroll
  for (int tt = 0; tt < TOK; ++tt) { sq[tt] = 0.f; sk[tt] = 0.f; }
  if (live) {
    // the inputs stay packed in the model dtype (the state's entries are projected values too: the conversion is exact); all
    // rows of the tile are requested before the first one is used
    R4 w[KM + 1][2], prev[KM][2], cur[TOK][2];
    const T* src = p.proj + (size_t)t0 * p.ld + p.q_col0 + c0;
#pragma unroll
    for (int tt = 0; tt < TOK; ++tt) {
      const T* r = src + (size_t)min(tt, nt - 1) * p.ld;
      cur[tt][0] = cq_raw4<T>(r + ca);
      cur[tt][1] = cq_raw4<T>(r + cb);
    }
#pragma unroll
    for (int j = 1; j <= KM; ++j)
      if (j <= K && j <= bef[0]) {
        prev[j - 1][0] = cq_raw4<T>(src - (long long)j * p.ld + ca);
        prev[j - 1][1] = cq_raw4<T>(src - (long long)j * p.ld + cb);
      }
#pragma unroll
    for (int j = 0; j <= KM; ++j)
      if (j <= K) {
        const T* wr = p.conv + (size_t)(K - j) * cols + c0;
        w[j][0] = cq_raw4<T>(wr + ca);
        w[j][1] = cq_raw4<T>(wr + cb);
      }
#pragma unroll
    for (int tt = 0; tt < TOK; ++tt) {
      if (tt >= nt) break;
      const int b = bef[tt];
      if (b < K) {                                   // a sequence that starts in the step within K rows: from its state
#pragma unroll
        for (int j = 1; j <= KM; ++j)
          if (j <= K && j > b) {
            const float* s = p.state + ((size_t)slot_of[tt] * p.state_len + (p.state_len - (j - b))) * p.state_cols + c0;
            float f[8];
#pragma unroll
            for (int i = 0; i < 4; ++i) { f[i] = s[ca + i]; f[4 + i] = s[cb + i]; }
            cq_store4<T>(reinterpret_cast<T*>(&prev[j - 1][0]), f);
            cq_store4<T>(reinterpret_cast<T*>(&prev[j - 1][1]), f + 4);
          }
      }
      float ss = 0.f;
#pragma unroll
      for (int g = 0; g < 2; ++g) {
        float a[4], x[4], f[4];
        cq_unpack4<T>(cur[tt][g], x);
        cq_unpack4<T>(w[0][g], f);
#pragma unroll
        for (int i = 0; i < 4; ++i) a[i] = x[i] * f[i];
#pragma unroll
        for (int j = 1; j <= KM; ++j)
          if (j <= K) {
            cq_unpack4<T>(prev[j - 1][g], x);
            cq_unpack4<T>(w[j][g], f);
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = fmaf(x[i], f[i], a[i]);
          }
#pragma unroll
        for (int i = 0; i < 4; ++i) { v[tt][4 * g + i] = a[i]; ss = fmaf(a[i], a[i], ss); }
#pragma unroll
        for (int j = KM; j >= 2; --j)
          if (j <= K) prev[j - 1][g] = prev[j - 2][g];
        if (K >= 1) prev[0][g] = cur[tt][g];
      }
      if (is_k) sk[tt] = ss; else sq[tt] = ss;
    }
  }
#pragma unroll
  for (int tt = 0; tt < TOK; ++tt) {
    const float a = warp_sum(sq[tt]), b = warp_sum(sk[tt]);
    if (lane == 0) { part[warp][2 * tt] = a; part[warp][2 * tt + 1] = b; }
  }
  __syncthreads();
  if (!live) return;
  const T* wv = is_k ? p.k_w : p.q_w;
  float nw[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) nw[i] = 1.f;
  if (wv) { cq_load4<T>(wv + hb + ca, nw); cq_load4<T>(wv + hb + cb, nw + 4); }
#pragma unroll
  for (int tt = 0; tt < TOK; ++tt) {
    if (tt >= nt) break;
    float iv = 1.f;
    if (wv) {
      float s = 0.f;
      for (int x = 0; x < warps; ++x) s += part[x][2 * tt + (is_k ? 1 : 0)];
      iv = 1.f / sqrtf(s / (float)(is_k ? nk : nq) + p.eps);
    }
    T* d = (is_k ? p.k_pool + row_of[tt] * nk : p.q_out + (size_t)(t0 + tt) * nq) + hb;
    if (is_k) {
      T* vd = p.v_pool + row_of[tt] * nk + hb;
      cq_store4<T>(vd + ca, v[tt]);
      cq_store4<T>(vd + cb, v[tt] + 4);
    }
    float o[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) o[i] = v[tt][i] * iv * nw[i];
    if (turned) {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 e = cs[tt * half + ca + i];
        const float a = o[i], b = o[4 + i];
        o[i] = a * e.x - b * e.y;
        o[4 + i] = b * e.x + a * e.y;
      }
    }
    cq_store4<T>(d + ca, o);
    cq_store4<T>(d + cb, o + 4);
  }
}

template <typename T, int TOK, int KM, int THREADS, int MINB>
static int launch_conv_qk_reg(const ConvQk<T>& p, cudaStream_t st) {
  const int items = (p.H + p.G) * (p.dim / 8), threads = (items + 31) / 32 * 32;
  return launch_pdl("conv_qk_append", conv_qk_reg_kernel<T, TOK, KM, THREADS, MINB>, dim3(cdiv(p.n_tokens, TOK)), dim3(threads),
                    sizeof(float) * TOK * (size_t)p.rot_dims, st, p);
}

template <typename T, int TOK>
static int launch_conv_qk(const ConvQk<T>& p, bool quad, cudaStream_t st) {
  const int cols = p.k_off + p.G * p.dim;
  const size_t smem = sizeof(float) * TOK * ((size_t)((cols + 3) & ~3) + p.rot_dims);
  PG_REQUIRE(smem <= 200 * 1024, "conv_qk_append: %d query and key columns do not fit shared memory", cols);
  auto kern = quad ? conv_qk_kernel<T, TOK, true> : conv_qk_kernel<T, TOK, false>;
  return launch_pdl("conv_qk_append", kern, dim3(cdiv(p.n_tokens, TOK)), dim3(256), smem, st, p);
}

}  // namespace pg

using namespace pg;

extern "C" int pg_conv_qk_append(void* q_out, const void* proj, int ld, int q_col0, int n_heads, int k_col0, int n_kv_heads,
                                 int dim, const void* conv, int taps, const float* state, int state_len, int state_cols,
                                 const void* q_w, const void* k_w, float eps, const float* freq, int rot_dims, void* k_pool,
                                 void* v_pool, const int32_t* page_table, int pt_stride, int page_size,
                                 const int32_t* tok_slot, const int32_t* tok_pos, int n_tokens, int dtype, void* stream) {
  if (n_tokens <= 0) return PG_OK;
  PG_REQUIRE(q_out && proj && conv && k_pool && v_pool && page_table && tok_slot && tok_pos && page_size > 0,
             "conv_qk_append: operands, pools and token map");
  const int k_off = k_col0 - q_col0, cols = k_off + n_kv_heads * dim;
  PG_REQUIRE(n_heads > 0 && n_kv_heads > 0 && dim > 0 && k_off >= n_heads * dim, "conv_qk_append: the keys lie behind the queries");
  PG_REQUIRE(taps >= 1 && (taps == 1 || (state && state_len >= taps - 1 && state_cols >= cols)),
             "conv_qk_append: %d taps over a state of %d rows of %d columns", taps, state_len, state_cols);
  PG_REQUIRE(rot_dims >= 0 && rot_dims <= dim && rot_dims % 2 == 0 && (rot_dims == 0 || freq),
             "conv_qk_append: %d rotated columns of %d (even, with a frequency table)", rot_dims, dim);
  PG_DISPATCH_DTYPE(dtype, T, {
    const ConvQk<T> p = {(T*)q_out, (const T*)proj, ld, q_col0, k_off, n_heads, n_kv_heads, dim, (const T*)conv, taps, state, state_len,
                         state_cols, (const T*)q_w, (const T*)k_w, eps, (const float2*)freq, rot_dims, (T*)k_pool, (T*)v_pool,
                         page_table, pt_stride, page_size, tok_slot, tok_pos, n_tokens};
    const size_t a4 = 4 * sizeof(T);
    const bool quad = dim % 4 == 0 && rot_dims % 8 == 0 && ld % 4 == 0 && q_col0 % 4 == 0 && k_off % 4 == 0 &&
                      ((uintptr_t)proj % a4) == 0 && ((uintptr_t)q_out % a4) == 0 && ((uintptr_t)k_pool % a4) == 0 &&
                      ((uintptr_t)v_pool % a4) == 0 && ((uintptr_t)conv % a4) == 0;
    const bool reg = quad && dim % 8 == 0 && taps <= 8 && (n_heads + n_kv_heads) * (dim / 8) <= 512 && rot_dims <= 1024 &&
                     ((uintptr_t)q_w % a4) == 0 && ((uintptr_t)k_w % a4) == 0;
    const int items = (n_heads + n_kv_heads) * (dim / 8);
    if (reg && taps <= 4 && n_tokens > 296)
      return items <= 320 ? launch_conv_qk_reg<T, 4, 3, 320, 2>(p, (cudaStream_t)stream) : launch_conv_qk_reg<T, 4, 3, 512, 1>(p, (cudaStream_t)stream);
    if (reg && taps <= 4) return launch_conv_qk_reg<T, 1, 3, 512, 1>(p, (cudaStream_t)stream);
    if (reg) return launch_conv_qk_reg<T, 1, 7, 512, 1>(p, (cudaStream_t)stream);
    if (n_tokens > 148 && (size_t)cols * 16 <= 96 * 1024) return launch_conv_qk<T, 4>(p, quad, (cudaStream_t)stream);
    return launch_conv_qk<T, 1>(p, quad, (cudaStream_t)stream);
  });
  return PG_OK;
}
