// Layers whose sublayers have a norm before and a norm behind them, over a float32 residual stream.
//
//   r   = residual + y / sqrt(mean(y^2) + eps) * wa + add        (y: a sublayer's output; add: one float32 row for all
//                                                                  tokens; both optional)
//   out = r / sqrt(mean(r^2) + eps) * wb                          (what the next sublayer reads), or without wb
//   out = r rounded to T                                          (for a product that reads the residual itself)
//
// in one pass: the output norm of one sublayer, the residual sum and the input norm of the next.  y comes as T
// [tokens, hidden], or as float32 partial sums [parts, tokens, hidden] of a product that was split over its inner
// dimension, which are added up in a fixed order and not rounded.  r is written back unrounded; with `rows` given only
// those rows are read and nothing is written back (the last norm before the logits).  A constant factor a channel on the
// output norm (a layer scale) is part of wa.  Everything is float32; out is rounded once.
//
// One block a row.  The row stays in registers between the sums (four neighbouring values an access, P accesses a
// thread, every load in flight before the first sum); sizes that do not fit that go through shared memory.  With few rows
// (EARLY) a row's latency counts: as many threads as give each one access, the weights asked for before the kernel before
// has ended.  With many rows the weights are read where they are used, which leaves registers for more rows an SM.
//
// `embed_norm`: the start of such a stream, out[t] = table[ids[t]] / sqrt(mean^2 + eps) * w in float32.
// `token_side_act`: g[t, j] <- gelu_tanh(g[t, j]) * table[ids[t], first + j] in place: a per-token table's part for one
// layer, gated by a projection of the residual.
#include "common.cuh"

template <typename T> __device__ __forceinline__ float4 sn_load4(const T* p);
template <> __device__ __forceinline__ float4 sn_load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 sn_load4<bf16>(const bf16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
template <typename T> __device__ __forceinline__ void sn_store4(T* p, float4 v);
template <> __device__ __forceinline__ void sn_store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void sn_store4<bf16>(bf16* p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<const unsigned*>(&a);
  u.y = *reinterpret_cast<const unsigned*>(&b);
  *reinterpret_cast<uint2*>(p) = u;
}
__device__ __forceinline__ float sn_sq(float4 v) { return (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w); }

template <typename T, int P, bool EARLY>
__global__ void __launch_bounds__(512)
sandwich_norm_kernel(T* __restrict__ out, float* __restrict__ residual, const T* __restrict__ y,
                     const float* __restrict__ partial, int parts, long part_stride, const float* __restrict__ wa,
                     float eps_a, const float* __restrict__ add, const float* __restrict__ wb, float eps_b, int hidden,
                     const int* __restrict__ rows, int write_residual) {
  __shared__ float scratch[32];
  const int tid = threadIdx.x, step = 4 * blockDim.x;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  auto weight = [&](const float* w, int i) { return w != nullptr && i < hidden ? sn_load4<float>(w + i) : zero; };
  float4 a4[EARLY ? P : 1], b4[EARLY ? P : 1], c4[EARLY ? P : 1];
  if (EARLY) {                     // (the weights do not depend on the kernel before)
#pragma unroll
    for (int p = 0; p < P; ++p) {
      const int i = 4 * tid + p * step;
      a4[p] = weight(wa, i);
      b4[p] = weight(wb, i);
      c4[p] = weight(add, i);
    }
  }
  LL_PDL_TRIGGER();
  LL_PDL_WAIT();
  const int r = rows ? rows[blockIdx.x] : (int)blockIdx.x;
  float* res = residual + (size_t)r * hidden;
  const bool has_y = y != nullptr || partial != nullptr;
  float4 v[P], x[P];
  float ss = 0.f;
#pragma unroll
  for (int p = 0; p < P; ++p) {
    const int i = 4 * tid + p * step;
    v[p] = x[p] = zero;
    if (i < hidden) {
      x[p] = sn_load4<float>(res + i);
      if (y) v[p] = sn_load4<T>(y + (size_t)r * hidden + i);
    }
  }
  if (partial) {
    for (int q = 0; q < parts; ++q)
#pragma unroll
      for (int p = 0; p < P; ++p) {
        const int i = 4 * tid + p * step;
        if (i < hidden) {
          const float4 u = sn_load4<float>(partial + (size_t)q * part_stride + (size_t)r * hidden + i);
          v[p].x += u.x, v[p].y += u.y, v[p].z += u.z, v[p].w += u.w;
        }
      }
  }
  float inv = 0.f;
  if (has_y) {
#pragma unroll
    for (int p = 0; p < P; ++p) ss += sn_sq(v[p]);
    inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)hidden + eps_a);
  }
  ss = 0.f;
#pragma unroll
  for (int p = 0; p < P; ++p) {
    const int i = 4 * tid + p * step;
    const float4 a = EARLY ? a4[EARLY ? p : 0] : weight(wa, i), c = EARLY ? c4[EARLY ? p : 0] : weight(add, i);
    x[p].x += v[p].x * inv * a.x + c.x;
    x[p].y += v[p].y * inv * a.y + c.y;
    x[p].z += v[p].z * inv * a.z + c.z;
    x[p].w += v[p].w * inv * a.w + c.w;
    ss += sn_sq(x[p]);
    if (write_residual && i < hidden) sn_store4<float>(res + i, x[p]);
  }
  if (out == nullptr) return;
  T* o = out + (size_t)blockIdx.x * hidden;
  float io = 1.0f;
  if (wb) io = 1.0f / sqrtf(block_sum(ss, scratch) / (float)hidden + eps_b);
#pragma unroll
  for (int p = 0; p < P; ++p) {
    const int i = 4 * tid + p * step;
    if (i < hidden) {
      float4 u = x[p];
      if (wb) {
        const float4 b = EARLY ? b4[EARLY ? p : 0] : weight(wb, i);
        u = make_float4(u.x * io * b.x, u.y * io * b.y, u.z * io * b.z, u.w * io * b.w);
      }
      sn_store4<T>(o + i, u);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(512)
sandwich_norm_any_kernel(T* __restrict__ out, float* __restrict__ residual, const T* __restrict__ y,
                         const float* __restrict__ partial, int parts, long part_stride, const float* __restrict__ wa,
                         float eps_a, const float* __restrict__ add, const float* __restrict__ wb, float eps_b, int hidden,
                         const int* __restrict__ rows, int write_residual) {
  extern __shared__ float row[];
  __shared__ float scratch[32];
  LL_PDL_TRIGGER();
  LL_PDL_WAIT();
  const int r = rows ? rows[blockIdx.x] : (int)blockIdx.x;
  float* res = residual + (size_t)r * hidden;
  const bool has_y = y != nullptr || partial != nullptr;
  float inv = 0.f, ss = 0.f;
  if (has_y) {
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
      float v = y ? to_f32<T>(y[(size_t)r * hidden + i]) : 0.f;
      if (partial)
        for (int q = 0; q < parts; ++q) v += partial[(size_t)q * part_stride + (size_t)r * hidden + i];
      row[i] = v;
      ss += v * v;
    }
    inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)hidden + eps_a);
  }
  ss = 0.f;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {       // (a thread's own places of `row`)
    float v = res[i];
    if (has_y) v += row[i] * inv * wa[i];
    if (add) v += add[i];
    row[i] = v;
    ss += v * v;
    if (write_residual) res[i] = v;
  }
  if (out == nullptr) return;
  float io = 1.0f;
  if (wb) io = 1.0f / sqrtf(block_sum(ss, scratch) / (float)hidden + eps_b);
  T* o = out + (size_t)blockIdx.x * hidden;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) o[i] = from_f32<T>(wb ? row[i] * io * wb[i] : row[i]);
}

// out: [n_out, hidden] of T or null; residual: float32 [tokens, hidden]; y: T [tokens, hidden], or `partial` float32
// [parts, tokens, hidden], or neither; wa (with y), add, wb: float32 [hidden]; rows: int32 [n_out] or null.
extern "C" int ll_sandwich_norm(int dtype, void* out, float* residual, const void* y, const float* partial, int parts,
                                long part_stride, const float* wa, float eps_a, const float* add, const float* wb,
                                float eps_b, int n_out, int hidden, const int* rows, int write_residual,
                                cudaStream_t stream) {
  if (n_out <= 0) return 0;
  if (hidden <= 0 || (y != nullptr && partial != nullptr) || ((y != nullptr || partial != nullptr) && wa == nullptr))
    return (int)cudaErrorInvalidValue;
  const uintptr_t ptrs = (uintptr_t)out | (uintptr_t)residual | (uintptr_t)y | (uintptr_t)partial | (uintptr_t)wa |
                         (uintptr_t)add | (uintptr_t)wb;
  if (hidden % 4 == 0 && ptrs % 16 == 0 && part_stride % 4 == 0 && hidden <= 512 * 4 * 4) {
    const int quads = hidden / 4;
    const bool early = n_out <= 296;
    const int most = early ? 512 : 256;
    int pieces = (quads + most - 1) / most;
    pieces = pieces <= 2 ? pieces : pieces <= 4 ? 4 : 8;
    const int threads = ((quads + pieces - 1) / pieces + 31) / 32 * 32;
#define SN_LAUNCH(P, E)                                                                                           \
  ll_launch(sandwich_norm_kernel<T, P, E>, dim3(n_out), dim3(threads), 0, stream, (T*)out, residual, (const T*)y,  \
            partial, parts, part_stride, wa, eps_a, add, wb, eps_b, hidden, rows, write_residual)
    LL_DISPATCH_DTYPE(dtype, {
      if (early && pieces == 1) SN_LAUNCH(1, true);
      else if (early && pieces == 2) SN_LAUNCH(2, true);
      else if (early) SN_LAUNCH(4, true);
      else if (pieces == 1) SN_LAUNCH(1, false);
      else if (pieces == 2) SN_LAUNCH(2, false);
      else if (pieces == 4) SN_LAUNCH(4, false);
      else SN_LAUNCH(8, false);
    });
#undef SN_LAUNCH
    return LL_LAUNCH_RESULT();
  }
  const size_t smem = sizeof(float) * (size_t)hidden;
  if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  const int threads = hidden >= 2048 ? 512 : hidden >= 512 ? 256 : 128;
  LL_DISPATCH_DTYPE(dtype, {
    if (smem > 48 * 1024)
      cudaFuncSetAttribute(sandwich_norm_any_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    ll_launch(sandwich_norm_any_kernel<T>, dim3(n_out), dim3(threads), smem, stream, (T*)out, residual, (const T*)y,
              partial, parts, part_stride, wa, eps_a, add, wb, eps_b, hidden, rows, write_residual);
  });
  return LL_LAUNCH_RESULT();
}

// ---------------------------------------------------------------------------------------------------------
// (VEC 4: rows of up to 4 x 256 x EN_PIECES numbers stay in registers)
#define EN_PIECES 4
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
embed_norm_kernel(float* __restrict__ out, const T* __restrict__ table, const int* __restrict__ ids,
                  const float* __restrict__ w, float eps, int hidden, int vocab, int* status) {
  __shared__ float scratch[32];
  LL_PDL_TRIGGER();
  LL_PDL_WAIT();
  const int id = ids[blockIdx.x];
  const bool ok = id >= 0 && id < vocab;
  if (!ok && threadIdx.x == 0) set_status(status, LL_ERR_TOKEN_RANGE);
  float* dst = out + (size_t)blockIdx.x * hidden;
  const T* src = table + (size_t)(ok ? id : 0) * hidden;
  float ss = 0.f;
  if (VEC == 4) {
    float4 v[EN_PIECES];
#pragma unroll
    for (int p = 0; p < EN_PIECES; ++p) {
      const int i = 4 * (threadIdx.x + p * 256);
      v[p] = (ok && i < hidden) ? sn_load4<T>(src + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += sn_sq(v[p]);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)hidden + eps);
#pragma unroll
    for (int p = 0; p < EN_PIECES; ++p) {
      const int i = 4 * (threadIdx.x + p * 256);
      if (i < hidden) {
        const float4 g = sn_load4<float>(w + i);
        sn_store4<float>(dst + i, make_float4(v[p].x * inv * g.x, v[p].y * inv * g.y, v[p].z * inv * g.z, v[p].w * inv * g.w));
      }
    }
    return;
  }
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
    const float v = ok ? to_f32<T>(src[i]) : 0.f;
    ss += v * v;
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)hidden + eps);
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) dst[i] = ok ? to_f32<T>(src[i]) * inv * w[i] : 0.f;
}

// An id outside [0, vocab) gives a row of zeros and sets the status word.
extern "C" int ll_embed_norm(int dtype, float* out, const void* table, const int* ids, const float* w, float eps,
                             int num_tokens, int hidden, int vocab, int* status, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (hidden <= 0 || vocab <= 0 || w == nullptr) return (int)cudaErrorInvalidValue;
  const bool wide = hidden % 4 == 0 && hidden <= 4 * 256 * EN_PIECES &&
                    ((uintptr_t)out | (uintptr_t)table | (uintptr_t)w) % 16 == 0;
  LL_DISPATCH_DTYPE(dtype, {
    if (wide)
      ll_launch(embed_norm_kernel<T, 4>, dim3(num_tokens), dim3(256), 0, stream, out, (const T*)table, ids, w, eps, hidden,
                vocab, status);
    else
      ll_launch(embed_norm_kernel<T, 1>, dim3(num_tokens), dim3(256), 0, stream, out, (const T*)table, ids, w, eps, hidden,
                vocab, status);
  });
  return LL_LAUNCH_RESULT();
}

// ---------------------------------------------------------------------------------------------------------
template <typename T, int VEC>
__global__ void token_side_act_kernel(T* __restrict__ g, long g_stride, const T* __restrict__ table, long table_stride,
                                      const int* __restrict__ ids, long total_vec, int dim, int vocab, int* status) {
  LL_PDL_TRIGGER();
  LL_PDL_WAIT();
  const int per_row = dim / VEC;
  const long step = (long)gridDim.x * blockDim.x;
  for (long idx = (long)blockIdx.x * blockDim.x + threadIdx.x; idx < total_vec; idx += step) {
    const long t = idx / per_row;
    const int j = (int)(idx - t * per_row) * VEC;
    const int id = ids[t];
    const bool ok = id >= 0 && id < vocab;
    if (!ok) set_status(status, LL_ERR_TOKEN_RANGE);
    T* gp = g + t * g_stride + j;
    const T* ep = table + (size_t)(ok ? id : 0) * table_stride + j;
    T v[VEC], e[VEC];
    if (VEC > 1) {
      *reinterpret_cast<uint4*>(v) = *reinterpret_cast<const uint4*>(gp);
      *reinterpret_cast<uint4*>(e) = *reinterpret_cast<const uint4*>(ep);
    } else {
      v[0] = gp[0];
      e[0] = ep[0];
    }
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = from_f32<T>(ok ? ll_gelu_tanh(to_f32<T>(v[i])) * to_f32<T>(e[i]) : 0.f);
    if (VEC > 1) *reinterpret_cast<uint4*>(gp) = *reinterpret_cast<const uint4*>(v);
    else gp[0] = v[0];
  }
}

// table: the first of the layer's columns (row stride table_stride, `vocab` rows).
extern "C" int ll_token_side_act(int dtype, void* g, long g_stride, const void* table, long table_stride, const int* ids,
                                 int num_tokens, int dim, int vocab, int sms, int* status, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (dim <= 0 || vocab <= 0) return (int)cudaErrorInvalidValue;
  const long most = (long)(sms > 0 ? sms : 148) * 16;
  LL_DISPATCH_DTYPE(dtype, {
    constexpr int VEC = 16 / (int)sizeof(T);
    const bool wide = dim % VEC == 0 && g_stride % VEC == 0 && table_stride % VEC == 0 && (uintptr_t)g % 16 == 0 &&
                      (uintptr_t)table % 16 == 0;
    const long total = (long)num_tokens * (wide ? dim / VEC : dim);
    const int threads = total >= 128 * 148 ? 256 : 64;
    const long want = (total + threads - 1) / threads;
    const dim3 grid((int)(want < most ? want : most));
    if (wide)
      ll_launch(token_side_act_kernel<T, VEC>, grid, dim3(threads), 0, stream, (T*)g, g_stride, (const T*)table,
                table_stride, ids, total, dim, vocab, status);
    else
      ll_launch(token_side_act_kernel<T, 1>, grid, dim3(threads), 0, stream, (T*)g, g_stride, (const T*)table,
                table_stride, ids, total, dim, vocab, status);
  });
  return LL_LAUNCH_RESULT();
}
