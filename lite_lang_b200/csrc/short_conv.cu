// Short causal convolutions over time, one filter a channel, and the norm that one of them follows.
//
//   conv(u)_t = sum_j w[j] u_(t - taps + 1 + j)        (j = 0 .. taps - 1; u before the request's start is zero)
//
//   norm_conv    the pre-norm of a sublayer over a float32 residual, fused with the residual sum before it and with
//                the convolution after it:  r <- r + (outputs pending);  h = r / sqrt(mean(r^2) + eps) * w;
//                out = h + conv(h).  Without taps it is the norm alone (of chosen rows: the last norm).
//   short_conv   the convolution of a projection's rows; the channels behind the first `q_w` may go straight into the
//                paged cache as keys and values.
//
// A request's last taps - 1 inputs are part of its state.  The record (float32, zeroed when the request's slot is
// opened) has two halves of [taps - 1][channels] (oldest first) and behind them two integers: how many tokens of the
// request stood before each half was left.  A step reads the half whose number is the request's context length and
// writes the other one, so the CTAs of one launch may read and write a request's record in any order, and a step
// that is run again at the same context gives the same result.
//
// All arithmetic is float32; sums run in an order that depends on the sizes only, and what a step brings is read as
// what earlier steps left, so where a prompt is cut does not show.
#include "common.cuh"

#define SC_ANY 5          // taps are a run-time number (more than four)

struct ConvRecord {
  float* state;           // record of request slot s at state + s * stride
  long stride;
  int write;              // 0: a run-step that only reads
  const int* token_req;   // entry of each token
  const int* cu_q;        // first token of each entry
  const int* ctx_len;     // tokens of the request before this step
  const int* req_slot;    // the request's slot, -1: padding
  int single;             // every entry brings one token: token t is entry t (two look-ups less in a row)
};

// What a token has to know of its entry
struct ConvToken {
  int first, last, ctx, slot;
  int rd;                 // the half to read
};
__device__ __forceinline__ ConvToken conv_token(const ConvRecord& c, int t, int halves) {
  ConvToken k;
  const int e = c.single ? t : c.token_req[t];
  k.slot = e >= 0 ? c.req_slot[e] : -1;
  k.ctx = e >= 0 ? c.ctx_len[e] : 0;
  k.first = k.last = t;
  if (!c.single && k.slot >= 0) {
    k.first = c.cu_q[e];
    k.last = c.cu_q[e + 1] - 1;
  }
  k.rd = 0;
  if (k.slot >= 0) {
    const int* tag = reinterpret_cast<const int*>(c.state + (size_t)k.slot * c.stride + halves);
    k.rd = tag[0] == k.ctx ? 0 : 1;
  }
  return k;
}

template <typename T, int VEC> __device__ __forceinline__ void sc_load(float (&v)[VEC], const T* p) {
  if constexpr (VEC == 1) {
    v[0] = to_f32<T>(p[0]);
  } else if constexpr (sizeof(T) == 4) {
#pragma unroll
    for (int i = 0; i < VEC; i += 4) {
      const float4 f = *reinterpret_cast<const float4*>(p + i);
      v[i] = f.x;
      v[i + 1] = f.y;
      v[i + 2] = f.z;
      v[i + 3] = f.w;
    }
  } else {
    unsigned u[VEC / 2];
    if constexpr (VEC == 8) {
      const uint4 q = *reinterpret_cast<const uint4*>(p);
      u[0] = q.x;
      u[1] = q.y;
      u[2] = q.z;
      u[3] = q.w;
    } else {
      const uint2 q = *reinterpret_cast<const uint2*>(p);
      u[0] = q.x;
      u[1] = q.y;
    }
#pragma unroll
    for (int i = 0; i < VEC / 2; ++i) {
      const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u[i]));
      v[2 * i] = f.x;
      v[2 * i + 1] = f.y;
    }
  }
}
template <typename T, int VEC> __device__ __forceinline__ void sc_store(T* p, const float (&v)[VEC]) {
  if constexpr (VEC == 1) {
    p[0] = from_f32<T>(v[0]);
  } else if constexpr (sizeof(T) == 4) {
#pragma unroll
    for (int i = 0; i < VEC; i += 4)
      *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
  } else {
    unsigned u[VEC / 2];
#pragma unroll
    for (int i = 0; i < VEC / 2; ++i) {
      const __nv_bfloat162 h = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
      u[i] = *reinterpret_cast<const unsigned*>(&h);
    }
    if constexpr (VEC == 8) *reinterpret_cast<uint4*>(p) = make_uint4(u[0], u[1], u[2], u[3]);
    else *reinterpret_cast<uint2*>(p) = make_uint2(u[0], u[1]);
  }
}

// The record after the step, as far as token t's channels c .. c + VEC - 1 (values `now`) decide it: one of the last
// `hist` tokens leaves its values; the last one also moves up what an entry shorter than that keeps of the half read.
template <int VEC>
__device__ __forceinline__ void conv_leave(const ConvRecord& rec, const ConvToken& k, int t, int hist, int channels, int c,
                                           const float (&now)[VEC]) {
  const int back = k.last - t;
  if (back >= hist && t != k.last) return;
  float* base = rec.state + (size_t)k.slot * rec.stride;
  float* dst = base + (size_t)(1 - k.rd) * hist * channels;
  if (back < hist) sc_store<float, VEC>(dst + (size_t)(hist - 1 - back) * channels + c, now);
  if (t == k.last) {
    const int L = k.last - k.first + 1;
    const float* src = base + (size_t)k.rd * hist * channels;
    for (int i = 0; i + L < hist; ++i) {
      float x[VEC];
      sc_load<float, VEC>(x, src + (size_t)(i + L) * channels + c);
      sc_store<float, VEC>(dst + (size_t)i * channels + c, x);
    }
    if (c == 0) reinterpret_cast<int*>(base + (size_t)2 * hist * channels)[1 - k.rd] = k.ctx + L;
  }
}

// ---------------------------------------------------------------------------------------------------------
// norm_conv
// ---------------------------------------------------------------------------------------------------------
struct NormConvParams {
  void* out;              // T [n, W]
  float* res_out;         // float32 [tokens, W] or null: where the summed residual goes.  It may be `res` itself only
                          // without a convolution (a CTA reads rows of tokens that another CTA owns)
  const float* res;       // float32 [tokens, W]
  const void* delta;      // T [tokens, W], or null
  const float* partial;   // float32 [parts][tokens, W], or null
  int parts;
  long part_stride;
  const void* rows_in;    // T [tokens, W] times rows_w[token], or null
  const float* rows_w;
  const float* extra;     // float32 [tokens, W], or null
  const float* w;         // the norm's factor a channel
  float eps;
  const float* conv_w;    // float32 [taps][W]
  int taps;
  ConvRecord rec;
  const int* rows;        // without a convolution: the tokens to norm, or null
  int n, W, C, segs;      // rows of `out`; tokens a CTA; pieces a row's sum is made of
};

// Any sizes: the rows of a few tokens (and those before them) wait in shared memory between the norm and the convolution.
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(512) norm_conv_kernel(const NormConvParams p) {
  constexpr bool CONV = TAPS > 0;
  constexpr int U = 4;                              // loads of a row in flight a lane
  extern __shared__ __align__(16) float sc_smem[];
  __shared__ ConvToken tok_s[16];
  const int taps = TAPS == SC_ANY ? p.taps : TAPS;
  const int hist = CONV ? taps - 1 : 0;
  const int W = p.W, C = p.C, segs = p.segs;
  float* rowv = sc_smem;                            // [C + hist][W]: the summed residual rows
  float* inv_s = rowv + (size_t)(C + hist) * W;     // [C + hist]
  float* red = inv_s + C + hist;                    // [C + hist][segs]
  LL_PDL_TRIGGER();
  LL_PDL_WAIT();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nwarps = blockDim.x >> 5;
  const int t0 = blockIdx.x * C, nt = min(C, p.n - t0);
  int from = t0;                                    // the first row this CTA needs
  if (CONV) {
    if (tid < nt) tok_s[tid] = conv_token(p.rec, t0 + tid, 2 * hist * W);
    const int e = p.rec.single ? -1 : p.rec.token_req[t0];
    from = max(e >= 0 ? p.rec.cu_q[e] : t0, t0 - hist);
  }
  const int vecs = W / VEC, per = (vecs + segs - 1) / segs;
  for (int it = warp; it < (hist + nt) * segs; it += nwarps) {
    const int r = it / segs, s = it - r * segs;
    const int t = t0 - hist + r;
    if (t < from) continue;
    const int tok = (!CONV && p.rows) ? p.rows[t] : t;
    const size_t off = (size_t)tok * W;
    const int end = min(vecs, (s + 1) * per);
    const float pw = p.rows_in ? p.rows_w[tok] : 0.f;
    const bool own = r >= hist && p.res_out != nullptr;
    float ss = 0.f;
    for (int v0 = s * per + lane; v0 < end; v0 += 32 * U) {
      float a[U][VEC], d[U][VEC];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int v = v0 + 32 * u;
#pragma unroll
        for (int i = 0; i < VEC; ++i) a[u][i] = d[u][i] = 0.f;
        if (v < end) {
          sc_load<float, VEC>(a[u], p.res + off + (size_t)v * VEC);
          if (p.delta) sc_load<T, VEC>(d[u], reinterpret_cast<const T*>(p.delta) + off + (size_t)v * VEC);
        }
      }
      if (p.partial) {
        for (int q = 0; q < p.parts; ++q) {
          const float* par = p.partial + (size_t)q * p.part_stride + off;
#pragma unroll
          for (int u = 0; u < U; ++u) {
            const int v = v0 + 32 * u;
            if (v < end) {
              float x[VEC];
              sc_load<float, VEC>(x, par + (size_t)v * VEC);
#pragma unroll
              for (int i = 0; i < VEC; ++i) d[u][i] += x[i];
            }
          }
        }
      }
      if (p.rows_in) {
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int v = v0 + 32 * u;
          if (v < end) {
            float x[VEC];
            sc_load<T, VEC>(x, reinterpret_cast<const T*>(p.rows_in) + off + (size_t)v * VEC);
#pragma unroll
            for (int i = 0; i < VEC; ++i) d[u][i] = fmaf(pw, x[i], d[u][i]);
          }
        }
      }
      if (p.extra) {
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int v = v0 + 32 * u;
          if (v < end) {
            float x[VEC];
            sc_load<float, VEC>(x, p.extra + off + (size_t)v * VEC);
#pragma unroll
            for (int i = 0; i < VEC; ++i) d[u][i] += x[i];
          }
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int v = v0 + 32 * u;
        if (v < end) {
#pragma unroll
          for (int i = 0; i < VEC; ++i) {
            a[u][i] += d[u][i];
            ss = fmaf(a[u][i], a[u][i], ss);
          }
          sc_store<float, VEC>(rowv + (size_t)r * W + (size_t)v * VEC, a[u]);
          if (own) sc_store<float, VEC>(p.res_out + off + (size_t)v * VEC, a[u]);
        }
      }
    }
    ss = warp_sum(ss);
    if (lane == 0) red[r * segs + s] = ss;
  }
  __syncthreads();
  if (tid < hist + nt && t0 - hist + tid >= from) {
    float ss = 0.f;
    for (int s = 0; s < segs; ++s) ss += red[tid * segs + s];
    inv_s[tid] = 1.0f / sqrtf(ss / (float)W + p.eps);
  }
  __syncthreads();
  T* out = reinterpret_cast<T*>(p.out);
  for (int v = tid; v < vecs; v += blockDim.x) {
    const int c = v * VEC;
    float w[VEC];
    sc_load<float, VEC>(w, p.w + c);
    float cw[(CONV && TAPS != SC_ANY) ? TAPS : 1][VEC];
    if constexpr (CONV && TAPS != SC_ANY) {
#pragma unroll
      for (int j = 0; j < TAPS; ++j) sc_load<float, VEC>(cw[j], p.conv_w + (size_t)j * W + c);
    }
    for (int i = 0; i < nt; ++i) {
      const int t = t0 + i, r = hist + i;
      float now[VEC], y[VEC];
      sc_load<float, VEC>(now, rowv + (size_t)r * W + c);
      const float inv = inv_s[r];
#pragma unroll
      for (int x = 0; x < VEC; ++x) {
        now[x] = now[x] * inv * w[x];
        y[x] = now[x];
      }
      if constexpr (CONV) {
        const ConvToken& k = tok_s[i];
        auto tap = [&](int j, const float (&f)[VEC]) {
          const int d = taps - 1 - j;               // how far back this tap looks
          float h[VEC];
          if (d == 0) {
#pragma unroll
            for (int x = 0; x < VEC; ++x) h[x] = now[x];
          } else if (t - d >= k.first) {
            sc_load<float, VEC>(h, rowv + (size_t)(r - d) * W + c);
            const float iv = inv_s[r - d];
#pragma unroll
            for (int x = 0; x < VEC; ++x) h[x] = h[x] * iv * w[x];
          } else if (k.slot >= 0) {                 // an input of an earlier step
            sc_load<float, VEC>(h, p.rec.state + (size_t)k.slot * p.rec.stride +
                                       ((size_t)k.rd * hist + (hist + t - k.first - d)) * W + c);
          } else {
#pragma unroll
            for (int x = 0; x < VEC; ++x) h[x] = 0.f;
          }
#pragma unroll
          for (int x = 0; x < VEC; ++x) y[x] = fmaf(f[x], h[x], y[x]);
        };
        if constexpr (TAPS == SC_ANY) {
          for (int j = 0; j < taps; ++j) {
            float f[VEC];
            sc_load<float, VEC>(f, p.conv_w + (size_t)j * W + c);
            tap(j, f);
          }
        } else {
#pragma unroll
          for (int j = 0; j < TAPS; ++j) tap(j, cw[j]);
        }
        if (k.slot >= 0 && p.rec.write) conv_leave<VEC>(p.rec, k, t, hist, W, c, now);
      }
      sc_store<T, VEC>(out + (size_t)t * W + c, y);
    }
  }
}

// The usual sizes (rows of up to 4,096 numbers, a multiple of four; up to four taps): a CTA walks a run of tokens, a
// thread keeps its four channels' last inputs, filters and norm weights in registers, and the rows of the next NW_AHEAD
// tokens are on their way to shared memory by cp.async while a row is summed (a thread reads back what it copied
// itself, so the copies need no barrier).  A row costs one barrier and is read once, but for the taps - 1 rows before a
// CTA's first token, which are normed again for the convolution.
#define NW_MAX_THREADS 1024
#define NW_AHEAD 4

template <int BYTES> __device__ __forceinline__ void nw_copy(unsigned dst, const void* src) {
  if constexpr (BYTES == 16)
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
  else
    asm volatile("cp.async.ca.shared.global [%0], [%1], %2;" ::"r"(dst), "l"(src), "n"(BYTES) : "memory");
}

template <typename T, int TAPS>
__global__ void __launch_bounds__(NW_MAX_THREADS) norm_conv_walk_kernel(const NormConvParams p) {
  constexpr int HIST = TAPS - 1, TB = 4 * (int)sizeof(T);
  constexpr int HN = HIST > 0 ? HIST : 1;
  extern __shared__ __align__(16) float sc_smem[];      // [NW_AHEAD][residual 16 | pending TB | rows TB][threads]
  __shared__ float red[2][32];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nthreads = blockDim.x, nwarps = nthreads >> 5;
  const int W = p.W, c = tid * 4;
  const bool active = c < W;
  // (the weights do not depend on the kernel before: they are on their way before the wait for it)
  float w[4] = {0.f, 0.f, 0.f, 0.f}, cw[TAPS][4];
  if (active) sc_load<float, 4>(w, p.w + c);
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {
    cw[j][0] = cw[j][1] = cw[j][2] = cw[j][3] = 0.f;
    if (active) sc_load<float, 4>(cw[j], p.conv_w + (size_t)j * W + c);
  }
  LL_PDL_TRIGGER();
  LL_PDL_WAIT();
  const int t0 = blockIdx.x * p.C, t1 = min(p.n, t0 + p.C);
  char* const ring = reinterpret_cast<char*>(sc_smem);
  const int stage = nthreads * (16 + 2 * TB);
  const int o_res = tid * 16, o_del = nthreads * 16 + tid * TB, o_row = nthreads * (16 + TB) + tid * TB;
  auto fetch = [&](int t) {                             // one group a token, empty behind the last
    if (active && t < t1) {
      const size_t off = (size_t)t * W + c;
      const unsigned dst = (unsigned)__cvta_generic_to_shared(ring + (t & (NW_AHEAD - 1)) * stage);
      nw_copy<16>(dst + o_res, p.res + off);
      if (p.delta) nw_copy<TB>(dst + o_del, reinterpret_cast<const T*>(p.delta) + off);
      if (p.rows_in) nw_copy<TB>(dst + o_row, reinterpret_cast<const T*>(p.rows_in) + off);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // rows that no entry of the CTA's first token needs are copied too where that saves a look-up first
  int from = max(t0 - HIST, 0);
  if (p.rec.single) from = t0;
#pragma unroll
  for (int i = 0; i < NW_AHEAD - 1; ++i) fetch(from + i);
  ConvToken k = conv_token(p.rec, t0, 2 * HIST * W);
  const int need = max(k.first, t0 - HIST);
  float h[HN][4];
#pragma unroll
  for (int i = 0; i < HN; ++i) h[i][0] = h[i][1] = h[i][2] = h[i][3] = 0.f;
  for (int t = from; t < t1; ++t) {
    fetch(t + NW_AHEAD - 1);
    asm volatile("cp.async.wait_group %0;" ::"n"(NW_AHEAD - 1) : "memory");
    if (t < need) continue;                             // (the same for all threads)
    if (t > k.last) k = conv_token(p.rec, t, 2 * HIST * W);
    const size_t off = (size_t)t * W + c;
    float v[4] = {0.f, 0.f, 0.f, 0.f};
    if (active) {
      const char* st = ring + (t & (NW_AHEAD - 1)) * stage;
      float d[4] = {0.f, 0.f, 0.f, 0.f}, x[4];
      sc_load<float, 4>(v, reinterpret_cast<const float*>(st + o_res));
      if (p.delta) {
        sc_load<T, 4>(d, reinterpret_cast<const T*>(st + o_del));
      } else if (p.partial) {
        const float* par = p.partial + off;
#pragma unroll 4
        for (int s = 0; s < p.parts; ++s) {
          sc_load<float, 4>(x, par + (size_t)s * p.part_stride);
#pragma unroll
          for (int i = 0; i < 4; ++i) d[i] += x[i];
        }
      }
      if (p.rows_in) {
        sc_load<T, 4>(x, reinterpret_cast<const T*>(st + o_row));
        const float pw = p.rows_w[t];
#pragma unroll
        for (int i = 0; i < 4; ++i) d[i] = fmaf(pw, x[i], d[i]);
      }
      if (p.extra) {
        sc_load<float, 4>(x, p.extra + off);
#pragma unroll
        for (int i = 0; i < 4; ++i) d[i] += x[i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) v[i] += d[i];
      if (t >= t0 && p.res_out) sc_store<float, 4>(p.res_out + off, v);
      if (HIST > 0 && t == k.first) {                   // the inputs of earlier steps (zeros at the request's start);
        const float* base = p.rec.state + (size_t)max(k.slot, 0) * p.rec.stride + c;   // needed behind the barrier only
#pragma unroll
        for (int i = 0; i < HIST; ++i) {
          h[i][0] = h[i][1] = h[i][2] = h[i][3] = 0.f;
          if (k.slot >= 0) sc_load<float, 4>(h[i], base + (size_t)(k.rd * HIST + i) * W);
        }
      }
    }
    const float ss = warp_sum(fmaf(v[0], v[0], v[1] * v[1]) + fmaf(v[2], v[2], v[3] * v[3]));
    float* slot = red[t & 1];                           // (two sets: a warp may be a row ahead of another's reads)
    if (lane == 0) slot[warp] = ss;
    __syncthreads();
    const float inv = 1.0f / sqrtf(warp_sum(lane < nwarps ? slot[lane] : 0.f) / (float)W + p.eps);
    if (!active) continue;
    float now[4], y[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      now[i] = v[i] * inv * w[i];
      y[i] = now[i];
    }
    if (t >= t0) {
#pragma unroll
      for (int j = 0; j < HIST; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) y[i] = fmaf(cw[j][i], h[j][i], y[i]);
#pragma unroll
      for (int i = 0; i < 4; ++i) y[i] = fmaf(cw[TAPS - 1][i], now[i], y[i]);
      sc_store<T, 4>(reinterpret_cast<T*>(p.out) + off, y);
      if (k.slot >= 0 && p.rec.write) conv_leave<4>(p.rec, k, t, HIST, W, c, now);
    }
#pragma unroll
    for (int j = 0; j + 1 < HIST; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) h[j][i] = h[j + 1][i];
#pragma unroll
    for (int i = 0; i < 4; ++i) h[HN - 1][i] = now[i];
  }
  asm volatile("cp.async.wait_all;" ::: "memory");
}

template <typename T, int TAPS>
static int nw_launch(NormConvParams p, int sms, cudaStream_t stream) {
  const int threads = (p.W / 4 + 31) / 32 * 32;
  const int slots = sms * (threads <= 512 ? 2 : 1);     // CTAs that are resident at once
  p.C = (p.n + slots - 1) / slots;
  const size_t smem = (size_t)NW_AHEAD * threads * (16 + 8 * sizeof(T));
  cudaFuncSetAttribute(norm_conv_walk_kernel<T, TAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  ll_launch(norm_conv_walk_kernel<T, TAPS>, dim3((p.n + p.C - 1) / p.C), dim3(threads), smem, stream, p);
  return LL_LAUNCH_RESULT();
}

template <typename T>
static int nw_taps(const NormConvParams& p, int sms, cudaStream_t stream) {
  switch (p.taps) {
    case 1: return nw_launch<T, 1>(p, sms, stream);
    case 2: return nw_launch<T, 2>(p, sms, stream);
    case 3: return nw_launch<T, 3>(p, sms, stream);
    default: return nw_launch<T, 4>(p, sms, stream);
  }
}

static size_t nc_smem(int W, int rows, int segs) { return sizeof(float) * ((size_t)rows * W + rows + (size_t)rows * segs); }

template <typename T, int VEC, int TAPS>
static int nc_launch(NormConvParams p, int sms, cudaStream_t stream) {
  const int hist = TAPS == 0 ? 0 : p.taps - 1;
  // tokens a CTA: one while that fills the device at most twice, up to eight for long portions (the rows before a
  // CTA's first token are normed again), as many as leave room for two CTAs an SM
  int C = (p.n + 2 * sms - 1) / (2 * sms);
  C = C < 1 ? 1 : C > 8 ? 8 : C;
  while (C > 1 && nc_smem(p.W, C + hist, 4) > 100 * 1024) --C;
  p.C = C;
  p.segs = C > 1 ? 4 : 8;
  const size_t smem = nc_smem(p.W, C + hist, p.segs);
  if (smem > 220 * 1024) return (int)cudaErrorInvalidValue;
  if (smem > 40 * 1024)
    cudaFuncSetAttribute(norm_conv_kernel<T, VEC, TAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  ll_launch(norm_conv_kernel<T, VEC, TAPS>, dim3((p.n + C - 1) / C), dim3(C > 1 ? 512 : 256), smem, stream, p);
  return LL_LAUNCH_RESULT();
}

template <typename T, int VEC>
static int nc_taps(const NormConvParams& p, int sms, cudaStream_t stream) {
  switch (p.conv_w == nullptr ? 0 : p.taps) {
    case 0: return nc_launch<T, VEC, 0>(p, sms, stream);
    case 1: return nc_launch<T, VEC, 1>(p, sms, stream);
    case 2: return nc_launch<T, VEC, 2>(p, sms, stream);
    case 3: return nc_launch<T, VEC, 3>(p, sms, stream);
    case 4: return nc_launch<T, VEC, 4>(p, sms, stream);
    default: return nc_launch<T, VEC, SC_ANY>(p, sms, stream);
  }
}

// out [n, W] of T.  conv_w (float32 [taps][W], or null: the norm alone); the arrays of a step (token_req ... req_slot)
// and the record are needed with it only.  rows (without a convolution): out[i] = norm of token rows[i].
extern "C" int ll_norm_conv(int dtype, void* out, float* res_out, const float* res, const void* delta,
                            const float* partial, int parts, long part_stride, const void* rows_in, const float* rows_w,
                            const float* extra, const float* w, float eps, const float* conv_w, int taps, float* state,
                            long state_stride, int write_state, const int* token_req, const int* cu_q,
                            const int* ctx_len, const int* req_slot, int single, const int* rows, int n, int W, int sms,
                            cudaStream_t stream) {
  if (n <= 0) return 0;
  if (W <= 0 || sms <= 0 || (conv_w != nullptr && (taps < 1 || taps > 64 || state == nullptr || rows != nullptr || res_out == res)) ||
      (rows_in != nullptr && rows_w == nullptr) || (partial != nullptr && parts < 1))
    return (int)cudaErrorInvalidValue;
  NormConvParams p;
  p.out = out;
  p.res_out = res_out;
  p.res = res;
  p.delta = delta;
  p.partial = partial;
  p.parts = parts;
  p.part_stride = part_stride;
  p.rows_in = rows_in;
  p.rows_w = rows_w;
  p.extra = extra;
  p.w = w;
  p.eps = eps;
  p.conv_w = conv_w;
  p.taps = taps;
  p.rec = {state, state_stride, write_state, token_req, cu_q, ctx_len, req_slot, single};
  p.rows = rows;
  p.n = n;
  p.W = W;
  p.C = p.segs = 1;
  // (all bases come from an allocator that aligns them well; rows of a multiple of four numbers then start on 16-byte
  // boundaries, and 8-byte ones of bfloat16)
  const bool v4 = (W % 4) == 0 && (part_stride % 4) == 0 && (state_stride % 4) == 0;
  if (v4 && conv_w != nullptr && taps <= 4 && W <= 4 * NW_MAX_THREADS)
    LL_DISPATCH_DTYPE(dtype, return nw_taps<T>(p, sms, stream));
  LL_DISPATCH_DTYPE(dtype, return v4 ? nc_taps<T, 4>(p, sms, stream) : nc_taps<T, 1>(p, sms, stream));
}

// ---------------------------------------------------------------------------------------------------------
// short_conv
// ---------------------------------------------------------------------------------------------------------
struct ShortConvParams {
  const void* x;          // T rows of x_stride, the first C numbers of each
  long x_stride;
  const float* w;         // float32 [taps][C]
  int taps, C;
  ConvRecord rec;
  void* out;              // T rows of out_stride: channels below out_w
  long out_stride;
  int out_w;
  int add;                // out = x + conv(x)
  // channels q_w .. q_w + k_w - 1 are keys (heads of hd), the rest values (heads of vd): into the cache plane
  const int* slot_map;    // null: no store
  void* k_cache;          // [pages, nkv, page_size, hd]
  void* v_cache;          // [pages, nkv, page_size, vd]
  int q_w, k_w, hd, vd, nkv, page_size;
  long num_slots;
  int* status;
  int n;                  // tokens
};

#define SC_TY 8
template <typename T, int VEC> struct ScRaw { T v[VEC]; };
template <typename T, int VEC> __device__ __forceinline__ void sc_load_raw(ScRaw<T, VEC>& r, const T* p) {
  if constexpr (VEC * sizeof(T) == 16) *reinterpret_cast<uint4*>(r.v) = *reinterpret_cast<const uint4*>(p);
  else r.v[0] = p[0];
}

// A thread works on VEC channels of NT neighbouring tokens: their rows and the taps - 1 before them are asked for at once.
template <typename T, int VEC, int TAPS, int NT>
__global__ void __launch_bounds__(32 * SC_TY) short_conv_kernel(const ShortConvParams p) {
  constexpr int HIST = TAPS == SC_ANY ? 0 : TAPS - 1;   // (SC_ANY: older rows are read where they are used)
  const int taps = TAPS == SC_ANY ? p.taps : TAPS;
  const int hist = taps - 1;
  const int c = (blockIdx.x * 32 + threadIdx.x) * VEC;
  const int ta = (blockIdx.y * SC_TY + threadIdx.y) * NT;
  const bool active = c < p.C && ta < p.n;
  float cw[TAPS == SC_ANY ? 1 : TAPS][VEC];
  if constexpr (TAPS != SC_ANY) {
    if (active) {
#pragma unroll
      for (int j = 0; j < TAPS; ++j) sc_load<float, VEC>(cw[j], p.w + (size_t)j * p.C + c);
    }
  }
  LL_PDL_TRIGGER();
  LL_PDL_WAIT();
  if (!active) return;
  const T* x = reinterpret_cast<const T*>(p.x) + c;
  ScRaw<T, VEC> raw[NT + HIST];
#pragma unroll
  for (int i = 0; i < NT + HIST; ++i) {
    const int t = ta - HIST + i;
    // (a step of single tokens never reads another token's row)
    if (t >= 0 && t < p.n && !(p.rec.single && i < HIST)) sc_load_raw<T, VEC>(raw[i], x + (size_t)t * p.x_stride);
    else
#pragma unroll
      for (int k = 0; k < VEC; ++k) raw[i].v[k] = from_f32<T>(0.f);
  }
  ConvToken k = conv_token(p.rec, ta, 2 * hist * p.C);
#pragma unroll
  for (int n = 0; n < NT; ++n) {
    const int t = ta + n;
    if (t >= p.n) break;
    if (t > k.last) k = conv_token(p.rec, t, 2 * hist * p.C);
    float now[VEC], y[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      now[i] = to_f32<T>(raw[n + HIST].v[i]);
      y[i] = p.add ? now[i] : 0.f;
    }
    const float* rec = p.rec.state + (size_t)max(k.slot, 0) * p.rec.stride + (size_t)k.rd * hist * p.C + c;
    if constexpr (TAPS == SC_ANY) {
      for (int j = 0; j < taps; ++j) {
        const int d = hist - j;
        float f[VEC], h[VEC];
        sc_load<float, VEC>(f, p.w + (size_t)j * p.C + c);
        if (t - d >= k.first) {
          sc_load<T, VEC>(h, x + (size_t)(t - d) * p.x_stride);
        } else if (k.slot >= 0) {
          sc_load<float, VEC>(h, rec + (size_t)(hist + t - k.first - d) * p.C);
        } else {
#pragma unroll
          for (int i = 0; i < VEC; ++i) h[i] = 0.f;
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) y[i] = fmaf(f[i], h[i], y[i]);
      }
    } else {
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        const int d = TAPS - 1 - j;
        float h[VEC];
        if (t - d >= k.first) {
#pragma unroll
          for (int i = 0; i < VEC; ++i) h[i] = to_f32<T>(raw[n + HIST - d].v[i]);
        } else if (k.slot >= 0) {
          sc_load<float, VEC>(h, rec + (size_t)(HIST + t - k.first - d) * p.C);
        } else {
#pragma unroll
          for (int i = 0; i < VEC; ++i) h[i] = 0.f;
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) y[i] = fmaf(cw[j][i], h[i], y[i]);
      }
    }
    if (k.slot >= 0 && p.rec.write) conv_leave<VEC>(p.rec, k, t, hist, p.C, c, now);
    if (c < p.out_w) sc_store<T, VEC>(reinterpret_cast<T*>(p.out) + (size_t)t * p.out_stride + c, y);
    if (p.slot_map != nullptr && c >= p.q_w) {
      const int slot = p.slot_map[t];
      if (slot < 0) continue;
      if (slot >= p.num_slots) {
        set_status(p.status, LL_ERR_SLOT_RANGE);
        continue;
      }
      const int page = slot / p.page_size, place = slot - page * p.page_size;
      const int kc = c - p.q_w;
      if (kc < p.k_w) {
        const int h = kc / p.hd;
        sc_store<T, VEC>(reinterpret_cast<T*>(p.k_cache) + (((size_t)page * p.nkv + h) * p.page_size + place) * p.hd +
                             (kc - h * p.hd), y);
      } else {
        const int vc = kc - p.k_w, h = vc / p.vd;
        sc_store<T, VEC>(reinterpret_cast<T*>(p.v_cache) + (((size_t)page * p.nkv + h) * p.page_size + place) * p.vd +
                             (vc - h * p.vd), y);
      }
    }
  }
}

template <typename T, int VEC, int TAPS>
static int sc_launch(const ShortConvParams& p, int sms, cudaStream_t stream) {
  const int gx = (p.C + 32 * VEC - 1) / (32 * VEC);
  // a token a thread while the step is short, four (which keep their filters and share their rows) for long portions
  if ((long)p.n * gx >= (long)SC_TY * sms * 8)
    ll_launch(short_conv_kernel<T, VEC, TAPS, 4>, dim3(gx, (p.n + 4 * SC_TY - 1) / (4 * SC_TY)), dim3(32, SC_TY), 0,
              stream, p);
  else
    ll_launch(short_conv_kernel<T, VEC, TAPS, 1>, dim3(gx, (p.n + SC_TY - 1) / SC_TY), dim3(32, SC_TY), 0, stream, p);
  return LL_LAUNCH_RESULT();
}

template <typename T, int VEC>
static int sc_taps(const ShortConvParams& p, int sms, cudaStream_t stream) {
  switch (p.taps) {
    case 1: return sc_launch<T, VEC, 1>(p, sms, stream);
    case 2: return sc_launch<T, VEC, 2>(p, sms, stream);
    case 3: return sc_launch<T, VEC, 3>(p, sms, stream);
    case 4: return sc_launch<T, VEC, 4>(p, sms, stream);
    default: return sc_launch<T, VEC, SC_ANY>(p, sms, stream);
  }
}

// x: the first C numbers of rows of x_stride; out: channels below out_w.  slot_map (or null): the channels from q_w on
// go into a cache plane, k_w of keys (heads of hd), then values (heads of vd).
extern "C" int ll_short_conv(int dtype, void* out, long out_stride, int out_w, const void* x, long x_stride, int C,
                             const float* w, int taps, int add, float* state, long state_stride, int write_state,
                             const int* token_req, const int* cu_q, const int* ctx_len, const int* req_slot,
                             int single, const int* slot_map, void* k_cache, void* v_cache, int q_w, int k_w, int hd, int vd, int nkv,
                             int page_size, long num_slots, int* status, int n, int sms, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (C <= 0 || taps < 1 || taps > 64 || state == nullptr || sms <= 0 || out_w < 0 || out_w > C ||
      (slot_map != nullptr && (hd <= 0 || vd <= 0 || nkv <= 0 || page_size <= 0 || q_w < 0 || k_w != nkv * hd ||
                               q_w + k_w + nkv * vd != C)))
    return (int)cudaErrorInvalidValue;
  ShortConvParams p;
  p.x = x;
  p.x_stride = x_stride;
  p.w = w;
  p.taps = taps;
  p.C = C;
  p.rec = {state, state_stride, write_state, token_req, cu_q, ctx_len, req_slot, single};
  p.out = out;
  p.out_stride = out_stride;
  p.out_w = out_w;
  p.add = add;
  p.slot_map = slot_map;
  p.k_cache = k_cache;
  p.v_cache = v_cache;
  p.q_w = q_w;
  p.k_w = k_w;
  p.hd = hd;
  p.vd = vd;
  p.nkv = nkv;
  p.page_size = page_size;
  p.num_slots = num_slots;
  p.status = status;
  p.n = n;
  const int v = dtype == LL_DTYPE_BF16 ? 8 : 4;
  const bool wide = C % v == 0 && x_stride % v == 0 && out_stride % v == 0 && out_w % v == 0 && state_stride % 4 == 0 &&
                    (uintptr_t)x % 16 == 0 && (uintptr_t)out % 16 == 0 &&
                    (slot_map == nullptr || (q_w % v == 0 && hd % v == 0 && vd % v == 0));
  if (dtype == LL_DTYPE_BF16) return wide ? sc_taps<bf16, 8>(p, sms, stream) : sc_taps<bf16, 1>(p, sms, stream);
  if (dtype == LL_DTYPE_F32) return wide ? sc_taps<float, 4>(p, sms, stream) : sc_taps<float, 1>(p, sms, stream);
  return (int)cudaErrorInvalidValue;
}
