// mixers_streams.cu — several residual streams per token (their mixing, a sublayer's output on its way in, the next sublayer's normed
// input on its way out) and linear attention with a decay per key channel.  sm_100a only.  Streams, norms, decays and recurrent
// state are fp32; D only where a projection, an operand or a weight is stored.
#include "mixers.cuh"

#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <math.h>

#include "common.cuh"

namespace cake {
namespace mx {

#define MX_DISPATCH(dtype, ...)                               \
  do {                                                        \
    if ((dtype) == 2) { typedef float T; __VA_ARGS__; }       \
    else if ((dtype) == 1) { typedef __half T; __VA_ARGS__; } \
    else { typedef __nv_bfloat16 T; __VA_ARGS__; }            \
  } while (0)
#define MX_DONE(n)                     \
  do {                                 \
    if (launches) *launches += (n);    \
    return (int)cudaGetLastError();    \
  } while (0)

__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

template <typename T> __device__ __forceinline__ void load4(const T *s, float (&v)[4]) {
  const uint2 u = *reinterpret_cast<const uint2 *>(s);
  const float2 a = DT<T>::unpack2(u.x), b = DT<T>::unpack2(u.y);
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
template <> __device__ __forceinline__ void load4<float>(const float *s, float (&v)[4]) {
  const float4 f = *reinterpret_cast<const float4 *>(s);
  v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
}
template <typename T> __device__ __forceinline__ void store4(T *d, const float (&v)[4]) {
  *reinterpret_cast<uint2 *>(d) = make_uint2(pack2x<T>(v[0], v[1]), pack2x<T>(v[2], v[3]));
}
template <> __device__ __forceinline__ void store4<float>(float *d, const float (&v)[4]) {
  *reinterpret_cast<float4 *>(d) = make_float4(v[0], v[1], v[2], v[3]);
}

__device__ __forceinline__ float block_sum(float a, float *red /* [32] */) {
  a = warp_sum(a);
  const int w = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  if ((threadIdx.x & 31) == 0) red[w] = a;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < nw; i++) t += red[i];
  return t;
}

// ---------------------------------------------------------------------------------------------- stream mixing
// A CTA per token.  A thread owns the 16-byte pieces i, i + 256, ... of the width: it reads the piece of every stream and of the
// sublayer's output, writes every stream, and keeps only the read-out u of the piece in registers until the row's sum of squares
// is known.  S: the number of streams at compile time (the coefficients and a piece of every stream stay in registers).
template <typename T, int S, int NV>
__global__ void __launch_bounds__(256) stream_mix_kernel(const StreamMix p) {
  __shared__ float red[32];
  const int m = blockIdx.x, n4 = p.n / 4;
  const size_t src = p.rows ? (size_t)p.rows[m] : (size_t)m * p.row_mul + p.row_add;
  const float4 *x4 = reinterpret_cast<const float4 *>(p.x + src * S * p.n);
  float4 *xo4 = reinterpret_cast<float4 *>(p.x_out + (size_t)m * S * p.n);
  const float4 *a4 = reinterpret_cast<const float4 *>(p.a ? p.a + (size_t)m * p.n : nullptr);
  const bool write = p.mix != nullptr;
  float mix[S][S], out[S], in[S];
#pragma unroll
  for (int s = 0; s < S; s++) {
    in[s] = p.in ? DT<T>::to_f(reinterpret_cast<const T *>(p.in)[s]) : 1.f;
    out[s] = write ? p.mult * DT<T>::to_f(reinterpret_cast<const T *>(p.out)[s]) : 0.f;
#pragma unroll
    for (int t = 0; t < S; t++) mix[s][t] = write ? DT<T>::to_f(reinterpret_cast<const T *>(p.mix)[s * S + t]) : (s == t ? 1.f : 0.f);
  }
  float4 u[NV];
  float ss = 0.f;
#pragma unroll
  for (int v = 0; v < NV; v++) {
    const int i = threadIdx.x + 256 * v;
    u[v] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < n4) {
      float4 x[S];
#pragma unroll
      for (int s = 0; s < S; s++) x[s] = x4[(size_t)s * n4 + i];
      if (write) {
        float4 y = a4 ? a4[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        if (p.y)
          for (int k = 0; k < p.top; k++) {
            const size_t pr = (size_t)m * p.top + k;
            if (p.ids[pr] >= p.experts) continue;
            const float4 e = reinterpret_cast<const float4 *>(p.y + (size_t)p.pos_of[pr] * p.n)[i];
            y.x += e.x; y.y += e.y; y.z += e.z; y.w += e.w;
          }
#pragma unroll
        for (int t = 0; t < S; t++) {
          float4 r = make_float4(out[t] * y.x, out[t] * y.y, out[t] * y.z, out[t] * y.w);
#pragma unroll
          for (int s = 0; s < S; s++) {
            r.x = fmaf(mix[s][t], x[s].x, r.x); r.y = fmaf(mix[s][t], x[s].y, r.y);
            r.z = fmaf(mix[s][t], x[s].z, r.z); r.w = fmaf(mix[s][t], x[s].w, r.w);
          }
          xo4[(size_t)t * n4 + i] = r;
          u[v].x = fmaf(in[t], r.x, u[v].x); u[v].y = fmaf(in[t], r.y, u[v].y);
          u[v].z = fmaf(in[t], r.z, u[v].z); u[v].w = fmaf(in[t], r.w, u[v].w);
        }
      } else {
#pragma unroll
        for (int s = 0; s < S; s++) {
          u[v].x = fmaf(in[s], x[s].x, u[v].x); u[v].y = fmaf(in[s], x[s].y, u[v].y);
          u[v].z = fmaf(in[s], x[s].z, u[v].z); u[v].w = fmaf(in[s], x[s].w, u[v].w);
        }
      }
    }
    ss = fmaf(u[v].x, u[v].x, ss); ss = fmaf(u[v].y, u[v].y, ss); ss = fmaf(u[v].z, u[v].z, ss); ss = fmaf(u[v].w, u[v].w, ss);
  }
  if (!p.h) return;
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)p.n + p.eps);
  const T *w = reinterpret_cast<const T *>(p.w);
  T *h = reinterpret_cast<T *>(p.h) + (size_t)m * p.n;
#pragma unroll
  for (int v = 0; v < NV; v++) {
    const int i = threadIdx.x + 256 * v;
    if (i >= n4) continue;
    float g[4];
    load4<T>(w + 4 * i, g);
    const float r[4] = {u[v].x * inv * g[0], u[v].y * inv * g[1], u[v].z * inv * g[2], u[v].w * inv * g[3]};
    store4<T>(h + 4 * i, r);
  }
}
// any width and up to MAX_STREAMS streams: entry by entry, the read-out waits in shared memory
template <typename T>
__global__ void __launch_bounds__(256) stream_mix_any_kernel(const StreamMix p) {
  extern __shared__ float us[];  // [n]
  __shared__ float red[32], mix[MAX_STREAMS * MAX_STREAMS], out[MAX_STREAMS], in[MAX_STREAMS];
  const int m = blockIdx.x, S = p.streams;
  const size_t src = p.rows ? (size_t)p.rows[m] : (size_t)m * p.row_mul + p.row_add;
  const bool write = p.mix != nullptr;
  for (int i = threadIdx.x; i < S * S; i += blockDim.x)
    mix[i] = write ? DT<T>::to_f(reinterpret_cast<const T *>(p.mix)[i]) : (i / S == i % S ? 1.f : 0.f);
  for (int i = threadIdx.x; i < S; i += blockDim.x) {
    in[i] = p.in ? DT<T>::to_f(reinterpret_cast<const T *>(p.in)[i]) : 1.f;
    out[i] = write ? p.mult * DT<T>::to_f(reinterpret_cast<const T *>(p.out)[i]) : 0.f;
  }
  __syncthreads();
  const float *xr = p.x + src * S * p.n;
  float ss = 0.f;
  for (int i = threadIdx.x; i < p.n; i += blockDim.x) {
    float x[MAX_STREAMS], u = 0.f;
#pragma unroll
    for (int s = 0; s < MAX_STREAMS; s++) x[s] = s < S ? xr[(size_t)s * p.n + i] : 0.f;
    if (write) {
      float y = p.a ? p.a[(size_t)m * p.n + i] : 0.f;
      if (p.y)
        for (int k = 0; k < p.top; k++) {
          const size_t pr = (size_t)m * p.top + k;
          if (p.ids[pr] < p.experts) y += p.y[(size_t)p.pos_of[pr] * p.n + i];
        }
      for (int t = 0; t < S; t++) {
        float r = out[t] * y;
#pragma unroll
        for (int s = 0; s < MAX_STREAMS; s++)
          if (s < S) r = fmaf(mix[s * S + t], x[s], r);
        p.x_out[((size_t)m * S + t) * p.n + i] = r;
        u = fmaf(in[t], r, u);
      }
    } else {
#pragma unroll
      for (int s = 0; s < MAX_STREAMS; s++)
        if (s < S) u = fmaf(in[s], x[s], u);
    }
    us[i] = u;
    ss = fmaf(u, u, ss);
  }
  if (!p.h) return;
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)p.n + p.eps);
  const T *w = reinterpret_cast<const T *>(p.w);
  for (int i = threadIdx.x; i < p.n; i += blockDim.x)  // a thread revisits the entries it wrote
    reinterpret_cast<T *>(p.h)[(size_t)m * p.n + i] = DT<T>::from_f(us[i] * inv * DT<T>::to_f(w[i]));
}
template <typename T, int S> static bool launch_stream_mix(cudaStream_t st, const StreamMix &p) {
  if (p.n <= 1024) stream_mix_kernel<T, S, 1><<<p.M, 256, 0, st>>>(p);
  else if (p.n <= 2048) stream_mix_kernel<T, S, 2><<<p.M, 256, 0, st>>>(p);
  else if (p.n <= 4096) stream_mix_kernel<T, S, 4><<<p.M, 256, 0, st>>>(p);
  else if (p.n <= 8192) stream_mix_kernel<T, S, 8><<<p.M, 256, 0, st>>>(p);
  else return false;
  return true;
}
int stream_mix(cudaStream_t st, int dtype, const StreamMix &p, uint64_t *launches) {
  if (p.M < 1 || p.n < 1 || p.streams < 1 || p.streams > MAX_STREAMS || !p.x || (p.h && !p.w) || (!p.h && !p.mix) ||
      (p.mix && (!p.out || !p.x_out || p.rows || p.row_mul != 1 || p.row_add != 0)) || (p.y && (!p.ids || !p.pos_of || p.top < 1)))
    return (int)cudaErrorInvalidValue;
  const bool vec = p.n % 4 == 0 && (((uintptr_t)p.x | (uintptr_t)p.x_out | (uintptr_t)p.a | (uintptr_t)p.y | (uintptr_t)p.h | (uintptr_t)p.w) & 15) == 0;
  bool done = false;
  if (vec) MX_DISPATCH(dtype, {
    switch (p.streams) {
      case 1: done = launch_stream_mix<T, 1>(st, p); break;
      case 2: done = launch_stream_mix<T, 2>(st, p); break;
      case 3: done = launch_stream_mix<T, 3>(st, p); break;
      case 4: done = launch_stream_mix<T, 4>(st, p); break;
      case 5: done = launch_stream_mix<T, 5>(st, p); break;
      case 6: done = launch_stream_mix<T, 6>(st, p); break;
      case 8: done = launch_stream_mix<T, 8>(st, p); break;
      default: break;
    }
  });
  if (done) MX_DONE(1);
  const size_t smem = (size_t)p.n * sizeof(float);
  if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  MX_DISPATCH(dtype, {
    if (smem > 40 * 1024) {
      cudaError_t e = cudaFuncSetAttribute(stream_mix_any_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return (int)e;
    }
    stream_mix_any_kernel<T><<<p.M, 256, smem, st>>>(p);
  });
  MX_DONE(1);
}

// ---------------------------------------------------------------------------------------------- decays per key channel
// A CTA: 128 channels x CD_TT tokens.  The tokens' low-rank rows are staged once (rank-major, so that one broadcast load feeds four
// tokens); a thread owns a channel.
constexpr int CD_TT = 16;
template <typename T>
__global__ void __launch_bounds__(128) channel_decay_kernel(const ChannelDecay p) {
  extern __shared__ __align__(16) float us[];  // [rank][CD_TT]
  const int m0 = blockIdx.y * CD_TT, nt = min(CD_TT, p.M - m0), ch = blockIdx.x * 128 + threadIdx.x;
  for (int i = threadIdx.x; i < CD_TT * p.rank; i += 128) {
    const int t = i / p.rank, j = i % p.rank;
    us[j * CD_TT + t] = t < nt ? DT<T>::to_f(reinterpret_cast<const T *>(p.u)[(size_t)(m0 + t) * p.ld + j]) : 0.f;
  }
  __syncthreads();
  if (ch >= p.channels) return;
  float z[CD_TT];
  const float b = DT<T>::to_f(reinterpret_cast<const T *>(p.bias)[ch]);
#pragma unroll
  for (int t = 0; t < CD_TT; t++) z[t] = b;
  const T *w = reinterpret_cast<const T *>(p.w) + (size_t)ch * p.rank;
  for (int j = 0; j < p.rank; j++) {
    const float wj = DT<T>::to_f(w[j]);
#pragma unroll
    for (int t = 0; t < CD_TT; t += 4) {
      const float4 u = *reinterpret_cast<const float4 *>(us + j * CD_TT + t);
      z[t] = fmaf(wj, u.x, z[t]); z[t + 1] = fmaf(wj, u.y, z[t + 1]); z[t + 2] = fmaf(wj, u.z, z[t + 2]); z[t + 3] = fmaf(wj, u.w, z[t + 3]);
    }
  }
  // sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau)
#pragma unroll
  for (int t = 0; t < CD_TT; t++)
    if (t < nt) p.a[(size_t)(m0 + t) * p.channels + ch] = expf(-softplus_f(-z[t]) / p.tau);
}
int channel_decay(cudaStream_t st, int dtype, const ChannelDecay &p, uint64_t *launches) {
  if (p.M < 1 || p.channels < 1 || p.rank < 1 || !(p.tau > 0.f)) return (int)cudaErrorInvalidValue;
  const size_t smem = (size_t)p.rank * CD_TT * sizeof(float);
  if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  MX_DISPATCH(dtype, {
    if (smem > 48 * 1024) {
      cudaError_t e = cudaFuncSetAttribute(channel_decay_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return (int)e;
    }
    channel_decay_kernel<T><<<dim3((p.channels + 127) / 128, (p.M + CD_TT - 1) / CD_TT), 128, smem, st>>>(p);
  });
  MX_DONE(1);
}

// ---------------------------------------------------------------------------------------------- recurrence with channel decays
// A CTA walks the step's tokens for CW * 16 columns of one (head, batch row)'s state.  Its eight warps are RW row groups of 32 key
// channels by CW column groups of 16; a lane keeps a 4 x 4 tile of the state in registers (lane & 7: which four rows, lane >> 3: which
// four columns), so that a token costs it four 16-byte shared-memory loads (q, k, a of its rows, v of its columns) for 48 multiply-adds.
// Tokens come in chunks of 16: the raw values of the next chunk wait in registers while the current one is computed; the partial
// outputs of a warp's rows are summed over its lanes by a transposing exchange, those of the row groups once per chunk.  Rows
// beyond dk and columns beyond dv hold zeros.
constexpr int CR_TT = 16;
template <typename T> struct Raw4 { typedef uint2 type; };
template <> struct Raw4<float> { typedef float4 type; };
template <typename T> __device__ __forceinline__ float4 raw_to_f4(const typename Raw4<T>::type &r) {
  const float2 a = DT<T>::unpack2(r.x), b = DT<T>::unpack2(r.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
template <> __device__ __forceinline__ float4 raw_to_f4<float>(const float4 &r) { return r; }

template <typename T, int RW>
__global__ void __launch_bounds__(256) recurrence_channels_kernel(const Recurrence p) {
  constexpr int CW = 8 / RW, DK = RW * 32, CB = CW * 16, NQ = (CR_TT * DK / 4 + 255) / 256;  // NQ: 4-entry pieces of q (k, a) per thread and chunk
  constexpr int NVP = (CR_TT * CB / 4 + 255) / 256;
  extern __shared__ __align__(16) float sm[];
  float *qs = sm, *ks = qs + CR_TT * DK, *as = ks + CR_TT * DK, *vs = as + CR_TT * DK, *part = vs + CR_TT * CB;  // part [RW][CR_TT][CB]
  const int ncb = (p.dv + CB - 1) / CB, h = blockIdx.x / ncb, c0 = (blockIdx.x % ncb) * CB, b = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, rw = warp % RW, cw = warp / RW;
  const int rl = lane & 7, cl = lane >> 3, row0 = rw * 32 + rl * 4, colb = cw * 16 + cl * 4, col0 = c0 + colb;
  const bool live = row0 < p.dk && col0 < p.dv;
  float *gs = p.state + (((size_t)b * p.heads + h) * p.dk + row0) * p.dv + col0;
  float St[4][4];
#pragma unroll
  for (int r = 0; r < 4; r++) {
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    if (live && p.pos0 > 0) s = *reinterpret_cast<const float4 *>(gs + (size_t)r * p.dv);
    St[r][0] = s.x; St[r][1] = s.y; St[r][2] = s.z; St[r][3] = s.w;
  }
  typedef typename Raw4<T>::type R4;
  R4 rq[NQ], rk[NQ], rv[NVP];
  float4 ra[NQ];
  const int dk4 = p.dk / 4, dv4 = p.dv / 4;
  auto fetch = [&](int t0) {  // indices are clamped: what lies beyond the chunk or the head is replaced when the chunk is staged
    const int nt = min(CR_TT, p.S - t0);
    const size_t m0 = (size_t)b * p.S + t0;
#pragma unroll
    for (int e = 0; e < NQ; e++) {
      const int idx = threadIdx.x + 256 * e, tt = min(idx / (DK / 4), nt - 1), i = min(idx % (DK / 4), dk4 - 1);
      rq[e] = *reinterpret_cast<const R4 *>(reinterpret_cast<const T *>(p.q) + (m0 + tt) * p.ldq + (size_t)h * p.dk + 4 * i);
      rk[e] = *reinterpret_cast<const R4 *>(reinterpret_cast<const T *>(p.k) + (m0 + tt) * p.ldk + (size_t)h * p.dk + 4 * i);
      ra[e] = *reinterpret_cast<const float4 *>(p.a_chan + ((m0 + tt) * p.heads + h) * p.dk + 4 * i);
    }
#pragma unroll
    for (int e = 0; e < NVP; e++) {
      const int idx = threadIdx.x + 256 * e, tt = min(idx / (CB / 4), nt - 1), i = min(c0 / 4 + idx % (CB / 4), dv4 - 1);
      rv[e] = *reinterpret_cast<const R4 *>(reinterpret_cast<const T *>(p.v) + (m0 + tt) * p.ldv + (size_t)h * p.dv + 4 * i);
    }
  };
  const bool hi1 = rl & 1, hi2 = rl & 2;
  const int pcol = colb + (rl & 1) * 2 + ((rl >> 1) & 1);  // the column whose sum this lane ends up with
  auto token = [&](int tt) {
    const float4 q = *reinterpret_cast<const float4 *>(qs + tt * DK + row0), k = *reinterpret_cast<const float4 *>(ks + tt * DK + row0);
    const float4 a = *reinterpret_cast<const float4 *>(as + tt * DK + row0), v = *reinterpret_cast<const float4 *>(vs + tt * CB + colb);
    const float qr[4] = {q.x, q.y, q.z, q.w}, kr[4] = {k.x, k.y, k.z, k.w}, ar[4] = {a.x, a.y, a.z, a.w}, vc[4] = {v.x, v.y, v.z, v.w};
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int r = 0; r < 4; r++)
#pragma unroll
      for (int c = 0; c < 4; c++) {
        St[r][c] = fmaf(ar[r], St[r][c], kr[r] * vc[c]);
        acc[c] = fmaf(St[r][c], qr[r], acc[c]);
      }
    // lanes that differ in rl share columns: two exchanges halve the columns a lane holds, the third adds the rest
    float k0 = hi1 ? acc[2] : acc[0], k1 = hi1 ? acc[3] : acc[1];
    k0 += __shfl_xor_sync(0xffffffffu, hi1 ? acc[0] : acc[2], 1);
    k1 += __shfl_xor_sync(0xffffffffu, hi1 ? acc[1] : acc[3], 1);
    float s = hi2 ? k1 : k0;
    s += __shfl_xor_sync(0xffffffffu, hi2 ? k0 : k1, 2);
    s += __shfl_xor_sync(0xffffffffu, s, 4);
    if (rl < 4) part[(rw * CR_TT + tt) * CB + pcol] = s;
  };
  fetch(0);
  for (int t0 = 0; t0 < p.S; t0 += CR_TT) {
    const int nt = min(CR_TT, p.S - t0);
    const size_t m0 = (size_t)b * p.S + t0;
    __syncthreads();  // the previous chunk's outputs have been added up
#pragma unroll
    for (int e = 0; e < NQ; e++) {
      const int idx = threadIdx.x + 256 * e;
      const bool in = idx % (DK / 4) < dk4;
      float4 q = raw_to_f4<T>(rq[e]), k = raw_to_f4<T>(rk[e]), a = ra[e];
      q.x *= p.qscale; q.y *= p.qscale; q.z *= p.qscale; q.w *= p.qscale;
      k.x *= p.kscale; k.y *= p.kscale; k.z *= p.kscale; k.w *= p.kscale;
      if (!in) q = k = a = make_float4(0.f, 0.f, 0.f, 0.f);
      if (idx >= CR_TT * DK / 4) continue;
      reinterpret_cast<float4 *>(qs)[idx] = q;
      reinterpret_cast<float4 *>(ks)[idx] = k;
      reinterpret_cast<float4 *>(as)[idx] = a;
    }
#pragma unroll
    for (int e = 0; e < NVP; e++) {
      const int idx = threadIdx.x + 256 * e;
      if (idx < CR_TT * CB / 4)
        reinterpret_cast<float4 *>(vs)[idx] = c0 / 4 + idx % (CB / 4) < dv4 ? raw_to_f4<T>(rv[e]) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    __syncthreads();
    if (t0 + CR_TT < p.S) fetch(t0 + CR_TT);  // in flight while this chunk is computed
    if (nt == CR_TT) {
#pragma unroll 4
      for (int tt = 0; tt < CR_TT; tt++) token(tt);
    } else {
      for (int tt = 0; tt < nt; tt++) token(tt);
    }
    __syncthreads();
    for (int idx = threadIdx.x; idx < nt * CB; idx += 256) {
      const int tt = idx / CB, j = idx % CB;
      float o = 0.f;
#pragma unroll
      for (int w = 0; w < RW; w++) o += part[(w * CR_TT + tt) * CB + j];
      if (c0 + j < p.dv) p.o[((m0 + tt) * p.heads + h) * p.dv + c0 + j] = o;
    }
  }
  if (live)
#pragma unroll
    for (int r = 0; r < 4; r++) *reinterpret_cast<float4 *>(gs + (size_t)r * p.dv) = make_float4(St[r][0], St[r][1], St[r][2], St[r][3]);
}
template <typename T, int RW> static cudaError_t launch_recurrence_channels(cudaStream_t st, const Recurrence &p) {
  constexpr int CB = 8 / RW * 16;
  const size_t smem = (size_t)(3 * CR_TT * RW * 32 + CR_TT * CB + RW * CR_TT * CB) * sizeof(float);
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(recurrence_channels_kernel<T, RW>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  recurrence_channels_kernel<T, RW><<<dim3(p.heads * ((p.dv + CB - 1) / CB), p.B), 256, smem, st>>>(p);
  return cudaSuccess;
}
int recurrence_channels(cudaStream_t st, int dtype, const Recurrence &p) {
  const uintptr_t in_align = dtype == 2 ? 15 : 7;
  if (p.dk > 256 || p.dk % 4 || p.dv % 4 || p.ldq % 4 || p.ldk % 4 || p.ldv % 4 || p.group_div != 1 ||
      (((uintptr_t)p.q | (uintptr_t)p.k | (uintptr_t)p.v) & in_align) || (((uintptr_t)p.a_chan | (uintptr_t)p.state) & 15))
    return (int)cudaErrorNotSupported;
  cudaError_t e = cudaSuccess;
  MX_DISPATCH(dtype, {
    if (p.dk <= 32) e = launch_recurrence_channels<T, 1>(st, p);
    else if (p.dk <= 64) e = launch_recurrence_channels<T, 2>(st, p);
    else if (p.dk <= 128) e = launch_recurrence_channels<T, 4>(st, p);
    else e = launch_recurrence_channels<T, 8>(st, p);
  });
  return (int)(e != cudaSuccess ? e : cudaGetLastError());
}

}  // namespace mx
}  // namespace cake
