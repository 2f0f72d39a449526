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
  // sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau); the rounding of 1 + exp(-|z|) moves the result by less than its last place / tau
  const float itau = 1.0f / p.tau;
#pragma unroll
  for (int t = 0; t < CD_TT; t++)
    if (t < nt) p.a[(size_t)(m0 + t) * p.channels + ch] = expf(-(fmaxf(-z[t], 0.f) + logf(1.0f + expf(-fabsf(z[t])))) * itau);
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
// four columns), so that a token costs it four shared-memory loads (q, k, a of its rows, v of its columns) for 48 multiply-adds.
// Tokens come in chunks of CR_TT, copied asynchronously as they are (q, k, v in D, a in fp32) into one of two buffers while the other is
// computed on; the partial outputs of a warp's rows are summed over its lanes by a transposing exchange, those of the row groups
// once per chunk.  Rows beyond dk and columns beyond dv hold zeros; places behind the step's last token leave the state as it is.
constexpr int CR_TT = 32;
template <typename T, int RW> struct ChannelTile {
  static constexpr int CW = 8 / RW, DK = RW * 32, CB = CW * 16;
  static constexpr int STAGE = CR_TT * (DK * (2 * (int)sizeof(T) + 4) + CB * (int)sizeof(T));  // a, q, k, v of a chunk in bytes
  static constexpr int SMEM = 2 * STAGE + RW * CR_TT * CB * 4;
};
// four entries global -> shared (8 bytes in 16-bit D, 16 in fp32); nothing is read and zeros arrive when !in
template <int BYTES> __device__ __forceinline__ void copy_async(void *dst, const void *src, bool in) {
  const int n = in ? BYTES : 0;
  asm volatile("cp.async.ca.shared.global [%0], [%1], %2, %3;" ::"r"(smem_u32(dst)), "l"(src), "n"(BYTES), "r"(n) : "memory");
}

template <typename T, int RW>
__global__ void __launch_bounds__(256, 1) recurrence_channels_kernel(const Recurrence p) {
  typedef ChannelTile<T, RW> C;
  constexpr int DK = C::DK, CB = C::CB, PB = 4 * (int)sizeof(T);
  extern __shared__ __align__(16) unsigned char raw[];
  float *part = reinterpret_cast<float *>(raw + 2 * C::STAGE);  // [RW][CR_TT][CB]
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
  auto fetch = [&](int t0, int stage) {
    const int nt = min(CR_TT, p.S - t0);
    const size_t m0 = (size_t)b * p.S + t0;
    float *as = reinterpret_cast<float *>(raw + stage * C::STAGE);
    T *qs = reinterpret_cast<T *>(as + CR_TT * DK), *ks = qs + CR_TT * DK, *vs = ks + CR_TT * DK;
    for (int idx = threadIdx.x; idx < CR_TT * DK / 4; idx += 256) {
      const int tt = idx / (DK / 4), i = 4 * (idx % (DK / 4));
      const bool in = tt < nt && i < p.dk;
      const size_t m = in ? m0 + tt : m0;
      const int e = h * p.dk + (in ? i : 0);
      copy_async<PB>(qs + 4 * idx, reinterpret_cast<const T *>(p.q) + m * p.ldq + e, in);
      copy_async<PB>(ks + 4 * idx, reinterpret_cast<const T *>(p.k) + m * p.ldk + e, in);
      if (tt < nt) copy_async<16>(as + 4 * idx, p.a_chan + m * p.heads * p.dk + e, in);
      else *reinterpret_cast<float4 *>(as + 4 * idx) = make_float4(1.f, 1.f, 1.f, 1.f);
    }
    for (int idx = threadIdx.x; idx < CR_TT * CB / 4; idx += 256) {
      const int tt = idx / (CB / 4), i = c0 + 4 * (idx % (CB / 4));
      const bool in = tt < nt && i < p.dv;
      copy_async<PB>(vs + 4 * idx, reinterpret_cast<const T *>(p.v) + (in ? m0 + tt : m0) * p.ldv + (size_t)h * p.dv + (in ? i : 0), in);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const bool b0 = rl & 1, b1 = rl & 2, b2 = rl & 4;
  // Four tokens at a time: their operands are loaded ahead of the updates, their 16 partial outputs (token j, column c at 4 j + c) are
  // summed over the eight lanes that share the columns by exchanges that halve what a lane holds: 8 + 4 + 2 shuffles leave it the
  // two sums of token 2 b0 + b1, columns 2 b2 and 2 b2 + 1 (b0, b1, b2: the bits of rl).
  auto four = [&](const float *as, const T *qs, const T *ks, const T *vs, int t4) {
    float q[4][4], k[4][4], a[4][4], v[4][4], x[16];
#pragma unroll
    for (int j = 0; j < 4; j++) {
      load4<T>(qs + (t4 + j) * DK + row0, q[j]);
      load4<T>(ks + (t4 + j) * DK + row0, k[j]);
      load4<float>(as + (t4 + j) * DK + row0, a[j]);
      load4<T>(vs + (t4 + j) * CB + colb, v[j]);
    }
#pragma unroll
    for (int j = 0; j < 4; j++) {
#pragma unroll
      for (int c = 0; c < 4; c++) x[4 * j + c] = 0.f;
#pragma unroll
      for (int r = 0; r < 4; r++)
#pragma unroll
        for (int c = 0; c < 4; c++) {
          St[r][c] = fmaf(a[j][r], St[r][c], k[j][r] * v[j][c]);
          x[4 * j + c] = fmaf(St[r][c], q[j][r], x[4 * j + c]);
        }
    }
    float y[8], z[4], o[2];
#pragma unroll
    for (int i = 0; i < 8; i++) y[i] = (b0 ? x[8 + i] : x[i]) + __shfl_xor_sync(0xffffffffu, b0 ? x[i] : x[8 + i], 1);
#pragma unroll
    for (int i = 0; i < 4; i++) z[i] = (b1 ? y[4 + i] : y[i]) + __shfl_xor_sync(0xffffffffu, b1 ? y[i] : y[4 + i], 2);
#pragma unroll
    for (int i = 0; i < 2; i++) o[i] = (b2 ? z[2 + i] : z[i]) + __shfl_xor_sync(0xffffffffu, b2 ? z[i] : z[2 + i], 4);
    *reinterpret_cast<float2 *>(part + (rw * CR_TT + t4 + 2 * b0 + b1) * CB + colb + 2 * b2) = make_float2(o[0], o[1]);
  };
  fetch(0, 0);
  for (int t0 = 0, stage = 0; t0 < p.S; t0 += CR_TT, stage ^= 1) {
    const int nt = min(CR_TT, p.S - t0);
    const size_t m0 = (size_t)b * p.S + t0;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // this chunk has landed; the other buffer and the partial outputs of the chunk before are free
    if (t0 + CR_TT < p.S) fetch(t0 + CR_TT, stage ^ 1);
    const float *as = reinterpret_cast<const float *>(raw + stage * C::STAGE);
    const T *qs = reinterpret_cast<const T *>(as + CR_TT * DK), *ks = qs + CR_TT * DK, *vs = ks + CR_TT * DK;
    for (int t4 = 0; t4 < nt; t4 += 4) four(as, qs, ks, vs, t4);
    __syncthreads();
    for (int idx = threadIdx.x; idx < nt * CB; idx += 256) {
      const int tt = idx / CB, j = idx % CB;
      float o = 0.f;
#pragma unroll
      for (int w = 0; w < RW; w++) o += part[(w * CR_TT + tt) * CB + j];
      if (c0 + j < p.dv) p.o[((m0 + tt) * p.heads + h) * p.dv + c0 + j] = o * p.qscale;  // the output is linear in q
    }
  }
  if (live)
#pragma unroll
    for (int r = 0; r < 4; r++) *reinterpret_cast<float4 *>(gs + (size_t)r * p.dv) = make_float4(St[r][0], St[r][1], St[r][2], St[r][3]);
}
template <typename T, int RW> static cudaError_t launch_recurrence_channels(cudaStream_t st, const Recurrence &p) {
  typedef ChannelTile<T, RW> C;
  static_assert(C::SMEM <= 227 * 1024, "the two buffers and the partial outputs fit an SM");
  static int attr_dev = -1;  // per instantiation: the device the attribute was last set on (the value never changes)
  int dev = 0;
  cudaGetDevice(&dev);
  if (C::SMEM > 48 * 1024 && attr_dev != dev) {
    cudaError_t e = cudaFuncSetAttribute(recurrence_channels_kernel<T, RW>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM);
    if (e != cudaSuccess) return e;
    attr_dev = dev;
  }
  recurrence_channels_kernel<T, RW><<<dim3(p.heads * ((p.dv + C::CB - 1) / C::CB), p.B), 256, C::SMEM, st>>>(p);
  return cudaSuccess;
}
int recurrence_channels(cudaStream_t st, int dtype, const Recurrence &p) {
  const uintptr_t in_align = dtype == 2 ? 15 : 7;
  if (p.dk > 256 || p.dk % 4 || p.dv % 4 || p.ldq % 4 || p.ldk % 4 || p.ldv % 4 || p.group_div != 1 || p.kscale != 1.f ||
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
