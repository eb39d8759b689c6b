// Several residual streams between the parts of a layer, in one pass over a token's row.
//
// A token has S streams x_1 .. x_S of W elements. A part reads a weighted sum of them, and
// its result y goes back into all of them while they are mixed:
//
//   z_t = sum_s mix[s, t] x_s + share[t] (y + bias)     (y the result of the part before;
//                                                         nothing pending: z = x)
//   u   = sum_t in[t] z_t                               (`in` absent: the plain sum)
//   out = u / sqrt(mean(u^2) + eps) * w                 (rounded to the activation type)
//
// All sums, statistics and streams are 32-bit. y may be float32 or bfloat16 rows, or
// `planes` float32 partial results of a split-K product, summed in plane order while they are
// read. `stream_stride` 0 in the input says that all streams are still one row (the stream
// as the embedding left it). One block a token: a thread owns the same elements of every
// stream, so the streams may be rewritten in place, and only u is kept.
#include "common.cuh"

namespace {

constexpr int MAX_STREAMS = 16;

struct StreamArgs {
  const float* x;            // [T][S][W] or, stride 0, [T][W]
  long long token_stride, stream_stride;
  const void* y;             // pending result, or null
  int planes; long long plane_stride;
  const float* bias;         // [W] or null: joins y
  const float* mix;          // [S][S], from x to
  const float* share;        // [S]
  const float* in;           // [S] or null: ones
  float* z;                  // [T][S][W]; null: the mixed streams are not kept
  const float* w;            // [W]
  int S, W;
  float eps, inv_w;
};

template <typename T>
__device__ __forceinline__ void ld4(const T* p, float (&v)[4]);
template <>
__device__ __forceinline__ void ld4<float>(const float* p, float (&v)[4]) {
  const float4 f = __ldcg(reinterpret_cast<const float4*>(p));
  v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
}
template <>
__device__ __forceinline__ void ld4<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 raw = __ldcg(reinterpret_cast<const uint2*>(p));
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
template <typename T>
__device__ __forceinline__ void st4(T* p, const float (&v)[4]) {
  if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  } else {
    uint2 raw;
    *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(v[0], v[1]);
    *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = raw;
  }
}

__device__ __forceinline__ void read_weights(const StreamArgs& p, float* mix, float* share,
                                             float* in) {
  for (int i = threadIdx.x; i < p.S * p.S; i += blockDim.x) mix[i] = p.y != nullptr ? p.mix[i] : 0.f;
  for (int i = threadIdx.x; i < p.S; i += blockDim.x) {
    share[i] = p.y != nullptr ? p.share[i] : 0.f;
    in[i] = p.in != nullptr ? p.in[i] : 1.0f;
  }
}

// Rows of whole 16-byte pieces and up to SM streams: a thread holds ITEMS pieces of u in
// registers, every piece's streams while it mixes them.
template <typename TY, typename TO, int SM, int ITEMS>
__global__ void __launch_bounds__(1024)
stream_mix_norm_kernel(const StreamArgs p, TO* __restrict__ out) {
  __shared__ float scratch[32];
  __shared__ float s_mix[SM * SM], s_share[SM], s_in[SM];
  const int S = p.S;
  read_weights(p, s_mix, s_share, s_in);  // (no earlier kernel's work: read before the wait)
  fb_pdl_launch();
  fb_pdl_wait();
  __syncthreads();
  const float* x = p.x + (size_t)blockIdx.x * p.token_stride;
  float* z = p.z != nullptr ? p.z + (size_t)blockIdx.x * S * p.W : nullptr;
  const size_t y0 = (size_t)blockIdx.x * p.W;
  const TY* y = reinterpret_cast<const TY*>(p.y);
  const int stride = blockDim.x * 4;
  float u[ITEMS][4];
  float ss = 0.f;
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int i = threadIdx.x * 4 + it * stride;
#pragma unroll
    for (int e = 0; e < 4; ++e) u[it][e] = 0.f;
    if (i >= p.W) continue;
    float xs[SM][4], yv[4];
#pragma unroll
    for (int s = 0; s < SM; ++s)
      if (s < S) ld4<float>(x + s * p.stream_stride + i, xs[s]);
    if (y == nullptr) {
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (s < S)
#pragma unroll
          for (int e = 0; e < 4; ++e) u[it][e] = fmaf(s_in[s], xs[s][e], u[it][e]);
    } else {
      ld4<TY>(y + y0 + i, yv);
      for (int k = 1; k < p.planes; ++k) {
        float q[4];
        ld4<TY>(y + k * p.plane_stride + y0 + i, q);
#pragma unroll
        for (int e = 0; e < 4; ++e) yv[e] += q[e];
      }
      if (p.bias != nullptr) {
        float b[4];
        ld4<float>(p.bias + i, b);
#pragma unroll
        for (int e = 0; e < 4; ++e) yv[e] += b[e];
      }
#pragma unroll
      for (int t = 0; t < SM; ++t) {
        if (t >= S) break;
        float zt[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) zt[e] = s_share[t] * yv[e];
#pragma unroll
        for (int s = 0; s < SM; ++s)
          if (s < S)
#pragma unroll
            for (int e = 0; e < 4; ++e) zt[e] = fmaf(s_mix[s * S + t], xs[s][e], zt[e]);
        if (z != nullptr) st4<float>(z + (size_t)t * p.W + i, zt);
#pragma unroll
        for (int e = 0; e < 4; ++e) u[it][e] = fmaf(s_in[t], zt[e], u[it][e]);
      }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) ss = fmaf(u[it][e], u[it][e], ss);
  }
  const float r = 1.0f / sqrtf(fb_block_sum(ss, scratch) * p.inv_w + p.eps);
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int i = threadIdx.x * 4 + it * stride;
    if (i >= p.W) continue;
    float w[4];
    ld4<float>(p.w + i, w);
#pragma unroll
    for (int e = 0; e < 4; ++e) u[it][e] *= r * w[e];
    st4<TO>(out + y0 + i, u[it]);
  }
}

// Any row length and up to MAX_STREAMS streams: element by element, u in shared memory.
template <typename TY, typename TO>
__global__ void __launch_bounds__(256)
stream_mix_norm_any_kernel(const StreamArgs p, TO* __restrict__ out) {
  extern __shared__ float s_u[];  // [W]
  __shared__ float scratch[32];
  __shared__ float s_mix[MAX_STREAMS * MAX_STREAMS], s_share[MAX_STREAMS], s_in[MAX_STREAMS];
  const int S = p.S;
  read_weights(p, s_mix, s_share, s_in);
  fb_pdl_launch();
  fb_pdl_wait();
  __syncthreads();
  const float* x = p.x + (size_t)blockIdx.x * p.token_stride;
  float* z = p.z != nullptr ? p.z + (size_t)blockIdx.x * S * p.W : nullptr;
  const size_t y0 = (size_t)blockIdx.x * p.W;
  const TY* y = reinterpret_cast<const TY*>(p.y);
  float ss = 0.f;
  for (int i = threadIdx.x; i < p.W; i += blockDim.x) {
    float xs[MAX_STREAMS], u = 0.f;
#pragma unroll
    for (int s = 0; s < MAX_STREAMS; ++s)
      xs[s] = s < S ? __ldcg(x + s * p.stream_stride + i) : 0.f;
    if (y == nullptr) {
#pragma unroll
      for (int s = 0; s < MAX_STREAMS; ++s)
        if (s < S) u = fmaf(s_in[s], xs[s], u);
    } else {
      float yv = fb_load_coherent<TY>(y + y0 + i);
      for (int k = 1; k < p.planes; ++k)
        yv += fb_load_coherent<TY>(y + k * p.plane_stride + y0 + i);
      if (p.bias != nullptr) yv += p.bias[i];
#pragma unroll 1
      for (int t = 0; t < S; ++t) {
        float zt = s_share[t] * yv;
#pragma unroll
        for (int s = 0; s < MAX_STREAMS; ++s)
          if (s < S) zt = fmaf(s_mix[s * S + t], xs[s], zt);
        if (z != nullptr) z[(size_t)t * p.W + i] = zt;
        u = fmaf(s_in[t], zt, u);
      }
    }
    s_u[i] = u;
    ss = fmaf(u, u, ss);
  }
  const float r = 1.0f / sqrtf(fb_block_sum(ss, scratch) * p.inv_w + p.eps);
  for (int i = threadIdx.x; i < p.W; i += blockDim.x)  // (a thread reads what it wrote)
    out[y0 + i] = fb_from_float<TO>(s_u[i] * r * p.w[i]);
}

bool whole16(const void* p) { return ((uintptr_t)p % 16) == 0; }
}  // namespace

// x: [T][S][W] with `stream_stride` W, or [T][W] with stride 0 (`z` then receives the streams
// and may not be x). `z` null: nothing is kept (the model's end). `y` null: nothing pending.
FB_API int fb_stream_mix_norm(const float* x, long long token_stride, long long stream_stride,
                              const void* y, int y_dtype, int planes, long long plane_stride,
                              const float* bias, const float* mix, const float* share,
                              const float* in, float* z, const float* w, void* out, int out_dtype,
                              int T, int S, int W, float eps, cudaStream_t stream) {
  FB_REQUIRE(T >= 0 && W > 0 && S >= 1 && S <= MAX_STREAMS && eps >= 0.f,
             "stream_mix_norm: T=%d S=%d (at most %d streams) W=%d", T, S, MAX_STREAMS, W);
  FB_REQUIRE(stream_stride == 0 || stream_stride == W, "stream_mix_norm: streams lie %lld apart",
             stream_stride);
  FB_REQUIRE(y == nullptr || (mix != nullptr && share != nullptr && planes >= 1),
             "stream_mix_norm: a pending result needs the mixing weights");
  FB_REQUIRE(planes == 1 || y_dtype == FB_F32, "stream_mix_norm: planes are float32");
  FB_REQUIRE(stream_stride != 0 || z == nullptr || (const float*)z != x,
             "stream_mix_norm: one row cannot become %d streams in place", S);
  if (T == 0) return 0;
  StreamArgs p{x, token_stride, stream_stride, y, planes, plane_stride, bias, mix, share, in, z, w,
               S, W, eps, 1.0f / (float)W};
  const bool vec = W % 4 == 0 && whole16(x) && whole16(y) && whole16(bias) && whole16(z) &&
                   whole16(w) && whole16(out) && token_stride % 4 == 0 && plane_stride % 4 == 0;
  const int yd = y != nullptr ? y_dtype : FB_F32;
  // (the block width decides the order of a row's sums, so it depends on W alone)
  const int threads = ((W + 3) / 4 + 63) / 64 * 32;  // two pieces each
  if (vec && S <= 4 && threads <= 1024) {
    FB_DISPATCH_DTYPE(yd, TY, FB_DISPATCH_DTYPE(out_dtype, TO, {
      if (S <= 2)
        fb_launch(stream_mix_norm_kernel<TY, TO, 2, 2>, dim3(T), dim3(threads), 0, stream, p, (TO*)out);
      else
        fb_launch(stream_mix_norm_kernel<TY, TO, 4, 2>, dim3(T), dim3(threads), 0, stream, p, (TO*)out);
    }));
    return fb_check_launch("stream_mix_norm");
  }
  const size_t smem = (size_t)W * 4;
  FB_REQUIRE(smem <= 200 * 1024, "stream_mix_norm: rows of %d are more than a block holds", W);
  FB_DISPATCH_DTYPE(yd, TY, FB_DISPATCH_DTYPE(out_dtype, TO, {
    static bool seen[64];
    if (smem > 40 * 1024 && fb_first_use_on_device(seen))
      cudaFuncSetAttribute(stream_mix_norm_any_kernel<TY, TO>,
                           cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    fb_launch(stream_mix_norm_any_kernel<TY, TO>, dim3(T), dim3(256), smem, stream, p, (TO*)out);
  }));
  return fb_check_launch("stream_mix_norm");
}
