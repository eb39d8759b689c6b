// RMS norms on a part's OUTPUT, fused with what follows: the residual sum and the
// next part's input.
//
//   y      = a                                                   one result, or
//   y      = s (a / rms(a) * wa + b / rms(b) * wb)               two results side by side
//   resid += y / rms(y) * w1                                     the norm behind the part
//   out    = resid                      rounded to the activation type, or
//   out    = resid / rms(resid) * w2    the norm in front of what runs next
//
// rms(x) = sqrt(mean(x^2) + eps) over the row. A block whose parts read the stream
// itself and whose norms stand behind the parts does the first three lines and the
// plain `out` once per part; the last part's result meets the model's final norm in
// the same pass. All sums, statistics and the residual are 32-bit; the weights are
// float32 (a norm whose stored weight is the distance from one adds the one at load).
//
// A result may be `planes` float32 partial results of a split-K product, summed in
// plane order while they are read. One block a row; a thread holds its elements in
// registers, so every row is read once.
#include "common.cuh"

namespace {

struct PostNormArgs {
  const float* a; int a_planes; long long a_stride;
  const float* b; int b_planes; long long b_stride;
  const float* wa; const float* wb;
  float pair_scale;
  const float* w1; const float* w2;
  float* resid;
  int W;
  float eps, inv_w;
};

// V: elements of one access (4: float4 pieces of 16-byte aligned rows; 1: any row).
template <int V> struct Piece { float v[V]; };
template <int V>
__device__ __forceinline__ Piece<V> ld(const float* p) {
  Piece<V> r;
  if constexpr (V == 4) {
    const float4 f = __ldcg(reinterpret_cast<const float4*>(p));
    r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w;
  } else {
    r.v[0] = __ldcg(p);
  }
  return r;
}
template <int V>
__device__ __forceinline__ Piece<V> zero() {
  Piece<V> r;
#pragma unroll
  for (int e = 0; e < V; ++e) r.v[e] = 0.f;
  return r;
}
template <int V, typename T>
__device__ __forceinline__ void st(T* p, const Piece<V>& x) {
  if constexpr (V == 4) {
    if constexpr (sizeof(T) == 4) {
      *reinterpret_cast<float4*>(p) = make_float4(x.v[0], x.v[1], x.v[2], x.v[3]);
    } else {
      uint2 raw;
      *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(x.v[0], x.v[1]);
      *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(x.v[2], x.v[3]);
      *reinterpret_cast<uint2*>(p) = raw;
    }
  } else {
    p[0] = fb_from_float<T>(x.v[0]);
  }
}

// Two block-wide sums at once (as fb_block_sum; `scratch` holds 64 floats).
__device__ __forceinline__ float2 block_sum2(float x, float y, float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  x = fb_warp_sum(x);
  y = fb_warp_sum(y);
  __syncthreads();
  if (lane == 0) { scratch[warp] = x; scratch[32 + warp] = y; }
  __syncthreads();
  const int nwarps = (blockDim.x + 31) >> 5;
  x = lane < nwarps ? scratch[lane] : 0.f;
  y = lane < nwarps ? scratch[32 + lane] : 0.f;
  return make_float2(fb_warp_sum(x), fb_warp_sum(y));
}

template <typename TO, int V, int ITEMS>
__global__ void post_norm_kernel(const PostNormArgs p, TO* __restrict__ out) {
  fb_pdl_launch();
  fb_pdl_wait();
  __shared__ float scratch[64];
  const size_t base = (size_t)blockIdx.x * p.W;
  const int stride = blockDim.x * V;
  Piece<V> x[ITEMS], y[ITEMS];
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int i = threadIdx.x * V + it * stride;
    x[it] = i < p.W ? ld<V>(p.resid + base + i) : zero<V>();
    y[it] = (i < p.W && p.a != nullptr) ? ld<V>(p.a + base + i) : zero<V>();
  }
  if (p.a != nullptr) {
    for (int s = 1; s < p.a_planes; ++s)
#pragma unroll
      for (int it = 0; it < ITEMS; ++it) {
        const int i = threadIdx.x * V + it * stride;
        if (i < p.W) {
          const Piece<V> q = ld<V>(p.a + s * p.a_stride + base + i);
#pragma unroll
          for (int e = 0; e < V; ++e) y[it].v[e] += q.v[e];
        }
      }
    if (p.b != nullptr) {
      Piece<V> z[ITEMS];
#pragma unroll
      for (int it = 0; it < ITEMS; ++it) {
        const int i = threadIdx.x * V + it * stride;
        z[it] = i < p.W ? ld<V>(p.b + base + i) : zero<V>();
      }
      for (int s = 1; s < p.b_planes; ++s)
#pragma unroll
        for (int it = 0; it < ITEMS; ++it) {
          const int i = threadIdx.x * V + it * stride;
          if (i < p.W) {
            const Piece<V> q = ld<V>(p.b + s * p.b_stride + base + i);
#pragma unroll
            for (int e = 0; e < V; ++e) z[it].v[e] += q.v[e];
          }
        }
      float sa = 0.f, sb = 0.f;
#pragma unroll
      for (int it = 0; it < ITEMS; ++it)
#pragma unroll
        for (int e = 0; e < V; ++e) {
          sa = fmaf(y[it].v[e], y[it].v[e], sa);
          sb = fmaf(z[it].v[e], z[it].v[e], sb);
        }
      const float2 sums = block_sum2(sa, sb, scratch);
      const float ra = 1.0f / sqrtf(sums.x * p.inv_w + p.eps);
      const float rb = 1.0f / sqrtf(sums.y * p.inv_w + p.eps);
#pragma unroll
      for (int it = 0; it < ITEMS; ++it) {
        const int i = threadIdx.x * V + it * stride;
        if (i < p.W) {
          const Piece<V> wa = ld<V>(p.wa + i), wb = ld<V>(p.wb + i);
#pragma unroll
          for (int e = 0; e < V; ++e)
            y[it].v[e] = p.pair_scale * (y[it].v[e] * ra * wa.v[e] + z[it].v[e] * rb * wb.v[e]);
        }
      }
    }
    float ss = 0.f;
#pragma unroll
    for (int it = 0; it < ITEMS; ++it)
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(y[it].v[e], y[it].v[e], ss);
    const float r = 1.0f / sqrtf(fb_block_sum(ss, scratch) * p.inv_w + p.eps);
#pragma unroll
    for (int it = 0; it < ITEMS; ++it) {
      const int i = threadIdx.x * V + it * stride;
      if (i < p.W) {
        const Piece<V> w = ld<V>(p.w1 + i);
#pragma unroll
        for (int e = 0; e < V; ++e) x[it].v[e] += y[it].v[e] * r * w.v[e];
        st<V, float>(p.resid + base + i, x[it]);
      }
    }
  }
  if (out == nullptr) return;
  if (p.w2 != nullptr) {
    float ss = 0.f;
#pragma unroll
    for (int it = 0; it < ITEMS; ++it)
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(x[it].v[e], x[it].v[e], ss);
    const float r = 1.0f / sqrtf(fb_block_sum(ss, scratch) * p.inv_w + p.eps);
#pragma unroll
    for (int it = 0; it < ITEMS; ++it) {
      const int i = threadIdx.x * V + it * stride;
      if (i < p.W) {
        const Piece<V> w = ld<V>(p.w2 + i);
#pragma unroll
        for (int e = 0; e < V; ++e) x[it].v[e] *= r * w.v[e];
      }
    }
  }
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int i = threadIdx.x * V + it * stride;
    if (i < p.W) st<V, TO>(out + base + i, x[it]);
  }
}

bool aligned16(const void* p) { return ((uintptr_t)p % 16) == 0; }
}  // namespace

FB_API int fb_post_norm_add(const float* a, int a_planes, long long a_stride, const float* b,
                            int b_planes, long long b_stride, const float* wa, const float* wb,
                            float pair_scale, const float* w1, const float* w2, float* resid,
                            void* out, int out_dtype, int T, int W, float eps,
                            cudaStream_t stream) {
  FB_REQUIRE(T >= 0 && W > 0 && eps > 0.f && resid != nullptr, "post_norm_add: bad sizes T=%d W=%d",
             T, W);
  FB_REQUIRE(a != nullptr || b == nullptr, "post_norm_add: a second result without a first");
  FB_REQUIRE(a == nullptr || (w1 != nullptr && a_planes >= 1), "post_norm_add: the norm behind the part has no weight");
  FB_REQUIRE(b == nullptr || (wa != nullptr && wb != nullptr && b_planes >= 1),
             "post_norm_add: two results need a weight each");
  if (T == 0 || (a == nullptr && out == nullptr)) return 0;
  PostNormArgs p{a, a_planes, a_stride, b, b_planes, b_stride, wa, wb, pair_scale, w1, w2, resid, W,
                 eps, 1.0f / (float)W};
  const bool vec = W % 4 == 0 && aligned16(a) && aligned16(b) && aligned16(wa) && aligned16(wb) &&
                   aligned16(w1) && aligned16(w2) && aligned16(resid) && aligned16(out) &&
                   a_stride % 4 == 0 && b_stride % 4 == 0;
  // (the block width decides the order of a row's sums, so it depends on W alone)
  const int pieces = vec ? W / 4 : W;
  int threads = 128;
  while (threads < 1024 && threads * 2 < pieces) threads *= 2;
  const int items = (pieces + threads - 1) / threads;
  FB_REQUIRE(items <= 16, "post_norm_add: rows of %d are more than a block holds", W);
#define FB_POST_NORM(TO, V, ITEMS) \
  fb_launch(post_norm_kernel<TO, V, ITEMS>, dim3(T), dim3(threads), 0, stream, p, (TO*)out)
#define FB_POST_NORM_ITEMS(TO, V)                    \
  do {                                               \
    if (items <= 2) FB_POST_NORM(TO, V, 2);          \
    else if (items <= 4) FB_POST_NORM(TO, V, 4);     \
    else FB_POST_NORM(TO, V, 16);                    \
  } while (0)
  const int od = out ? out_dtype : FB_F32;
  FB_DISPATCH_DTYPE(od, TO, {
    if (vec) FB_POST_NORM_ITEMS(TO, 4);
    else FB_POST_NORM_ITEMS(TO, 1);
  });
#undef FB_POST_NORM_ITEMS
#undef FB_POST_NORM
  return fb_check_launch("post_norm_add");
}
