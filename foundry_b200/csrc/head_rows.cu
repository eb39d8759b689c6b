// What stands between an attention's projections and its keys and queries: biases,
// per-head norms, rotation, and the cache write, in one pass over a token's rows.
//
//   x = row + bias                                        (bias where given)
//   q, k: per head  x / sqrt(mean(x^2) + eps) * w         (w [dim], the same for every head;
//         absent: no weight), then the first `rot` elements of a head turned: elements
//         i and i + rot/2 (or 2i and 2i + 1) by the angle p * f_i at position p, with
//         cosine and sine times a constant
//   v:    per head  x / sqrt(mean(x^2) + eps)  where `value_norm`; cached so
//
// With `key_scales` keys and values are one row: x is cached as it is and 1 / sqrt(mean(x^2) +
// eps) beside it, as the factor of that row's scores (the key norm's weight then belongs to
// the queries' weight); such keys are not rotated, and rows are [q | k | anything].
//
// The angles of a step are the same for all of its layers that share the frequencies, so
// they come from a table that one small kernel makes per step: the angle is the
// double-precision product of the position and a double-precision frequency, its cosine
// and sine exact to 32 bits at any position.
#include "common.cuh"

namespace {

// out[t] = (cos of the step's token t for every frequency | sin of the same) * factor
__global__ void step_angles_kernel(const int* __restrict__ positions, const double* __restrict__ freq,
                                   float factor, int T, int half, float* __restrict__ out) {
  fb_pdl_launch();
  fb_pdl_wait();
  const long long n = (long long)T * half;
  for (long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x; idx < n;
       idx += (long long)gridDim.x * blockDim.x) {
    const long long t = idx / half;
    const int i = (int)(idx - t * half);
    double sn, c;
    sincos((double)positions[t] * freq[i], &sn, &c);
    out[t * 2 * half + i] = (float)c * factor;
    out[t * 2 * half + half + i] = (float)sn * factor;
  }
}

// One block a token. Rows of `qkv` are [q: H x dim | k: G x dim | v: G x vdim] in
// float32. Queries go to `q_out` in the activation type, keys and values into the
// token's cache row. `qk_norm` 0 leaves queries and keys as they are; `interleaved`
// 1 turns elements (2i, 2i + 1) instead of (i, i + rot / 2); G may be 0 (a mixer that
// reads another's keys and values has queries only).
template <typename T>
__global__ void head_norm_rope_cache_kernel(const float* qkv, long long ld,
                                            const float* __restrict__ bias, T* __restrict__ q_out,
                                            const float* __restrict__ wq,
                                            const float* __restrict__ wk, float eps,
                                            int qk_norm, int value_norm,
                                            const float* angles, int rot, int interleaved,
                                            const int* __restrict__ positions,
                                            const int* __restrict__ seq_of_token,
                                            const int* __restrict__ page_table, int max_pages,
                                            T* __restrict__ k_cache, T* __restrict__ v_cache,
                                            long long k_page, long long k_head, long long v_page,
                                            long long v_head, int H, int G, int dim, int vdim,
                                            int write_cache, int head_floats, float* key_scales,
                                            long long s_page, long long s_head) {
  fb_pdl_launch();
  fb_pdl_wait();
  extern __shared__ float sg_smem[];  // cos [rot/2] | sin [rot/2] | a head's elements per warp
  const int t = blockIdx.x;
  const int seq = seq_of_token[t];
  const int pos = seq >= 0 ? positions[t] : 0;
  const int half = rot / 2;
  float* cs = sg_smem;
  for (int i = threadIdx.x; i < rot; i += blockDim.x) cs[i] = __ldcg(angles + (size_t)t * rot + i);
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
  float* buf = sg_smem + rot + (size_t)warp * head_floats;
  const float* row = qkv + (size_t)t * ld;
  long long page = 0;
  int r_in_page = 0;
  const bool cached = write_cache && seq >= 0;
  if (cached) {
    page = page_table[(size_t)seq * max_pages + pos / FB_PAGE];
    r_in_page = pos % FB_PAGE;
  }
  // a warp a head; a token's heads (queries, keys, values) are spread over blockIdx.y
  const int units = H + (key_scales != nullptr ? G : 2 * G);
  for (int u = blockIdx.y * nwarps + warp; u < units; u += gridDim.y * nwarps) {
    const bool is_q = u < H, is_k = !is_q && u < H + G;
    const int g = is_q ? u : (is_k ? u - H : u - H - G);
    const int n = (is_q || is_k) ? dim : vdim;
    const float* src = is_q ? row + (size_t)g * dim
                            : is_k ? row + (size_t)H * dim + (size_t)g * dim
                                   : row + (size_t)(H + G) * dim + (size_t)g * vdim;
    const float* badd = bias != nullptr ? bias + (src - row) : nullptr;
    float ss = 0.f;
    for (int d = lane; d < n; d += 32) {
      const float x = __ldcg(src + d) + (badd != nullptr ? badd[d] : 0.f);
      buf[d] = x;
      ss = fmaf(x, x, ss);
    }
    ss = fb_warp_sum(ss);
    const bool normed = (is_q || is_k) ? qk_norm != 0 : value_norm != 0;
    float r = normed ? 1.0f / sqrtf(ss / (float)n + eps) : 1.0f;
    const float* w = is_q ? wq : is_k ? wk : nullptr;
    if (is_k && key_scales != nullptr) {  // the row as it is, its factor beside it
      if (cached && lane == 0) key_scales[page * s_page + (long long)g * s_head + r_in_page] = r;
      r = 1.0f;
    }
    __syncwarp();
    for (int d = lane; d < n; d += 32) buf[d] = buf[d] * r * (w != nullptr ? w[d] : 1.0f);
    __syncwarp();
    if (is_q || is_k) {
      for (int i = lane; i < half; i += 32) {
        const int ia = interleaved ? 2 * i : i, ib = interleaved ? 2 * i + 1 : i + half;
        const float a = buf[ia], b = buf[ib];
        const float c = cs[i], s = cs[half + i];
        buf[ia] = a * c - b * s;
        buf[ib] = b * c + a * s;
      }
      __syncwarp();
    }
    if (is_q) {
      T* dst = q_out + ((size_t)t * H + g) * dim;
      for (int d = lane; d < n; d += 32) dst[d] = fb_from_float<T>(buf[d]);
    } else if (cached) {
      T* dst = is_k ? k_cache + page * k_page + (long long)g * k_head + (long long)r_in_page * dim
                    : v_cache + page * v_page + (long long)g * v_head + (long long)r_in_page * vdim;
      for (int d = lane; d < n; d += 32) dst[d] = fb_from_float<T>(buf[d]);
    }
    __syncwarp();
  }
}


// The same for heads of whole 16-byte pieces up to 128 elements: a head lies in the
// registers of LPH lanes, four neighbouring elements a lane, 32 / LPH heads a warp; the
// element a rotation pairs with is in the same lane (neighbours) or a shuffle away (halves).
template <typename T>
__device__ __forceinline__ void store4(T* p, const float (&x)[4]) {
  if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
  } else {
    uint2 raw;
    *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(x[0], x[1]);
    *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(x[2], x[3]);
    *reinterpret_cast<uint2*>(p) = raw;
  }
}
__device__ __forceinline__ void load4(const float* p, float (&x)[4]) {
  const float4 f = __ldcg(reinterpret_cast<const float4*>(p));
  x[0] = f.x; x[1] = f.y; x[2] = f.z; x[3] = f.w;
}

template <typename T, int LPH>
__global__ void __launch_bounds__(128)
head_rows_vec_kernel(const float* qkv, long long ld, const float* __restrict__ bias,
                     T* __restrict__ q_out, const float* __restrict__ wq,
                     const float* __restrict__ wk, float eps, int qk_norm, int value_norm,
                     const float* angles, int rot, int interleaved,
                     const int* __restrict__ positions, const int* __restrict__ seq_of_token,
                     const int* __restrict__ page_table, int max_pages, T* __restrict__ k_cache,
                     T* __restrict__ v_cache, long long k_page, long long k_head,
                     long long v_page, long long v_head, int H, int G, int dim, int vdim,
                     int write_cache, int n_tokens, float* key_scales, long long s_page,
                     long long s_head) {
  fb_pdl_launch();
  fb_pdl_wait();
  // heads of a token: queries, keys, values
  const int units = H + (key_scales != nullptr ? G : 2 * G);
  const long long at = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / LPH;
  const int lane = threadIdx.x % LPH;
  if (at - (threadIdx.x % 32) / LPH >= (long long)n_tokens * units) return;  // (a whole warp)
  const bool there = at < (long long)n_tokens * units;
  const int t = there ? (int)(at / units) : 0;
  const int u = there ? (int)(at - (long long)t * units) : 0;
  const bool is_q = u < H, is_v = u >= H + G;
  const int g = is_q ? u : is_v ? u - H - G : u - H;
  const int n = is_v ? vdim : dim, d = lane * 4;
  const bool in = there && d < n;
  const long long from = is_q ? (long long)g * dim
                              : !is_v ? (long long)(H + g) * dim
                                      : (long long)(H + G) * dim + (long long)g * vdim;
  float x[4] = {0.f, 0.f, 0.f, 0.f};
  if (in) {
    load4(qkv + (size_t)t * ld + from + d, x);
    if (bias != nullptr) {
      float b[4];
      load4(bias + from + d, b);
#pragma unroll
      for (int e = 0; e < 4; ++e) x[e] += b[e];
    }
  }
  const bool normed = is_v ? value_norm != 0 : qk_norm != 0;
  float ss = x[0] * x[0] + x[1] * x[1] + x[2] * x[2] + x[3] * x[3];
#pragma unroll
  for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const bool as_is = key_scales != nullptr && !is_q;
  const float r = 1.0f / sqrtf(ss / (float)n + eps);
  if (normed && !as_is) {
    const float* w = is_q ? wq : is_v ? nullptr : wk;
    float wv[4] = {1.f, 1.f, 1.f, 1.f};
    if (w != nullptr && in) load4(w + d, wv);
#pragma unroll
    for (int e = 0; e < 4; ++e) x[e] *= r * wv[e];
  }
  if (rot > 0) {  // (the shuffles need every lane, whatever its head)
    const int half = rot / 2;
    const bool turns = in && !is_v && d < rot;
    const float* row = angles + (size_t)t * rot;
    if (interleaved) {
      if (turns) {
        const float2 c = __ldcg(reinterpret_cast<const float2*>(row + d / 2));
        const float2 s = __ldcg(reinterpret_cast<const float2*>(row + half + d / 2));
        const float a0 = x[0] * c.x - x[1] * s.x, b0 = x[1] * c.x + x[0] * s.x;
        const float a1 = x[2] * c.y - x[3] * s.y, b1 = x[3] * c.y + x[2] * s.y;
        x[0] = a0; x[1] = b0; x[2] = a1; x[3] = b1;
      }
    } else {
      const bool low = d < half;
      const int base = (threadIdx.x & 31) - lane, off = half / 4;
      const int partner = base + (low ? min(lane + off, LPH - 1) : max(lane - off, 0));
      float y[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] = __shfl_sync(0xffffffffu, x[e], partner);
      if (turns) {
        float c[4], s[4];
        load4(row + (low ? d : d - half), c);
        load4(row + half + (low ? d : d - half), s);
#pragma unroll
        for (int e = 0; e < 4; ++e) x[e] = low ? x[e] * c[e] - y[e] * s[e] : x[e] * c[e] + y[e] * s[e];
      }
    }
  }
  if (!in) return;
  if (is_q) {
    store4<T>(q_out + ((size_t)t * H + g) * dim + d, x);
    return;
  }
  const int seq = seq_of_token[t];
  if (!write_cache || seq < 0) return;
  const int pos = positions[t];
  const long long page = page_table[(size_t)seq * max_pages + pos / FB_PAGE];
  const int r_in_page = pos % FB_PAGE;
  if (as_is && lane == 0) key_scales[page * s_page + (long long)g * s_head + r_in_page] = r;
  store4<T>(is_v ? v_cache + page * v_page + (long long)g * v_head + (long long)r_in_page * vdim + d
                 : k_cache + page * k_page + (long long)g * k_head + (long long)r_in_page * dim + d, x);
}
}  // namespace

FB_API int fb_step_angles(const int* positions, const double* freq, float factor, int T, int half,
                          float* out, cudaStream_t stream) {
  FB_REQUIRE(T >= 0 && half > 0, "step_angles: bad sizes T=%d half=%d", T, half);
  if (T == 0) return 0;
  const long long n = (long long)T * half;
  const int blocks = (int)((n + 127) / 128 < 8192 ? (n + 127) / 128 : 8192);
  fb_launch(step_angles_kernel, dim3(blocks), dim3(128), 0, stream, positions, freq, factor, T, half,
            out);
  return fb_check_launch("step_angles");
}

// `angles`: float32 [T, rot] as fb_step_angles leaves them (rot 0: none).
FB_API int fb_head_norm_rope_cache_write(const float* qkv, long long ld, const float* bias,
                                         void* q_out, int dtype, const float* wq, const float* wk,
                                         float eps, int qk_norm, int value_norm,
                                         const float* angles, int rot, int interleaved,
                                         const int* positions, const int* seq_of_token,
                                         const int* page_table, int max_pages, void* k_cache,
                                         void* v_cache, long long k_page, long long k_head,
                                         long long v_page, long long v_head, int T, int H, int G,
                                         int dim, int vdim, int write_cache, float* key_scales,
                                         long long s_page, long long s_head, cudaStream_t stream) {
  FB_REQUIRE(T >= 0 && H > 0 && G >= 0 && dim > 0 && vdim > 0, "head_norm_rope_cache_write: bad sizes");
  FB_REQUIRE(G > 0 || !write_cache, "head_norm_rope_cache_write: no keys to write");
  FB_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= dim && (rot == 0 || angles != nullptr),
             "head_norm_rope_cache_write: %d rotated elements of %d", rot, dim);
  FB_REQUIRE(key_scales == nullptr || (G > 0 && qk_norm && rot == 0),
             "head_norm_rope_cache_write: keys with a factor beside them are not rotated");
  FB_REQUIRE(ld >= (long long)(H + G) * dim + (key_scales != nullptr ? 0 : (long long)G * vdim),
             "head_norm_rope_cache_write: rows of %lld are too short", ld);
  if (T == 0) return 0;
  const int heads = H + (key_scales != nullptr ? G : 2 * G);
  auto whole = [](const void* p) { return ((uintptr_t)p % 16) == 0; };
  const int longest = G > 0 && vdim > dim ? vdim : dim;
  if (dim % 4 == 0 && vdim % 4 == 0 && longest <= 128 && rot % (interleaved ? 4 : 8) == 0 &&
      ld % 4 == 0 && whole(qkv) && whole(bias) && whole(q_out) && whole(wq) && whole(wk) &&
      whole(angles) && (!write_cache || (whole(k_cache) && whole(v_cache) && k_page % 4 == 0 &&
      k_head % 4 == 0 && v_page % 4 == 0 && v_head % 4 == 0))) {
#define FB_HEAD_ROWS(E, LPH)                                                                        \
  fb_launch(head_rows_vec_kernel<E, LPH>, dim3((unsigned)(((long long)T * heads * LPH + 127) / 128)), \
            dim3(128), 0, stream, qkv, ld, bias, (E*)q_out, wq, wk, eps, qk_norm, value_norm, angles, \
            rot, interleaved, positions, seq_of_token, page_table, max_pages, (E*)k_cache,            \
            (E*)v_cache, k_page, k_head, v_page, v_head, H, G, dim, vdim, write_cache, T, key_scales,    \
            s_page, s_head)
    FB_DISPATCH_DTYPE(dtype, E, {
      if (longest <= 16) FB_HEAD_ROWS(E, 4);
      else if (longest <= 32) FB_HEAD_ROWS(E, 8);
      else if (longest <= 64) FB_HEAD_ROWS(E, 16);
      else FB_HEAD_ROWS(E, 32);
    });
#undef FB_HEAD_ROWS
    return fb_check_launch("head_norm_rope_cache_write");
  }
  const int warps = heads < 8 ? heads : 8;
  const int head_floats = dim > vdim ? dim : vdim;
  const size_t smem = (size_t)(rot + warps * head_floats) * 4;
  FB_REQUIRE(smem <= 48 * 1024, "head_norm_rope_cache_write: heads of %d do not fit", head_floats);
  const int parts = T <= 256 ? (heads + warps - 1) / warps : 1;  // few tokens: more blocks
  FB_DISPATCH_DTYPE(dtype, E, (fb_launch(head_norm_rope_cache_kernel<E>, dim3(T, parts), dim3(warps * 32),
      smem, stream, qkv, ld, bias, (E*)q_out, wq, wk, eps, qk_norm, value_norm, angles, rot, interleaved,
      positions, seq_of_token, page_table, max_pages, (E*)k_cache, (E*)v_cache, k_page, k_head, v_page,
      v_head, H, G, dim, vdim, write_cache, head_floats, key_scales, s_page, s_head)));
  return fb_check_launch("head_norm_rope_cache_write");
}
