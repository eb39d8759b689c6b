// Gated linear attention for single tokens, everything between its two products as one
// kernel: the decays from their low-rank projection, one step of the recurrence on the
// state, the norm of a head's output and the output gate.
//
//   a = sigmoid(low Wa2^T + b)^(1 / tau)                    per key channel
//   S <- diag(a) S + k v^T;   o = scale S^T q
//   out = o / sqrt(mean(o^2) + eps) * w * act(gate) * out_scale
//
// A step is a pass over the state: read, changed and written once. The thread-block
// clusters of a (sequence, head) cut the head's value columns into slices; a thread owns
// four neighbouring columns of every R-th key row, and asks for them before it waits for
// the kernel in front (the state was written a whole step ago; the weights are constants).
// The slices' sums of squares meet through the cluster's shared memory for the norm. All
// arithmetic is 32-bit.
#include "common.cuh"

namespace {

constexpr int THREADS = 256;
constexpr int MAX_RANK = 256;

struct StepArgs {
  const float* p; long long ld;          // float32 rows of the input projection
  int at_q, at_k, at_v, at_gate, at_low; // where in a row they begin
  const void* a2; const float* a2_bias;  // [H * dim, rank] as stored, [H * dim]
  float inv_tau;
  const float* norm;                     // [vdim]
  float* state; long long state_stride; long long s_offset;
  void* out; long long out_ld;
  const int* cu_tokens; const int* slots;
  int H, dim, vdim, rank, act;
  float q_scale, eps, out_scale;
};

__device__ __forceinline__ float sigmoidf_(float x) { return 1.0f / (1.0f + expf(-x)); }

__device__ __forceinline__ float read_peer(const float* mine, unsigned rank) {
  uint32_t local = (uint32_t)__cvta_generic_to_shared(mine), remote;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local), "r"(rank));
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(remote) : "memory");
  return v;
}
__device__ __forceinline__ void cluster_barrier() {
  asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
  asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}

// NR: key rows a thread holds at most. TO: the activation type (decays' weight and output).
template <typename TO, int NR>
__global__ void __launch_bounds__(THREADS) linear_step_kernel(const StepArgs a) {
  extern __shared__ __align__(16) float sm[];
  const int dim = a.dim, dim4 = (dim + 3) / 4 * 4, cols = a.vdim / gridDim.z, CG = cols / 4, R = THREADS / CG;
  float* sq = sm;               // [dim] each: scaled query, key, decay
  float* sk = sq + dim4;        // (each padded to whole 16-byte pieces)
  float* sa = sk + dim4;
  float* sv = sa + dim4;        // [cols]
  float* low = sv + cols;       // [rank]
  float* part = low + (a.rank + 3) / 4 * 4;  // [R][cols]
  __shared__ float scratch[32];
  __shared__ float square;
  const int seq = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int t = a.cu_tokens[seq];
  const int cg = tid % CG, rg = tid / CG, col0 = blockIdx.z * cols;
  const bool active = rg < R;
  float* S = a.state + (long long)a.slots[seq] * a.state_stride + a.s_offset +
             (long long)h * dim * a.vdim + col0 + cg * 4;
  float4 s[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int row = rg + i * R;
    s[i] = (active && row < dim) ? __ldcg(reinterpret_cast<const float4*>(S + (long long)row * a.vdim))
                                 : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  fb_pdl_wait();
  const float* p = a.p + (long long)t * a.ld;
  for (int i = tid; i < a.rank; i += THREADS) low[i] = __ldcg(p + a.at_low + i);
  for (int i = tid; i < dim; i += THREADS) {
    sq[i] = __ldcg(p + a.at_q + h * dim + i) * a.q_scale;
    sk[i] = __ldcg(p + a.at_k + h * dim + i);
  }
  for (int i = tid; i < cols; i += THREADS) sv[i] = __ldcg(p + a.at_v + (long long)h * a.vdim + col0 + i);
  __syncthreads();
  // the decays: two lanes a channel, so that 128 channels keep the block's threads busy
  for (int i0 = 0; i0 < dim; i0 += THREADS / 2) {
    const int i = i0 + tid / 2;
    float z = 0.f;
    if (i < dim) {
      const TO* w = (const TO*)a.a2 + ((long long)h * dim + i) * a.rank;
#pragma unroll 8
      for (int r = tid & 1; r < a.rank; r += 2) z = fmaf(low[r], fb_to_float<TO>(w[r]), z);
    }
    z += __shfl_xor_sync(0xffffffffu, z, 1);
    if (i < dim && (tid & 1) == 0) {
      z += a.a2_bias[h * dim + i];
      sa[i] = expf((fminf(z, 0.f) - logf(1.0f + expf(-fabsf(z)))) * a.inv_tau);
    }
  }
  __syncthreads();
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  if (active) {
    const float4 v = *reinterpret_cast<const float4*>(sv + cg * 4);
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int row = rg + i * R;
      if (row < dim) {
        const float g = sa[row], k = sk[row], q = sq[row];
        s[i].x = fmaf(g, s[i].x, k * v.x); s[i].y = fmaf(g, s[i].y, k * v.y);
        s[i].z = fmaf(g, s[i].z, k * v.z); s[i].w = fmaf(g, s[i].w, k * v.w);
        o.x = fmaf(q, s[i].x, o.x); o.y = fmaf(q, s[i].y, o.y);
        o.z = fmaf(q, s[i].z, o.z); o.w = fmaf(q, s[i].w, o.w);
        *reinterpret_cast<float4*>(S + (long long)row * a.vdim) = s[i];
      }
    }
    *reinterpret_cast<float4*>(part + rg * cols + cg * 4) = o;
  }
  fb_pdl_launch();
  __syncthreads();
  float sum = 0.f, y = 0.f;  // (a column a thread: slices have at most THREADS columns)
  if (tid < cols) {
    for (int r = 0; r < R; ++r) y += part[r * cols + tid];
    sum = y * y;
  }
  sum = fb_block_sum(sum, scratch);
  if (gridDim.z > 1) {
    if (tid == 0) square = sum;
    __syncthreads();
    cluster_barrier();
    sum = 0.f;
    for (unsigned c = 0; c < gridDim.z; ++c) sum += read_peer(&square, c);  // in slice order
    cluster_barrier();  // peers may have been reading this block's memory until here
  }
  if (tid < cols) {
    const float r = 1.0f / sqrtf(sum / (float)a.vdim + a.eps);
    const float gz = __ldcg(p + a.at_gate + (long long)h * a.vdim + col0 + tid);
    const float ga = a.act == 0 ? sigmoidf_(gz) : gz * sigmoidf_(gz);
    ((TO*)a.out)[(long long)t * a.out_ld + (long long)h * a.vdim + col0 + tid] =
        fb_from_float<TO>(y * r * a.norm[col0 + tid] * ga * a.out_scale);
  }
}

bool whole(const void* p) { return ((uintptr_t)p % 16) == 0; }

// Slices of a head's columns: as many blocks as fill the device, slices of whole 16-byte
// pieces, and of at most THREADS columns. 0: no such cut.
int slices_for(int n_seqs, int H, int dim, int vdim) {
  if (vdim % 4) return 0;
  int best = 0;
  for (int c = 1; c <= 8; c *= 2) {
    if (vdim % (4 * c)) break;
    const int cols = vdim / c, rows = THREADS / (cols / 4);
    if (cols > THREADS || rows < 1 || (dim + rows - 1) / rows > 16) continue;
    best = c;
    if ((long long)n_seqs * H * c >= 148 || cols / 2 < 32) break;
  }
  return best;
}
}  // namespace

// Whether fb_linear_step takes these sizes.
FB_API int fb_linear_step_fits(int dim, int vdim, int rank) {
  return dim <= 1024 && rank <= MAX_RANK && slices_for(1, 1, dim, vdim) > 0 ? 1 : 0;
}

FB_API int fb_linear_step(const float* p, long long ld, int at_q, int at_k, int at_v, int at_gate,
                          int at_low, const void* a2, const float* a2_bias, float tau,
                          const float* norm, int act, float* state, long long state_stride,
                          long long s_offset, void* out, long long out_ld, int dtype,
                          const int* cu_tokens, const int* slots, int n_seqs, int H, int dim,
                          int vdim, int rank, float q_scale, float eps, float out_scale,
                          cudaStream_t stream) {
  FB_REQUIRE(n_seqs >= 0 && H > 0 && dim > 0 && vdim > 0 && rank > 0 && tau > 0.f &&
             (act == 0 || act == 1) && out_ld >= (long long)H * vdim, "linear_step: bad arguments");
  const int slices = slices_for(n_seqs, H, dim, vdim);
  FB_REQUIRE(slices > 0 && rank <= MAX_RANK && dim <= 1024,
             "linear_step: heads of %d x %d (rank %d) are not built", dim, vdim, rank);
  FB_REQUIRE(whole(state + s_offset) && state_stride % 4 == 0, "linear_step: states must be 16-byte aligned");
  if (n_seqs == 0) return 0;
  StepArgs a{p, ld, at_q, at_k, at_v, at_gate, at_low, a2, a2_bias, 1.0f / tau, norm, state,
             state_stride, s_offset, out, out_ld, cu_tokens, slots, H, dim, vdim, rank, act, q_scale,
             eps, out_scale};
  const int cols = vdim / slices, R = THREADS / (cols / 4), rows = (dim + R - 1) / R;
  const size_t smem = (size_t)(3 * ((dim + 3) / 4 * 4) + cols + (rank + 3) / 4 * 4 + R * cols) * 4;
  FB_REQUIRE(smem <= 48 * 1024, "linear_step: heads of %d x %d do not fit", dim, vdim);
  const dim3 grid(n_seqs, H, slices);
#define FB_LINEAR_STEP(E, NR) \
  fb_launch_cluster(linear_step_kernel<E, NR>, grid, dim3(THREADS), smem, stream, (unsigned)slices, a)
  FB_DISPATCH_DTYPE(dtype, E, {
    if (rows <= 4) FB_LINEAR_STEP(E, 4);
    else if (rows <= 8) FB_LINEAR_STEP(E, 8);
    else FB_LINEAR_STEP(E, 16);
  });
#undef FB_LINEAR_STEP
  return fb_check_launch("linear_step");
}
