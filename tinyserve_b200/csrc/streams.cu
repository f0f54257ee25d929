// Several parallel residual streams instead of one (hyper-connections).
//
// A token has S streams x_1 .. x_S (32-bit rows of n elements, [T, S, n]).  A sub-layer reads
// u = sum_s in[s] x_s through its norm and gives y; then every stream becomes, from the old ones,
//   x_t <- sum_s mix[s, t] x_s + out[t] y            (mix is indexed [from, to]).
// One kernel does what lies between two sub-layers: it takes in the y of the sub-layer before (a tensor of
// the compute type, or split-K partial tiles plus a bias row), brings the streams up to date, reads them with
// the next sub-layer's weights and writes the norm of that sum: a layer norm (mean taken off, optional
// bias) or an RMS norm.  The model's last norm is the same kernel with the reading weights all one.
//
// Before the first update all streams are one and the same row (the embedding output): the source
// then has a stream stride of 0, and no copy of it is ever made.  All arithmetic is 32-bit.
#include "common.cuh"

TS_DEFINE_LAST_ERROR()

namespace {

constexpr int MAX_STREAMS = 32;
constexpr int HELD_STREAMS = 4;         // up to this many the coefficients live in registers
constexpr int ROW_CLUSTER = 8;          // blocks that share a row when there are few rows
constexpr int PARTIAL_BATCH = 8;

struct MixParams {
  const float* src; long long src_row, src_stream;     // strides in elements; src_stream 0: one row for all streams
  float* dst;                                          // [T, S, n], null: the streams are not written
  const void* x; PartialSrc ps; VecParam bias;         // y: a tensor, or partial tiles (plus bias), or neither
  VecParam mix, out;                                   // [S, S], [S]; read only with a y
  VecParam in;                                         // [S]; ptr null: ones
  VecParam w, b;                                       // the norm's weight and bias (ptr null: none)
  float eps;
  int centred;                                         // 1: layer norm, 0: RMS norm
  void* h;                                             // [rows, n]
  const int* rows;                                     // row i of h is token rows[i]; null: token i
  int n, S;
};

template <typename T> struct Four;
template <> struct Four<float> {
  static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
    const float4 q = *reinterpret_cast<const float4*>(p);
    v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
};
template <> struct Four<__nv_bfloat16> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[4]) {
    const uint2 q = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&q.x), b = *reinterpret_cast<const __nv_bfloat162*>(&q.y);
    v[0] = __low2float(a); v[1] = __high2float(a); v[2] = __low2float(b); v[3] = __high2float(b);
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[4]) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 q;
    q.x = *reinterpret_cast<uint32_t*>(&a);
    q.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = q;
  }
};

__device__ __forceinline__ void four_param(const VecParam& w, int c, float (&v)[4]) {
  if (w.is_f32) Four<float>::load(static_cast<const float*>(w.ptr) + c, v);
  else Four<__nv_bfloat16>::load(static_cast<const __nv_bfloat16*>(w.ptr) + c, v);
}

// Any number of streams, any row length: the row u waits in shared memory between the passes.
template <typename T>
__global__ void stream_mix_kernel(MixParams p) {
  extern __shared__ float row[];
  __shared__ float scratch[33];
  __shared__ float coef[MAX_STREAMS * MAX_STREAMS + 2 * MAX_STREAMS];
  pdl_trigger();
  const int S = p.S, n = p.n;
  const bool has_y = p.x != nullptr || p.ps.base != nullptr;
  float *mix = coef, *out = coef + S * S, *in = out + S;
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) mix[i] = has_y ? p.mix[i] : 0.f;
  for (int i = threadIdx.x; i < S; i += blockDim.x) {
    out[i] = has_y ? p.out[i] : 0.f;
    in[i] = p.in.ptr ? p.in[i] : 1.f;
  }
  pdl_wait();
  __syncthreads();
  const size_t i = blockIdx.x, r = p.rows ? (size_t)p.rows[i] : i;
  float sum = 0.f;
  for (int c = threadIdx.x; c < n; c += blockDim.x) {
    float xs[MAX_STREAMS];
    for (int s = 0; s < S; ++s) xs[s] = p.src[r * p.src_row + s * p.src_stream + c];
    float u = 0.f;
    if (has_y) {
      float y = p.ps.base ? p.ps.load1((int)r, c) : to_f32<T>(static_cast<const T*>(p.x)[r * n + c]);
      if (p.bias.ptr) y += p.bias[c];
      for (int t = 0; t < S; ++t) {
        float v = out[t] * y;
        for (int s = 0; s < S; ++s) v = fmaf(mix[s * S + t], xs[s], v);
        if (p.dst) p.dst[(r * S + t) * n + c] = v;
        u = fmaf(in[t], v, u);
      }
    } else {
      for (int s = 0; s < S; ++s) u = fmaf(in[s], xs[s], u);
    }
    row[c] = u;
    sum += u;
  }
  const float mean = p.centred ? block_sum(sum, scratch) / (float)n : 0.f;
  float dev = 0.f;
  for (int c = threadIdx.x; c < n; c += blockDim.x) {
    const float d = row[c] - mean;
    dev = fmaf(d, d, dev);
  }
  const float rstd = rsqrtf(block_sum(dev, scratch) / (float)n + p.eps);
  T* h = static_cast<T*>(p.h) + i * n;
  for (int c = threadIdx.x; c < n; c += blockDim.x) {
    float v = (row[c] - mean) * rstd * p.w[c];
    if (p.b.ptr) v += p.b[c];
    h[c] = from_f32<T>(v);
  }
}

// Four columns at a time, the row u in registers.  CLUSTER: ROW_CLUSTER blocks share a row, and
// exchange (mean, sum of squared deviations) of their parts once; parts combine as
// M2 = sum_k M2_k + n_k (mean_k - mean)^2.
template <typename T, int S, int ITEMS, bool CLUSTER, int MAX_THREADS = 512>
__global__ void __launch_bounds__(MAX_THREADS) stream_mix_vec_kernel(MixParams p, int quads_per_block) {
  __shared__ float scratch[33];
  __shared__ float part_mean, part_dev;
  pdl_trigger();
  const int n = p.n;
  const bool has_y = p.x != nullptr || p.ps.base != nullptr;
  float mix[S][S], out[S], in[S];
#pragma unroll
  for (int t = 0; t < S; ++t) {
#pragma unroll
    for (int s = 0; s < S; ++s) mix[s][t] = has_y ? p.mix[s * S + t] : 0.f;
    out[t] = has_y ? p.out[t] : 0.f;
    in[t] = p.in.ptr ? p.in[t] : 1.f;
  }
  const int base = CLUSTER ? (int)cluster_rank() * quads_per_block : 0;
  pdl_wait();
  const size_t i = CLUSTER ? blockIdx.y : blockIdx.x, r = p.rows ? (size_t)p.rows[i] : i;
  float u[ITEMS][4];
  float sum = 0.f;
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int q = threadIdx.x + it * blockDim.x, c = (base + q) * 4;
#pragma unroll
    for (int e = 0; e < 4; ++e) u[it][e] = 0.f;
    if (q >= quads_per_block || c >= n) continue;
    float xs[S][4], y[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int s = 0; s < S; ++s) Four<float>::load(p.src + r * p.src_row + s * p.src_stream + c, xs[s]);
    if (p.ps.base) {
      if (CLUSTER) {
        // all loads of a batch are issued before the first is used; the sum runs in split order
        for (int s0 = 0; s0 < p.ps.splits; s0 += PARTIAL_BATCH) {
          float4 part[PARTIAL_BATCH];
#pragma unroll
          for (int s = 0; s < PARTIAL_BATCH; ++s)
            if (s0 + s < p.ps.splits) part[s] = __ldcg(reinterpret_cast<const float4*>(p.ps.base + p.ps.offset(s0 + s, (int)r, c)));
#pragma unroll
          for (int s = 0; s < PARTIAL_BATCH; ++s)
            if (s0 + s < p.ps.splits) { y[0] += part[s].x; y[1] += part[s].y; y[2] += part[s].z; y[3] += part[s].w; }
        }
      } else {
        p.ps.load4((int)r, c, y);
      }
    } else if (p.x) {
      Four<T>::load(static_cast<const T*>(p.x) + r * n + c, y);
    }
    if (has_y) {
      if (p.bias.ptr) {
        float bv[4];
        four_param(p.bias, c, bv);
#pragma unroll
        for (int e = 0; e < 4; ++e) y[e] += bv[e];
      }
#pragma unroll
      for (int t = 0; t < S; ++t) {
        float v[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          v[e] = out[t] * y[e];
#pragma unroll
          for (int s = 0; s < S; ++s) v[e] = fmaf(mix[s][t], xs[s][e], v[e]);
          u[it][e] = fmaf(in[t], v[e], u[it][e]);
        }
        if (p.dst) Four<float>::store(p.dst + (r * S + t) * n + c, v);
      }
    } else {
#pragma unroll
      for (int s = 0; s < S; ++s)
#pragma unroll
        for (int e = 0; e < 4; ++e) u[it][e] = fmaf(in[s], xs[s][e], u[it][e]);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) sum += u[it][e];
  }
  const int here = CLUSTER ? max(0, min(quads_per_block * 4, n - base * 4)) : n;       // elements of the row in this block
  float mean = p.centred && here > 0 ? block_sum(sum, scratch) / (float)here : 0.f;
  float dev = 0.f;
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int q = threadIdx.x + it * blockDim.x, c = (base + q) * 4;
    if (q >= quads_per_block || c >= n) continue;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float d = u[it][e] - mean;
      dev = fmaf(d, d, dev);
    }
  }
  float total = block_sum(dev, scratch);
  if (CLUSTER) {
    if (threadIdx.x == 0) {
      part_mean = mean;
      part_dev = total;
    }
    cluster_arrive();
    cluster_wait();
    float means[ROW_CLUSTER], devs[ROW_CLUSTER], all = 0.f;
#pragma unroll
    for (int k = 0; k < ROW_CLUSTER; ++k) {
      means[k] = cluster_load_f32(&part_mean, k);
      devs[k] = cluster_load_f32(&part_dev, k);
      all += means[k] * (float)max(0, min(quads_per_block * 4, n - k * quads_per_block * 4));
    }
    cluster_arrive();        // this block has read its peers; it may not leave before they have read it
    mean = all / (float)n;
    total = 0.f;
#pragma unroll
    for (int k = 0; k < ROW_CLUSTER; ++k) {
      const float d = means[k] - mean;
      total += devs[k] + (float)max(0, min(quads_per_block * 4, n - k * quads_per_block * 4)) * d * d;
    }
  }
  const float rstd = rsqrtf(total / (float)n + p.eps);
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int q = threadIdx.x + it * blockDim.x, c = (base + q) * 4;
    if (q >= quads_per_block || c >= n) continue;
    float wv[4], o[4];
    four_param(p.w, c, wv);
#pragma unroll
    for (int e = 0; e < 4; ++e) o[e] = (u[it][e] - mean) * rstd * wv[e];
    if (p.b.ptr) {
      four_param(p.b, c, wv);
#pragma unroll
      for (int e = 0; e < 4; ++e) o[e] += wv[e];
    }
    Four<T>::store(static_cast<T*>(p.h) + i * n + c, o);
  }
  if (CLUSTER) cluster_wait();
}

template <typename T, int S>
int launch_vec(const MixParams& p, int num_out, cudaStream_t stream) {
  const int n = p.n, quads = n / 4;
  if (num_out <= 64 && n >= 1024 && n <= ROW_CLUSTER * 4 * 256) {
    const int per = (quads + ROW_CLUSTER - 1) / ROW_CLUSTER;
    cudaError_t e = ts_launch_cluster(stream_mix_vec_kernel<T, S, 1, true, 256>, dim3(ROW_CLUSTER, num_out), dim3((per + 31) / 32 * 32), 0,
                                      stream, dim3(ROW_CLUSTER), p, per);
    if (e != cudaSuccess) return ts_fail("stream_mix: %s", cudaGetErrorString(e));
    return 0;
  }
  int items = quads <= 512 ? 1 : (quads <= 1024 ? 2 : (quads <= 2048 ? 4 : 8));
  if (num_out >= 512 && quads >= 256 && items < 4) items *= 2;       // (many rows: fewer threads a row, more rows in flight)
  const int threads = ((quads + items - 1) / items + 31) / 32 * 32;
#define TS_MIX(...) TS_LAUNCH("stream_mix", (stream_mix_vec_kernel<T, S, __VA_ARGS__>), num_out, threads, 0, stream, p, quads)
  if (items == 1) TS_MIX(1, false);
  else if (items == 2 && threads <= 256) TS_MIX(2, false, 256);
  else if (items == 2) TS_MIX(2, false);
  else if (items == 4 && threads <= 256) TS_MIX(4, false, 256);
  else if (items == 4) TS_MIX(4, false);
  else TS_MIX(8, false);
#undef TS_MIX
  return 0;
}

template <typename T>
int launch_mix(const MixParams& p, int num_out, cudaStream_t stream) {
  const uintptr_t all = (uintptr_t)p.src | (uintptr_t)p.dst | (uintptr_t)p.x | (uintptr_t)p.bias.ptr | (uintptr_t)p.w.ptr |
                        (uintptr_t)p.b.ptr | (uintptr_t)p.h;
  if (p.n % 4 == 0 && all % 16 == 0 && p.n <= 4 * 8 * 512 && p.S <= HELD_STREAMS) {
    switch (p.S) {
      case 1: return launch_vec<T, 1>(p, num_out, stream);
      case 2: return launch_vec<T, 2>(p, num_out, stream);
      case 3: return launch_vec<T, 3>(p, num_out, stream);
      default: return launch_vec<T, 4>(p, num_out, stream);
    }
  }
  const int threads = p.n >= 2048 ? 512 : (p.n >= 512 ? 256 : 128);
  const size_t smem = (size_t)p.n * sizeof(float);
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(stream_mix_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return ts_fail("stream_mix: a row of %d elements does not fit shared memory", p.n);
  }
  TS_LAUNCH("stream_mix", stream_mix_kernel<T>, num_out, threads, smem, stream, p);
  return 0;
}

}  // namespace

TS_EXPORT int ts_stream_mix_max_streams() { return MAX_STREAMS; }

// src [., S, n] (or [., n] with src_stream 0) -> dst [., S, n] (null: not written, dst may be src); h [num_out, n].
// y: x [., n], or partial tiles, plus bias; none of the three: the streams are read as they are.
TS_EXPORT int ts_stream_mix(int dtype, const float* src, long long src_row, long long src_stream, float* dst, const void* x,
                            const float* partials, int splits, int n_tiles, int t_tiles, int tile_t, const void* bias, int bias_is_f32,
                            const void* mix, const void* out, const void* in, int coef_is_f32, const void* w, int w_is_f32,
                            const void* b, int b_is_f32, float eps, int centred, void* h, const int* rows, int num_out, int n, int S,
                            cudaStream_t stream) {
  TS_REQUIRE(num_out > 0 && n > 0 && src && w && h, "stream_mix: empty input");
  TS_REQUIRE(S >= 1 && S <= MAX_STREAMS, "stream_mix: 1 to %d streams, got %d", MAX_STREAMS, S);
  TS_REQUIRE((size_t)n * sizeof(float) <= 180 * 1024, "stream_mix: rows of %d elements are too long", n);
  TS_REQUIRE(x == nullptr || partials == nullptr, "stream_mix: one sub-layer output, a tensor or partial tiles");
  const bool has_y = x || partials;
  TS_REQUIRE(!has_y || (mix && out), "stream_mix: a sub-layer output comes with its coefficients");
  TS_REQUIRE(has_y || (dst == nullptr && bias == nullptr), "stream_mix: without a sub-layer output the streams stay as they are");
  TS_REQUIRE(partials == nullptr || (splits > 0 && n_tiles * 128 >= n && tile_t > 0), "stream_mix: partial tiles do not fit the row length");
  TS_REQUIRE(src_stream == 0 || src_stream >= n, "stream_mix: overlapping streams");
  MixParams p{src, src_row, src_stream, dst, x, PartialSrc{partials, splits, n_tiles, t_tiles, tile_t}, VecParam{bias, bias_is_f32},
              VecParam{mix, coef_is_f32}, VecParam{out, coef_is_f32}, VecParam{in, coef_is_f32}, VecParam{w, w_is_f32},
              VecParam{b, b_is_f32}, eps, centred, h, rows, n, S};
  if (dtype == TS_F32) return launch_mix<float>(p, num_out, stream);
  if (dtype == TS_BF16) return launch_mix<__nv_bfloat16>(p, num_out, stream);
  return ts_fail("stream_mix: unknown dtype %d", dtype);
}
