// Gated delta rule: a matrix memory whose content under a key is replaced, not added to, for one key size per
// build (-DTS_KEY_DIM=...).  Per request and head, S of key size x value size:
//
//   S <- g_t S;   u_t = beta_t (v_t - S^T k_t);   S <- S + k_t u_t^T;   o_t = S^T q_t
//
// with unit vectors q_t, k_t (x / sqrt(sum(x^2) + 1e-6) of the rows the caller brings; q times a constant),
// beta_t = sigmoid(b_t) and g_t = exp(-exp(rate_h) softplus(a_t + bias_h)) from 32-bit logits, one of each per
// (token, head).  Several heads may share one q and k (`qk_group`).  The head's output is divided by its root mean
// square over the value size, multiplied by a weight and by silu(gate), and stored as T.
//
// The state is 32-bit, lives in the request's state slot between steps, and starts at zero for a request whose
// first token is in this step.  Everything after the projections and their convolution is 32-bit arithmetic.
//
// The value columns of S never meet: column c of S needs q, k, the gates and column c of v.  A block owns some
// columns of one (request, head); a thread keeps ROWS x COLS elements of S in registers, and the GROUPS threads that share
// its columns are neighbouring lanes.  A token needs one exchange among them: with S the state before the
// token, p = S^T k and r = S^T q are summed together, and then
//   u = beta (v - g p),   o = g r + (k . q) u,   S <- g S + k u^T.
// k . q, the gates and the unit vectors do not depend on S: extra warps (the stagers) prepare the next `chunk`
// tokens in shared memory, and store the outputs of the chunk before, while the others compute.
//
// Two forms: wide, four columns a thread (a few tokens: the state's transfer is what counts; where a block takes a
// whole head the output norm runs in the kernel), and narrow, one column a thread (portions: the chain from
// token to token is what counts, so many blocks with short sums).  Where a head is spread over several blocks
// its outputs leave in 32-bit and a second kernel norms and gates them.
#include "common.cuh"

#ifndef TS_KEY_DIM
#error "compile with -DTS_KEY_DIM=<key size>"
#endif

TS_DEFINE_LAST_ERROR()

namespace {

constexpr int DIM = TS_KEY_DIM;
constexpr int STAGERS = 4;                // warps that stage and store
constexpr int MAX_CHUNK = 16;             // tokens staged at a time
constexpr int WIDE_THREADS = 512;         // threads that compute, wide form, at most
constexpr int NARROW_THREADS = 256;       // ... narrow form
constexpr float UNIT_EPS = 1e-6f;

// rows of S per thread: whole runs of four; rows behind DIM are zeros
constexpr int rows_of(int groups) { return (DIM + 4 * groups - 1) / (4 * groups) * 4; }
template <int GROUPS> struct Rows { static constexpr int N = rows_of(GROUPS); };
// threads that share a column: as few as keep a thread's rows at `most` (32 at most)
constexpr int pick_groups(int most) {
  for (int g = 1; g <= 32; g *= 2)
    if (rows_of(g) <= most) return g;
  return 32;
}
constexpr int NARROW_GROUPS = pick_groups(12);         // one column a thread
constexpr int WIDE_GROUPS = pick_groups(8);         // four columns a thread
static_assert(rows_of(NARROW_GROUPS) <= 32 && rows_of(WIDE_GROUPS) <= 32, "key sizes of up to 1,024");

struct DeltaParams {
  const void* q; const void* k; const void* v; const void* gate;
  long long ldq, ldk, ldv, ldg;                     // row strides in elements
  const float* logits; long long ld_logits;         // [T, 2 H]: a, then b
  VecParam bias, rate;                              // [H] each
  float q_scale;
  float* state;                                     // [slots, H, DIM, vdim]
  const int* state_slots; const int* fresh; const int* cu_q;
  VecParam norm_weight; float eps;                  // [vdim]
  void* out; long long ldo;                         // [T, H vdim]
  float* raw;                                       // [T, H vdim]: 32-bit outputs before norm and gate, or null (a block takes a whole head)
  int H, vdim, qk_group;
  int cols, col_tiles;                              // value columns of a block; blocks of a head
  int chunk;
};

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

template <typename T, int GROUPS, int COLS>
__global__ void __launch_bounds__((COLS == 1 ? NARROW_THREADS : WIDE_THREADS) + 32 * STAGERS, 1) delta_rule_kernel(DeltaParams p) {
  constexpr int R = Rows<GROUPS>::N, PD = R * GROUPS, NE = (PD + 31) / 32;
  extern __shared__ float4 smem4[];
  const int chunk = p.chunk, cols = p.cols, vdim = p.vdim;
  float4* gates = smem4;                                      // [2][chunk]: g, beta, k . q
  float* sk = reinterpret_cast<float*>(gates + 2 * chunk);    // [2][chunk][PD]
  float* sq = sk + 2 * chunk * PD;                            // [2][chunk][PD]
  float* sv = sq + 2 * chunk * PD;                            // [2][chunk][cols]
  float* so = sv + 2 * chunk * cols;                          // [2][chunk][cols]
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.x / p.col_tiles, col0 = (blockIdx.x % p.col_tiles) * cols, h = blockIdx.y;
  const int t0 = p.cu_q[b], t1 = p.cu_q[b + 1];
  if (t1 <= t0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int compute_threads = cols / COLS * GROUPS;           // whole warps: see the launch
  const int stager = warp - (compute_threads >> 5);           // negative: a computing warp
  const int hq = h / p.qk_group;
  const T* q = static_cast<const T*>(p.q) + (size_t)hq * DIM;
  const T* k = static_cast<const T*>(p.k) + (size_t)hq * DIM;
  const T* v = static_cast<const T*>(p.v) + (size_t)h * vdim + col0;
  const int chunks = (t1 - t0 + chunk - 1) / chunk;

  // tokens [base, base + n) -> buffer `buf`; a warp per token
  auto stage = [&](int index, int who, int warps) {
    const int base = t0 + index * chunk, n = min(chunk, t1 - base), buf = index & 1;
    const float bias = p.bias[h], rate = p.rate[h];
    for (int tok = who; tok < n; tok += warps) {
      const size_t t = base + tok;
      float kv[NE], qv[NE], kk = 0.f, qq = 0.f, kq = 0.f;
#pragma unroll
      for (int j = 0; j < NE; ++j) {
        const int i = lane + 32 * j;
        kv[j] = i < DIM ? to_f32<T>(__ldg(k + t * p.ldk + i)) : 0.f;
        qv[j] = i < DIM ? to_f32<T>(__ldg(q + t * p.ldq + i)) : 0.f;
      }
      const float a = __ldg(p.logits + t * p.ld_logits + h), bl = __ldg(p.logits + t * p.ld_logits + p.H + h);
      for (int i = lane; i < cols; i += 32) sv[(buf * chunk + tok) * cols + i] = col0 + i < vdim ? to_f32<T>(__ldg(v + t * p.ldv + i)) : 0.f;
#pragma unroll
      for (int j = 0; j < NE; ++j) {
        kk = fmaf(kv[j], kv[j], kk);
        qq = fmaf(qv[j], qv[j], qq);
        kq = fmaf(kv[j], qv[j], kq);
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        kk += __shfl_xor_sync(0xffffffffu, kk, o);
        qq += __shfl_xor_sync(0xffffffffu, qq, o);
        kq += __shfl_xor_sync(0xffffffffu, kq, o);
      }
      const float ik = rsqrtf(kk + UNIT_EPS), iq = rsqrtf(qq + UNIT_EPS) * p.q_scale;
      float* dk = sk + (buf * chunk + tok) * PD;
      float* dq = sq + (buf * chunk + tok) * PD;
#pragma unroll
      for (int j = 0; j < NE; ++j) {
        const int i = lane + 32 * j;
        if (PD % 32 == 0 || i < PD) {
          dk[i] = kv[j] * ik;
          dq[i] = qv[j] * iq;
        }
      }
      if (lane == 0)
        gates[buf * chunk + tok] = make_float4(expf(-expf(rate) * softplus_f(a + bias)), sigmoid_f(bl), kq * ik * iq, 0.f);
    }
  };
  // the outputs of a chunk: norm over the head, weight, gate; or 32-bit as they are.  A warp per token
  auto emit = [&](int index, int who, int warps) {
    const int base = t0 + index * chunk, n = min(chunk, t1 - base), buf = index & 1;
    for (int tok = who; tok < n; tok += warps) {
      const size_t t = base + tok;
      const float* o = so + (buf * chunk + tok) * cols;
      if (p.raw) {
        for (int i = lane; i < cols && col0 + i < vdim; i += 32) p.raw[t * p.H * vdim + (size_t)h * vdim + col0 + i] = o[i];
        continue;
      }
      float acc = 0.f;
      for (int i = lane; i < vdim; i += 32) acc = fmaf(o[i], o[i], acc);
      const float rstd = rsqrtf(warp_sum(acc) / (float)vdim + p.eps);
      const T* gate = static_cast<const T*>(p.gate) + t * p.ldg + (size_t)h * vdim;
      T* out = static_cast<T*>(p.out) + t * p.ldo + (size_t)h * vdim;
      for (int i = lane; i < vdim; i += 32) {
        const float x = to_f32<T>(gate[i]);
        out[i] = from_f32<T>(o[i] * rstd * p.norm_weight[i] * (x * sigmoid_f(x)));
      }
    }
  };

  if (stager >= 0) {
    stage(0, stager, STAGERS);
    for (int c = 0; c < chunks; ++c) {
      __syncthreads();                    // chunk c is staged, chunk c - 1 is computed
      if (c + 1 < chunks) stage(c + 1, stager, STAGERS);
      if (c > 0) emit(c - 1, stager, STAGERS);
    }
    __syncthreads();
    emit(chunks - 1, warp, blockDim.x >> 5);
    return;
  }
  // thread (columns lc COLS .. + COLS, group g) keeps the rows 4 (j GROUPS + g) + e
  const int lc = tid / GROUPS, g = tid % GROUPS;
  const int c0 = col0 + lc * COLS;
  float* S = p.state + ((size_t)p.state_slots[b] * p.H + h) * DIM * vdim + c0;
  const bool from = p.fresh[b] == 0;
  const bool quad = COLS == 4 && c0 + 3 < vdim && vdim % 4 == 0;
  float s[R][COLS];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int row = 4 * ((r >> 2) * GROUPS + g) + (r & 3);
    if (COLS == 4 && from && quad && row < DIM) {
      const float4 x = *reinterpret_cast<const float4*>(S + (size_t)row * vdim);
      s[r][0] = x.x; s[r][COLS > 1 ? 1 : 0] = x.y; s[r][COLS > 2 ? 2 : 0] = x.z; s[r][COLS > 3 ? 3 : 0] = x.w;
    } else {
#pragma unroll
      for (int j = 0; j < COLS; ++j) s[r][j] = from && row < DIM && c0 + j < vdim ? S[(size_t)row * vdim + j] : 0.f;
    }
  }
  for (int c = 0; c < chunks; ++c) {
    __syncthreads();
    const int n = min(chunk, t1 - (t0 + c * chunk)), buf = c & 1;
    const float4* kr = reinterpret_cast<const float4*>(sk + buf * chunk * PD) + g;
    const float4* qr = reinterpret_cast<const float4*>(sq + buf * chunk * PD) + g;
    const float* vr = sv + buf * chunk * cols + lc * COLS;
    float* orow = so + buf * chunk * cols + lc * COLS;
    const float4* gr = gates + buf * chunk;
#pragma unroll(COLS == 1 ? 2 : 1)
    for (int tok = 0; tok < n; ++tok) {
      const float4 ga = gr[tok];
      float kx[R], pk[COLS], pq[COLS];
#pragma unroll
      for (int j = 0; j < COLS; ++j) pk[j] = pq[j] = 0.f;
#pragma unroll
      for (int r4 = 0; r4 < R / 4; ++r4) {
        const float4 k4 = kr[tok * (PD / 4) + r4 * GROUPS], q4 = qr[tok * (PD / 4) + r4 * GROUPS];
        kx[4 * r4] = k4.x; kx[4 * r4 + 1] = k4.y; kx[4 * r4 + 2] = k4.z; kx[4 * r4 + 3] = k4.w;
        const float qx[4] = {q4.x, q4.y, q4.z, q4.w};
        // (short chains: the four products of a run are summed in pairs)
#pragma unroll
        for (int j = 0; j < COLS; ++j) {
          const float ka = fmaf(s[4 * r4][j], kx[4 * r4], s[4 * r4 + 1][j] * kx[4 * r4 + 1]);
          const float kb = fmaf(s[4 * r4 + 2][j], kx[4 * r4 + 2], s[4 * r4 + 3][j] * kx[4 * r4 + 3]);
          const float qa = fmaf(s[4 * r4][j], qx[0], s[4 * r4 + 1][j] * qx[1]);
          const float qb = fmaf(s[4 * r4 + 2][j], qx[2], s[4 * r4 + 3][j] * qx[3]);
          pk[j] += ka + kb;
          pq[j] += qa + qb;
        }
      }
#pragma unroll
      for (int o = 1; o < GROUPS; o <<= 1) {
#pragma unroll
        for (int j = 0; j < COLS; ++j) {
          pk[j] += __shfl_xor_sync(0xffffffffu, pk[j], o);
          pq[j] += __shfl_xor_sync(0xffffffffu, pq[j], o);
        }
      }
      float u[COLS];
#pragma unroll
      for (int j = 0; j < COLS; ++j) {
        u[j] = ga.y * (vr[tok * cols + j] - ga.x * pk[j]);
        pq[j] = fmaf(ga.x, pq[j], ga.z * u[j]);
      }
#pragma unroll
      for (int r4 = 0; r4 < R / 4; ++r4) {
        // (a thread of many elements has no registers to keep k in)
        const float4 k4 = COLS == 1 ? make_float4(kx[4 * r4], kx[4 * r4 + 1], kx[4 * r4 + 2], kx[4 * r4 + 3]) : kr[tok * (PD / 4) + r4 * GROUPS];
        const float ke[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
          for (int j = 0; j < COLS; ++j) s[4 * r4 + e][j] = fmaf(ke[e], u[j], ga.x * s[4 * r4 + e][j]);
      }
      if (g == 0) {
#pragma unroll
        for (int j = 0; j < COLS; ++j) orow[tok * cols + j] = pq[j];
      }
    }
  }
  __syncthreads();
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int row = 4 * ((r >> 2) * GROUPS + g) + (r & 3);
    if (row >= DIM) continue;
    if (COLS == 4 && quad) {
      *reinterpret_cast<float4*>(S + (size_t)row * vdim) = make_float4(s[r][0], s[r][COLS > 1 ? 1 : 0], s[r][COLS > 2 ? 2 : 0], s[r][COLS > 3 ? 3 : 0]);
    } else {
#pragma unroll
      for (int j = 0; j < COLS; ++j)
        if (c0 + j < vdim) S[(size_t)row * vdim + j] = s[r][j];
    }
  }
  emit(chunks - 1, warp, blockDim.x >> 5);
}

// 32-bit outputs -> o / rms(o) * weight * silu(gate), stored as T: a warp per (token, head)
constexpr int FINISH_HOLD = 8;
template <typename T>
__global__ void delta_finish_kernel(DeltaParams p, long long pairs) {
  pdl_trigger();
  const int lane = threadIdx.x & 31, vdim = p.vdim;
  const long long pair = blockIdx.x * (long long)(blockDim.x >> 5) + (threadIdx.x >> 5);
  pdl_wait();
  if (pair >= pairs) return;
  const size_t t = pair / p.H;
  const int h = (int)(pair % p.H);
  const float* o = p.raw + (t * p.H + h) * vdim;
  const T* gate = static_cast<const T*>(p.gate) + t * p.ldg + (size_t)h * vdim;
  T* out = static_cast<T*>(p.out) + t * p.ldo + (size_t)h * vdim;
  float held[FINISH_HOLD], x[FINISH_HOLD], acc = 0.f;
#pragma unroll
  for (int j = 0; j < FINISH_HOLD; ++j) {
    const int i = lane + 32 * j;
    held[j] = i < vdim ? o[i] : 0.f;
    x[j] = i < vdim ? to_f32<T>(gate[i]) : 0.f;
    acc = fmaf(held[j], held[j], acc);
  }
  for (int i = lane + 32 * FINISH_HOLD; i < vdim; i += 32) acc = fmaf(o[i], o[i], acc);
  const float rstd = rsqrtf(warp_sum(acc) / (float)vdim + p.eps);
#pragma unroll
  for (int j = 0; j < FINISH_HOLD; ++j) {
    const int i = lane + 32 * j;
    if (i < vdim) out[i] = from_f32<T>(held[j] * rstd * p.norm_weight[i] * (x[j] * sigmoid_f(x[j])));
  }
  for (int i = lane + 32 * FINISH_HOLD; i < vdim; i += 32) {
    const float g = to_f32<T>(gate[i]);
    out[i] = from_f32<T>(o[i] * rstd * p.norm_weight[i] * (g * sigmoid_f(g)));
  }
}

// value columns of a block: whole warps, about `want` of the narrow form, as many as fit of the wide form
int narrow_columns(int vdim, int want) {
  const int step = NARROW_GROUPS >= 32 ? 1 : 32 / NARROW_GROUPS;
  const int most = NARROW_THREADS / NARROW_GROUPS;
  const int cols = want < step ? step : (want > most ? most : want) / step * step;
  const int padded = (vdim + step - 1) / step * step;
  return cols < padded ? cols : padded;
}
int wide_columns(int vdim) {
  const int step = WIDE_GROUPS >= 32 ? 4 : 4 * (32 / WIDE_GROUPS);
  const int most = WIDE_THREADS / WIDE_GROUPS * 4;
  const int padded = (vdim + step - 1) / step * step;
  return padded < most ? padded : most;
}

template <typename T, int GROUPS, int COLS>
int launch(DeltaParams p, int num_requests, cudaStream_t stream) {
  constexpr int PD = rows_of(GROUPS) * GROUPS;
  auto bytes = [&](int chunk) { return (size_t)2 * chunk * (4 + 2 * PD + 2 * p.cols) * sizeof(float); };
  while (p.chunk > 1 && bytes(p.chunk) > 200 * 1024) p.chunk /= 2;
  const size_t smem = bytes(p.chunk);
  static size_t allowed = 48 * 1024;
  if (smem > allowed) {
    cudaError_t e = cudaFuncSetAttribute(delta_rule_kernel<T, GROUPS, COLS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return ts_fail("delta_rule: %zu bytes of shared memory: %s", smem, cudaGetErrorString(e));
    allowed = smem;
  }
  TS_LAUNCH("delta_rule", (delta_rule_kernel<T, GROUPS, COLS>), dim3(num_requests * p.col_tiles, p.H),
            p.cols / COLS * GROUPS + 32 * STAGERS, smem, stream, p);
  return 0;
}

template <typename T>
int run(DeltaParams& p, bool narrow, int num_requests, int num_tokens, cudaStream_t stream) {
  if (int rc = narrow ? launch<T, NARROW_GROUPS, 1>(p, num_requests, stream) : launch<T, WIDE_GROUPS, 4>(p, num_requests, stream)) return rc;
  if (p.raw == nullptr) return 0;
  const long long pairs = (long long)num_tokens * p.H;
  TS_LAUNCH("delta_finish", delta_finish_kernel<T>, (int)((pairs + 7) / 8), 256, 0, stream, p, pairs);
  return 0;
}

}  // namespace

// blocks that a head of `vdim` value columns is spread over: narrow form with tiles of about `tile` columns, tile 0: wide form
TS_EXPORT int ts_delta_rule_column_tiles(int vdim, int tile) {
  const int cols = tile > 0 ? narrow_columns(vdim, tile) : wide_columns(vdim);
  return (vdim + cols - 1) / cols;
}

// raw [T, H vdim]: scratch of heads that are spread over several blocks, else null
TS_EXPORT int ts_delta_rule(int dtype, const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv,
                            const void* gate, long long ldg, const float* logits, long long ld_logits, const void* bias,
                            int bias_is_f32, const void* rate, int rate_is_f32, float q_scale, float* state, const int* state_slots,
                            const int* fresh, const int* cu_q, int num_requests, int max_q_len, int num_tokens,
                            const void* norm_weight, int norm_weight_is_f32, float eps, void* out, long long ldo, float* raw, int H,
                            int vdim, int qk_group, int tile, cudaStream_t stream) {
  TS_REQUIRE(num_requests > 0 && H > 0 && H <= 65535 && vdim > 0 && num_tokens > 0 && max_q_len > 0, "delta_rule: empty input");
  TS_REQUIRE(qk_group >= 1 && H % qk_group == 0, "delta_rule: %d heads in groups of %d", H, qk_group);
  TS_REQUIRE(q && k && v && gate && logits && bias && rate && state && state_slots && fresh && cu_q && norm_weight && out,
             "delta_rule: a null operand");
  TS_REQUIRE(ld_logits >= 2 * H, "delta_rule: two logits per head and token");
  const int cols = tile > 0 ? narrow_columns(vdim, tile) : wide_columns(vdim), col_tiles = (vdim + cols - 1) / cols;
  TS_REQUIRE((col_tiles > 1) == (raw != nullptr), "delta_rule: heads spread over %d blocks of %d columns: a 32-bit scratch or none", col_tiles, cols);
  DeltaParams p{q, k, v, gate, ldq, ldk, ldv, ldg, logits, ld_logits, VecParam{bias, bias_is_f32}, VecParam{rate, rate_is_f32},
                q_scale, state, state_slots, fresh, cu_q, VecParam{norm_weight, norm_weight_is_f32}, eps, out, ldo, raw, H, vdim,
                qk_group, cols, col_tiles, max_q_len < MAX_CHUNK ? max_q_len : MAX_CHUNK};
  if (dtype == TS_F32) return run<float>(p, tile > 0, num_requests, num_tokens, stream);
  if (dtype == TS_BF16) return run<__nv_bfloat16>(p, tile > 0, num_requests, num_tokens, stream);
  return ts_fail("delta_rule: unknown dtype %d", dtype);
}
