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
// columns of one (request, head); a thread keeps some rows of two columns (or of four) of S in registers, and the
// GROUPS threads that share a column are neighbouring lanes.  Extra warps (the stagers) prepare the next chunk of
// tokens in shared memory, and store the outputs of the chunk before, while the others compute.  Two forms:
//
// * Wide, four columns a thread (a few tokens a request: the state's transfer is what counts).  A token needs one
//   exchange among the lanes of a column: with S the state before it, p = S^T k and r = S^T q are summed together, then
//     u = beta (v - g p),   o = g r + (k . q) u,   S <- g S + k u^T.
//   Where a block takes a whole head the output norm runs in the kernel.
// * Narrow, two columns a thread (portions: the chain from token to token is what counts, and how fast shared memory
//   fills registers, which is why a thread uses what it loads for two columns).  Four tokens share an exchange.
//   With S the state before the four, p_i = S^T k_i, r_i = S^T q_i, and P(j, i) = g_(j+1) ... g_i,
//     u_i = beta_i v_i - beta_i P(-1, i) p_i - sum_(j < i) beta_i P(j, i) (k_i . k_j) u_j
//     o_i = P(-1, i) r_i + sum_(j <= i) P(j, i) (q_i . k_j) u_j
//     S <- P(-1, 3) S + sum_j P(j, 3) k_j u_j^T,
//   which is the recurrence written out.  Everything but p, r and the u does not depend on S: a kernel ahead of this one
//   makes these coefficients for all tokens side by side (the factors that turn q and k into unit vectors among them).
//   Nothing is divided by a decay.
//
// Where a head is spread over several blocks its outputs leave in 32-bit and a second kernel norms and gates them.
#include "common.cuh"

#ifndef TS_KEY_DIM
#error "compile with -DTS_KEY_DIM=<key size>"
#endif

TS_DEFINE_LAST_ERROR()

namespace {

constexpr int DIM = TS_KEY_DIM;
constexpr int STAGERS = 4;                // warps that stage and store
constexpr int MAX_CHUNK = 16;             // tokens staged at a time
constexpr int QUAD = 4;                   // tokens that share an exchange in the narrow form
static_assert(MAX_CHUNK / QUAD == STAGERS, "a stager prepares one group of tokens");
constexpr int WIDE_THREADS = 512;         // threads that compute, wide form, at most
constexpr int NARROW_THREADS = 256;       // ... narrow form
constexpr float UNIT_EPS = 1e-6f;

// rows of S per thread: whole runs of four; rows behind DIM are zeros
constexpr int rows_of(int groups) { return (DIM + 4 * groups - 1) / (4 * groups) * 4; }
template <int GROUPS> struct Rows { static constexpr int N = rows_of(GROUPS); };
// threads that share a column: as few as keep a thread's rows at `most` (32 at most)
constexpr int pick_groups(int most, int fewest) {
  for (int g = fewest; g <= 32; g *= 2)
    if (rows_of(g) <= most) return g;
  return 32;
}
constexpr int NARROW_COLS = 2;
constexpr int SUMS = NARROW_COLS * 2 * QUAD;                  // sums of an exchange, spread over the lanes that share columns
constexpr int NARROW_GROUPS = pick_groups(8, SUMS);
constexpr int WIDE_GROUPS = pick_groups(8, 1);
static_assert(NARROW_THREADS / NARROW_GROUPS * NARROW_COLS <= 32, "a stager's lanes hold four values each of four tokens");
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
  float4* groups;                                   // narrow form: [group slots, H, CO_COUNT] coefficients
};

// where the coefficients of the i-th group of four tokens of request b lie, t0 its first token of the step: no two
// requests share a slot, and num_tokens / 4 + requests + 1 slots are enough
__device__ __forceinline__ size_t group_slot(int b, int t0, int i) { return (size_t)(t0 / QUAD + b + i); }

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

template <typename T>
__global__ void __launch_bounds__(WIDE_THREADS + 32 * STAGERS, 1) delta_rule_wide_kernel(DeltaParams p) {
  constexpr int GROUPS = WIDE_GROUPS, COLS = 4, R = Rows<GROUPS>::N, PD = R * GROUPS, NE = (PD + 31) / 32;
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
  const bool quad = c0 + 3 < vdim && vdim % 4 == 0;
  float s[R][COLS];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int row = 4 * ((r >> 2) * GROUPS + g) + (r & 3);
    if (from && quad && row < DIM) {
      const float4 x = *reinterpret_cast<const float4*>(S + (size_t)row * vdim);
      s[r][0] = x.x; s[r][1] = x.y; s[r][2] = x.z; s[r][3] = x.w;
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
#pragma unroll 1
    for (int tok = 0; tok < n; ++tok) {
      const float4 ga = gr[tok];
      float pk[COLS], pq[COLS];
#pragma unroll
      for (int j = 0; j < COLS; ++j) pk[j] = pq[j] = 0.f;
#pragma unroll
      for (int r4 = 0; r4 < R / 4; ++r4) {
        const float4 k4 = kr[tok * (PD / 4) + r4 * GROUPS], q4 = qr[tok * (PD / 4) + r4 * GROUPS];
        const float kx[4] = {k4.x, k4.y, k4.z, k4.w};
        const float qx[4] = {q4.x, q4.y, q4.z, q4.w};
        // (short chains: the four products of a run are summed in pairs)
#pragma unroll
        for (int j = 0; j < COLS; ++j) {
          const float ka = fmaf(s[4 * r4][j], kx[0], s[4 * r4 + 1][j] * kx[1]);
          const float kb = fmaf(s[4 * r4 + 2][j], kx[2], s[4 * r4 + 3][j] * kx[3]);
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
        const float4 k4 = kr[tok * (PD / 4) + r4 * GROUPS];
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
    if (quad) {
      *reinterpret_cast<float4*>(S + (size_t)row * vdim) = make_float4(s[r][0], s[r][1], s[r][2], s[r][3]);
    } else {
#pragma unroll
      for (int j = 0; j < COLS; ++j)
        if (c0 + j < vdim) S[(size_t)row * vdim + j] = s[r][j];
    }
  }
  emit(chunks - 1, warp, blockDim.x >> 5);
}

// ------------------------------------------------------------------ narrow form
// The coefficients of a group of four tokens, as the computing warps read them (float4 each)
enum { CO_BETA = 0, CO_P = 1, CO_A = 2, CO_O = 4, CO_W = 8, CO_R = 9, CO_COUNT = 10 };
constexpr int CO_TOTAL = 14;              // float of the table that holds P(-1, 3)

// 32 sums over a warp: every exchange halves what a lane still adds up, and lane i ends up with sum i
__device__ __forceinline__ float spread_sum32(float (&v)[32], int lane) {
#pragma unroll
  for (int half = 16; half >= 1; half >>= 1) {
    const bool upper = (lane & half) != 0;
#pragma unroll
    for (int i = 0; i < half; ++i) {
      const float send = upper ? v[i] : v[i + half], keep = upper ? v[i + half] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, send, half);
    }
  }
  return v[0];
}

// four neighbouring elements of a row as they come
template <typename T> struct RawFour;
template <> struct RawFour<float> {
  float4 raw;
  __device__ __forceinline__ void load(const float* p, int left, bool vec) {
    if (vec) raw = __ldg(reinterpret_cast<const float4*>(p));
    else raw = make_float4(left > 0 ? __ldg(p) : 0.f, left > 1 ? __ldg(p + 1) : 0.f, left > 2 ? __ldg(p + 2) : 0.f, left > 3 ? __ldg(p + 3) : 0.f);
  }
  __device__ __forceinline__ void zero() { raw = make_float4(0.f, 0.f, 0.f, 0.f); }
  __device__ __forceinline__ float4 get() const { return raw; }
};
template <> struct RawFour<__nv_bfloat16> {
  uint2 raw;
  __device__ __forceinline__ void load(const __nv_bfloat16* p, int left, bool vec) {
    if (vec) {
      raw = __ldg(reinterpret_cast<const uint2*>(p));
    } else {
      const unsigned short* e = reinterpret_cast<const unsigned short*>(p);
      const uint32_t a = left > 0 ? __ldg(e) : 0, b = left > 1 ? __ldg(e + 1) : 0, c = left > 2 ? __ldg(e + 2) : 0, d = left > 3 ? __ldg(e + 3) : 0;
      raw = make_uint2(a | b << 16, c | d << 16);
    }
  }
  __device__ __forceinline__ void zero() { raw = make_uint2(0, 0); }
  __device__ __forceinline__ float4 get() const {
    return make_float4(__uint_as_float(raw.x << 16), __uint_as_float(raw.x & 0xffff0000u), __uint_as_float(raw.y << 16),
                       __uint_as_float(raw.y & 0xffff0000u));
  }
};

// The coefficients of every group of four tokens: a warp per (request, group, query/key head), for all heads that
// share it.  A token behind the request's last one changes nothing: g 1, beta 0, q and k 0.
constexpr int PREPARE_WARPS = 4;
template <typename T>
__global__ void __launch_bounds__(32 * PREPARE_WARPS) delta_prepare_kernel(DeltaParams p, int vec) {
  constexpr int NQ = (DIM + 127) / 128;
  __shared__ float all_scratch[PREPARE_WARPS][40];
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t0 = p.cu_q[b], t1 = p.cu_q[b + 1], first = t0 + blockIdx.x * QUAD, hq = blockIdx.y * PREPARE_WARPS + warp;
  if (first >= t1 || hq * p.qk_group >= p.H) return;
  float* scratch = all_scratch[warp];                         // dots [32], then g and beta [4] each
  const T* q = static_cast<const T*>(p.q) + (size_t)hq * DIM;
  const T* k = static_cast<const T*>(p.k) + (size_t)hq * DIM;
  float dot[32];
#pragma unroll
  for (int d = 0; d < 32; ++d) dot[d] = 0.f;
#pragma unroll
  for (int j = 0; j < NQ; ++j) {
    const int at = 4 * (lane + 32 * j);
    RawFour<T> raw[2 * QUAD];
#pragma unroll
    for (int i = 0; i < 2 * QUAD; ++i) {
      const int t = first + (i & (QUAD - 1));
      if (t < t1 && at < DIM) raw[i].load((i < QUAD ? k + (size_t)t * p.ldk : q + (size_t)t * p.ldq) + at, DIM - at, vec != 0);
      else raw[i].zero();
    }
    float4 x[2 * QUAD];
#pragma unroll
    for (int i = 0; i < 2 * QUAD; ++i) x[i] = raw[i].get();
    auto add = [&](int d, const float4& a, const float4& c) {
      dot[d] = fmaf(a.x, c.x, fmaf(a.y, c.y, fmaf(a.z, c.z, fmaf(a.w, c.w, dot[d]))));
    };
#pragma unroll
    for (int i = 0; i < QUAD; ++i) {
#pragma unroll
      for (int l = 0; l <= i; ++l) {
        add(i * (i + 1) / 2 + l, x[i], x[l]);                          // k_i . k_l
        add(10 + i * (i + 1) / 2 + l, x[QUAD + i], x[l]);              // q_i . k_l
      }
      add(20 + i, x[QUAD + i], x[QUAD + i]);                           // q_i . q_i
    }
  }
  scratch[lane] = spread_sum32(dot, lane);
  __syncwarp();
  auto inv_k = [&](int i) { return rsqrtf(scratch[i * (i + 1) / 2 + i] + UNIT_EPS); };
  auto inv_q = [&](int i) { return rsqrtf(scratch[20 + i] + UNIT_EPS) * p.q_scale; };
  const int t = first + (lane & 3);
  for (int h = hq * p.qk_group; h < (hq + 1) * p.qk_group; ++h) {
    if (lane < 8) {
      const bool live = t < t1;
      const float logit = live ? __ldg(p.logits + (size_t)t * p.ld_logits + (lane < 4 ? h : p.H + h)) : 0.f;
      scratch[32 + lane] = !live ? (lane < 4 ? 1.f : 0.f)
                                 : (lane < 4 ? expf(-expf(p.rate[h]) * softplus_f(logit + p.bias[h])) : sigmoid_f(logit));
    }
    __syncwarp();
    const float* g = scratch + 32;
    auto fade = [&](int from, int to) {                     // P(from, to)
      float x = 1.f;
#pragma unroll
      for (int l = 0; l < QUAD; ++l)
        if (l > from && l <= to) x *= g[l];
      return x;
    };
    float value = 0.f;
    if (lane < 4) {
      value = g[4 + lane];
    } else if (lane < 8) {
      const int i = lane - 4;
      value = g[4 + i] * fade(-1, i) * inv_k(i);
    } else if (lane < 14) {
      const int a = lane - 8, i = a < 1 ? 1 : (a < 3 ? 2 : 3), j = a - i * (i - 1) / 2;
      value = g[4 + i] * fade(j, i) * scratch[i * (i + 1) / 2 + j] * inv_k(i) * inv_k(j);
    } else if (lane == CO_TOTAL) {
      value = fade(-1, QUAD - 1);
    } else if (lane >= 16) {
      const int i = (lane - 16) >> 2, j = lane & 3;
      if (j <= i) value = fade(j, i) * scratch[10 + i * (i + 1) / 2 + j] * inv_q(i) * inv_k(j);
    }
    float* table = reinterpret_cast<float*>(p.groups + (group_slot(b, t0, blockIdx.x) * p.H + h) * CO_COUNT);
    table[lane] = value;
    if (lane < 8) table[32 + lane] = lane < 4 ? fade(lane, QUAD - 1) * inv_k(lane) : fade(-1, lane - 4) * inv_q(lane - 4);
    __syncwarp();
  }
}

// two neighbouring 32-bit numbers in one instruction
typedef unsigned long long pair_t;
__device__ __forceinline__ pair_t both(float x) {
  pair_t r;
  asm("mov.b64 %0, {%1, %1};" : "=l"(r) : "f"(x));
  return r;
}
__device__ __forceinline__ pair_t join(float x, float y) {
  pair_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(x), "f"(y));
  return r;
}
__device__ __forceinline__ float2 parts(pair_t p) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(p));
  return r;
}
__device__ __forceinline__ pair_t fma2(pair_t a, pair_t b, pair_t c) {
  pair_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ pair_t mul2(pair_t a, pair_t b) {
  pair_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

template <typename T>
__global__ void __launch_bounds__(NARROW_THREADS + 32 * STAGERS, 1) delta_rule_narrow_kernel(DeltaParams p, int vec) {
  constexpr int GROUPS = NARROW_GROUPS, R = Rows<GROUPS>::N, PD = R * GROUPS, NQ = (PD / 4 + 31) / 32;
  constexpr bool AHEAD = NQ <= 2;                             // (longer rows: no registers to fetch a chunk ahead)
  extern __shared__ float4 smem4[];
  const int chunk = p.chunk, cols = p.cols, vdim = p.vdim, per_chunk = chunk / QUAD;
  float4* co = smem4;                                         // [2][per_chunk][CO_COUNT]
  float4* sk = co + 2 * per_chunk * CO_COUNT;                 // [2][chunk][PD / 4]
  float4* sq = sk + 2 * chunk * (PD / 4);                     // [2][chunk][PD / 4]
  float4* sv = sq + 2 * chunk * (PD / 4);                     // [2][per_chunk][cols]: four tokens of a column
  float* so = reinterpret_cast<float*>(sv + 2 * per_chunk * cols);      // [2][chunk][cols]
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.x / p.col_tiles, col0 = (blockIdx.x % p.col_tiles) * cols, h = blockIdx.y;
  const int t0 = p.cu_q[b], t1 = p.cu_q[b + 1];
  if (t1 <= t0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int stager = warp - (cols / NARROW_COLS * GROUPS >> 5);      // negative: a computing warp
  const int chunks = (t1 - t0 + chunk - 1) / chunk;

  // the outputs of a chunk, a warp per token: 32-bit as they are, or normed and gated
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
    const int hq = h / p.qk_group;
    const T* q = static_cast<const T*>(p.q) + (size_t)hq * DIM + 4 * lane;
    const T* k = static_cast<const T*>(p.k) + (size_t)hq * DIM + 4 * lane;
    // lane -> four value columns of one of the group's tokens
    const int v_tok = lane & 3, v_col = (lane >> 2) * 4;
    const T* v = static_cast<const T*>(p.v) + (size_t)h * vdim + col0 + v_col;
    RawFour<T> kq[AHEAD ? 2 * QUAD : 1][NQ], vq;              // k rows, then q rows, of this stager's group; its values
    float4 coefficients;
    // this stager's group of chunk `index` (its first token may lie behind the request's last one)
    auto row_quad = [&](int first, int i, int j, RawFour<T>& to) {
      const int t = first + (i & (QUAD - 1)), left = DIM - 4 * (lane + 32 * j);
      if (t < t1 && left > 0) to.load((i < QUAD ? k + (size_t)t * p.ldk : q + (size_t)t * p.ldq) + 128 * j, left, (vec & 1) != 0);
      else to.zero();
    };
    auto fetch = [&](int index) {
      const int first = t0 + index * chunk + stager * QUAD;
      if (AHEAD) {
#pragma unroll
        for (int i = 0; i < 2 * QUAD; ++i)
#pragma unroll
          for (int j = 0; j < NQ; ++j) row_quad(first, i, j, kq[AHEAD ? i : 0][j]);
      }
      const int left = min(cols, vdim - col0) - v_col;
      if (first + v_tok < t1 && left > 0) vq.load(v + (size_t)(first + v_tok) * p.ldv, left, (vec & 2) != 0);
      else vq.zero();
      if (lane < CO_COUNT && first < t1)
        coefficients = __ldg(p.groups + (group_slot(b, t0, (first - t0) / QUAD) * p.H + h) * CO_COUNT + lane);
    };
    // chunk `index`, whose rows fetch() asked for, to buffer index & 1
    auto stage = [&](int index) {
      const int first = t0 + index * chunk + stager * QUAD, buf = index & 1;
      if (first >= t1) return;
      float4* rows = sk + (size_t)(buf * chunk + stager * QUAD) * (PD / 4) + lane;
#pragma unroll
      for (int i = 0; i < 2 * QUAD; ++i)
#pragma unroll
        for (int j = 0; j < NQ; ++j) {
          if (!AHEAD) row_quad(first, i, j, kq[0][j]);
          if (PD / 4 % 32 == 0 || lane + 32 * j < PD / 4)
            rows[(i < QUAD ? 0 : 2 * chunk * (PD / 4)) + (i & (QUAD - 1)) * (PD / 4) + 32 * j] = kq[AHEAD ? i : 0][j].get();
        }
      float* vt = reinterpret_cast<float*>(sv + (size_t)(buf * per_chunk + stager) * cols) + v_tok;
      const float4 x = vq.get();
      const float e[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (v_col + i < cols) vt[4 * (v_col + i)] = e[i];
      if (lane < CO_COUNT) co[(size_t)(buf * per_chunk + stager) * CO_COUNT + lane] = coefficients;
    };
    const bool works = stager < per_chunk;
    if (works) {
      fetch(0);
      stage(0);
      if (chunks > 1) fetch(1);
    }
    for (int c = 0; c < chunks; ++c) {
      __syncthreads();                    // chunk c is staged, chunk c - 1 is computed
      if (works && c + 1 < chunks) {
        stage(c + 1);
        if (c + 2 < chunks) fetch(c + 2);
      }
      if (c > 0) emit(c - 1, stager, STAGERS);
    }
    __syncthreads();
    emit(chunks - 1, warp, blockDim.x >> 5);
    return;
  }
  // thread (columns 2 lc and 2 lc + 1, group g) keeps the rows 4 (j GROUPS + g) + e
  const int lc = tid / GROUPS * NARROW_COLS, g = tid % GROUPS;
  const int c0 = col0 + lc;
  float* S = p.state + ((size_t)p.state_slots[b] * p.H + h) * DIM * vdim + c0;
  const bool from = p.fresh[b] == 0;
  pair_t s[NARROW_COLS][R / 2];
#pragma unroll
  for (int r = 0; r < R; r += 2) {
    const int row = 4 * ((r >> 2) * GROUPS + g) + (r & 3);
#pragma unroll
    for (int j = 0; j < NARROW_COLS; ++j) {
      const bool live = from && c0 + j < vdim;
      s[j][r / 2] = join(live && row < DIM ? S[(size_t)row * vdim + j] : 0.f, live && row + 1 < DIM ? S[(size_t)(row + 1) * vdim + j] : 0.f);
    }
  }
  constexpr int SPAN = GROUPS / SUMS;                         // lanes that end up with the same sum
  // the sum this lane ends up with: column `column` of the thread's two; p_0 .. p_3, r_0 .. r_3
  const int column = g / (GROUPS / NARROW_COLS), mine = g / SPAN % (2 * QUAD);
  const bool first_lane = g % SPAN == 0, solves = mine == 0 && first_lane, reads_out = mine >= QUAD && first_lane;
  const int leader = lane & ~(GROUPS - 1), own = leader + column * (GROUPS / NARROW_COLS);
  const float4 nothing = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int c = 0; c < chunks; ++c) {
    __syncthreads();
    const int n = min(chunk, t1 - (t0 + c * chunk)), buf = c & 1, groups = (n + QUAD - 1) / QUAD;
#pragma unroll 1
    for (int grp = 0; grp < groups; ++grp) {
      const ulonglong2* kr = reinterpret_cast<const ulonglong2*>(sk + (size_t)(buf * chunk + grp * QUAD) * (PD / 4) + g);
      const ulonglong2* qr = reinterpret_cast<const ulonglong2*>(sq + (size_t)(buf * chunk + grp * QUAD) * (PD / 4) + g);
      const float4* table = co + (size_t)(buf * per_chunk + grp) * CO_COUNT;
      pair_t kx[QUAD][R / 2];
      float acc[SUMS];
#pragma unroll
      for (int i = 0; i < QUAD; ++i) {
        pair_t a[NARROW_COLS], d[NARROW_COLS];
#pragma unroll
        for (int j = 0; j < NARROW_COLS; ++j) a[j] = d[j] = 0;
#pragma unroll
        for (int r4 = 0; r4 < R / 4; ++r4) {
          const ulonglong2 k4 = kr[i * (PD / 4) + r4 * GROUPS], q4 = qr[i * (PD / 4) + r4 * GROUPS];
          kx[i][2 * r4] = k4.x;
          kx[i][2 * r4 + 1] = k4.y;
#pragma unroll
          for (int j = 0; j < NARROW_COLS; ++j) {
            a[j] = fma2(s[j][2 * r4 + 1], k4.y, fma2(s[j][2 * r4], k4.x, a[j]));
            d[j] = fma2(s[j][2 * r4 + 1], q4.y, fma2(s[j][2 * r4], q4.x, d[j]));
          }
        }
#pragma unroll
        for (int j = 0; j < NARROW_COLS; ++j) {
          const float2 ap = parts(a[j]), dp = parts(d[j]);
          acc[j * 2 * QUAD + i] = ap.x + ap.y;
          acc[j * 2 * QUAD + QUAD + i] = dp.x + dp.y;
        }
      }
      // what the lanes that solve and that read out need of the coefficients (a load costs by the lanes that take part)
      const float4 beta = solves ? table[CO_BETA] : nothing, cp = solves ? table[CO_P] : nothing;
      const float4 a0 = solves ? table[CO_A] : nothing, a1 = solves ? table[CO_A + 1] : nothing;
      const float4 vv = solves ? sv[(size_t)(buf * per_chunk + grp) * cols + lc + column] : nothing;
      const float4 ob = reads_out ? table[CO_O + mine - QUAD] : nothing;
      const float fade = reads_out ? reinterpret_cast<const float*>(table + CO_R)[mine - QUAD] : 0.f;
      const float4 w = table[CO_W];
      const float faded = reinterpret_cast<const float*>(table)[CO_TOTAL];
      // the sums spread over the lanes: every exchange halves what a lane still adds up
      int kept = SUMS;
#pragma unroll
      for (int o = GROUPS / 2; o >= 1; o >>= 1) {
        if (kept > 1) {
          kept >>= 1;
          const bool upper = (g & o) != 0;
#pragma unroll
          for (int i = 0; i < SUMS / 2; ++i) {
            if (i >= kept) continue;
            const float send = upper ? acc[i] : acc[i + kept], keep = upper ? acc[i + kept] : acc[i];
            acc[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
          }
        } else {
          acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], o);
        }
      }
      const float p0 = acc[0], p1 = __shfl_sync(0xffffffffu, acc[0], own + SPAN);          // (p_0 is the solving lane's own)
      const float p2 = __shfl_sync(0xffffffffu, acc[0], own + 2 * SPAN), p3 = __shfl_sync(0xffffffffu, acc[0], own + 3 * SPAN);
      float z[QUAD], u[NARROW_COLS][QUAD];
      z[0] = fmaf(-cp.x, p0, beta.x * vv.x);
      z[1] = fmaf(-a0.x, z[0], fmaf(-cp.y, p1, beta.y * vv.y));
      z[2] = fmaf(-a0.z, z[1], fmaf(-a0.y, z[0], fmaf(-cp.z, p2, beta.z * vv.z)));
      z[3] = fmaf(-a1.y, z[2], fmaf(-a1.x, z[1], fmaf(-a0.w, z[0], fmaf(-cp.w, p3, beta.w * vv.w))));
#pragma unroll
      for (int j = 0; j < NARROW_COLS; ++j)
#pragma unroll
        for (int i = 0; i < QUAD; ++i) u[j][i] = __shfl_sync(0xffffffffu, z[i], leader + j * (GROUPS / NARROW_COLS));
      const pair_t total = both(faded);
#pragma unroll
      for (int j = 0; j < NARROW_COLS; ++j) {
        const pair_t w0 = both(w.x * u[j][0]), w1 = both(w.y * u[j][1]), w2 = both(w.z * u[j][2]), w3 = both(w.w * u[j][3]);
#pragma unroll
        for (int r = 0; r < R / 2; ++r)
          s[j][r] = fma2(kx[3][r], w3, fma2(kx[2][r], w2, fma2(kx[1][r], w1, fma2(kx[0][r], w0, mul2(total, s[j][r])))));
      }
      float out = fade * acc[0];
      out = fmaf(ob.x, column ? u[1][0] : u[0][0], out);
      out = fmaf(ob.y, column ? u[1][1] : u[0][1], out);
      out = fmaf(ob.z, column ? u[1][2] : u[0][2], out);
      out = fmaf(ob.w, column ? u[1][3] : u[0][3], out);
      if (reads_out) so[(buf * chunk + grp * QUAD + mine - QUAD) * cols + lc + column] = out;
    }
  }
  __syncthreads();
#pragma unroll
  for (int r = 0; r < R; r += 2) {
    const int row = 4 * ((r >> 2) * GROUPS + g) + (r & 3);
#pragma unroll
    for (int j = 0; j < NARROW_COLS; ++j) {
      if (c0 + j >= vdim) continue;
      const float2 x = parts(s[j][r / 2]);
      if (row < DIM) S[(size_t)row * vdim + j] = x.x;
      if (row + 1 < DIM) S[(size_t)(row + 1) * vdim + j] = x.y;
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
  const int step = NARROW_COLS * (32 / NARROW_GROUPS);
  const int most = NARROW_THREADS / NARROW_GROUPS * NARROW_COLS;
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

template <typename Kernel>
int allow_smem(Kernel kernel, size_t smem, size_t& allowed) {
  if (smem <= allowed) return 0;
  cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return ts_fail("delta_rule: %zu bytes of shared memory: %s", smem, cudaGetErrorString(e));
  allowed = smem;
  return 0;
}

template <typename T>
int launch_wide(DeltaParams p, int num_requests, int max_q_len, cudaStream_t stream) {
  constexpr int PD = rows_of(WIDE_GROUPS) * WIDE_GROUPS;
  auto bytes = [&](int chunk) { return (size_t)2 * chunk * (4 + 2 * PD + 2 * p.cols) * sizeof(float); };
  p.chunk = max_q_len < MAX_CHUNK ? max_q_len : MAX_CHUNK;
  while (p.chunk > 1 && bytes(p.chunk) > 200 * 1024) p.chunk /= 2;
  static size_t allowed = 48 * 1024;
  if (int rc = allow_smem(delta_rule_wide_kernel<T>, bytes(p.chunk), allowed)) return rc;
  TS_LAUNCH("delta_rule", delta_rule_wide_kernel<T>, dim3(num_requests * p.col_tiles, p.H), p.cols / 4 * WIDE_GROUPS + 32 * STAGERS,
            bytes(p.chunk), stream, p);
  return 0;
}

template <typename T>
int launch_narrow(DeltaParams p, int num_requests, int max_q_len, cudaStream_t stream) {
  constexpr int PD = rows_of(NARROW_GROUPS) * NARROW_GROUPS;
  auto bytes = [&](int chunk) {
    return (size_t)2 * (chunk / QUAD) * CO_COUNT * sizeof(float4) + (size_t)2 * chunk * (2 * PD + 2 * p.cols) * sizeof(float);
  };
  p.chunk = MAX_CHUNK;
  while (p.chunk > QUAD && bytes(p.chunk) > 200 * 1024) p.chunk /= 2;
  const uintptr_t at = (uintptr_t)p.q | (uintptr_t)p.k;
  const int vec = (DIM % 4 == 0 && p.ldq % 4 == 0 && p.ldk % 4 == 0 && at % (4 * sizeof(T)) == 0 ? 1 : 0) |
                  (p.cols % 4 == 0 && p.vdim % 4 == 0 && p.ldv % 4 == 0 && (uintptr_t)p.v % (4 * sizeof(T)) == 0 ? 2 : 0);
  const int qk_heads = p.H / p.qk_group;
  TS_LAUNCH("delta_prepare", delta_prepare_kernel<T>,
            dim3((max_q_len + QUAD - 1) / QUAD, (qk_heads + PREPARE_WARPS - 1) / PREPARE_WARPS, num_requests), 32 * PREPARE_WARPS, 0, stream, p, vec & 1);
  static size_t allowed = 48 * 1024;
  if (int rc = allow_smem(delta_rule_narrow_kernel<T>, bytes(p.chunk), allowed)) return rc;
  TS_LAUNCH("delta_rule", delta_rule_narrow_kernel<T>, dim3(num_requests * p.col_tiles, p.H), p.cols / NARROW_COLS * NARROW_GROUPS + 32 * STAGERS,
            bytes(p.chunk), stream, p, vec);
  return 0;
}

template <typename T>
int run(DeltaParams& p, bool narrow, int num_requests, int max_q_len, int num_tokens, cudaStream_t stream) {
  if (int rc = narrow ? launch_narrow<T>(p, num_requests, max_q_len, stream) : launch_wide<T>(p, num_requests, max_q_len, stream)) return rc;
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

// floats of the coefficients' scratch that the narrow form needs
TS_EXPORT long long ts_delta_rule_scratch(int num_tokens, int num_requests, int H) {
  return ((long long)num_tokens / QUAD + num_requests + 1) * H * CO_COUNT * 4;
}

// raw [T, H vdim]: scratch of heads that are spread over several blocks, else null; groups: scratch of the narrow form
TS_EXPORT int ts_delta_rule(int dtype, const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv,
                            const void* gate, long long ldg, const float* logits, long long ld_logits, const void* bias,
                            int bias_is_f32, const void* rate, int rate_is_f32, float q_scale, float* state, const int* state_slots,
                            const int* fresh, const int* cu_q, int num_requests, int max_q_len, int num_tokens,
                            const void* norm_weight, int norm_weight_is_f32, float eps, void* out, long long ldo, float* raw, int H,
                            int vdim, int qk_group, int tile, float* groups, cudaStream_t stream) {
  TS_REQUIRE(num_requests > 0 && num_requests <= 65535 && H > 0 && H <= 65535 && vdim > 0 && num_tokens > 0 && max_q_len > 0, "delta_rule: empty input");
  TS_REQUIRE(qk_group >= 1 && H % qk_group == 0, "delta_rule: %d heads in groups of %d", H, qk_group);
  TS_REQUIRE(q && k && v && gate && logits && bias && rate && state && state_slots && fresh && cu_q && norm_weight && out,
             "delta_rule: a null operand");
  TS_REQUIRE(tile <= 0 || (groups && (uintptr_t)groups % 16 == 0), "delta_rule: the narrow form needs scratch for its coefficients");
  TS_REQUIRE(ld_logits >= 2 * H, "delta_rule: two logits per head and token");
  const int cols = tile > 0 ? narrow_columns(vdim, tile) : wide_columns(vdim), col_tiles = (vdim + cols - 1) / cols;
  TS_REQUIRE((col_tiles > 1) == (raw != nullptr), "delta_rule: heads spread over %d blocks of %d columns: a 32-bit scratch or none", col_tiles, cols);
  DeltaParams p{q, k, v, gate, ldq, ldk, ldv, ldg, logits, ld_logits, VecParam{bias, bias_is_f32}, VecParam{rate, rate_is_f32},
                q_scale, state, state_slots, fresh, cu_q, VecParam{norm_weight, norm_weight_is_f32}, eps, out, ldo, raw, H, vdim,
                qk_group, cols, col_tiles, 0, reinterpret_cast<float4*>(groups)};
  if (dtype == TS_F32) return run<float>(p, tile > 0, num_requests, max_q_len, num_tokens, stream);
  if (dtype == TS_BF16) return run<__nv_bfloat16>(p, tile > 0, num_requests, max_q_len, num_tokens, stream);
  return ts_fail("delta_rule: unknown dtype %d", dtype);
}
