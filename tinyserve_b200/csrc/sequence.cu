// Kernels on rows of a step that depend on a token's neighbours in its own sequence, and the
// small 32-bit steps around recurrent mixers.  All arithmetic is 32-bit; inputs and outputs are
// float or bfloat16 (an `is_f32` flag per operand, so that the 32-bit residual stream and the
// projections of the compute type go through the same kernels).
//
//  * ts_add_position_rows: residual[t] += table[positions[t]] (learned positions).
//  * ts_causal_conv: y_t = (x_t +) (bias +) sum_j w[:, j] x_(t - taps + 1 + j) per channel, zeros
//    before a sequence's start, optionally through silu.  The last taps - 1 inputs of every
//    request live in its state slot and are replaced at the end of the step.
//  * ts_conv_heads_kvwrite: the same convolution on the rows of a fused q/k/v projection, whose results
//    go straight to padded query rows (times a factor per head) and to the token's cache slot.
//  * ts_group_norm / ts_group_norm_add: RMS norm of every one of `groups` equal consecutive parts
//    of a row, times a weight; written out (optionally only some rows), or added to the 32-bit
//    residual.
//  * ts_axpby: out = a x + b y.
//  * ts_gate_columns: out[t, h * vdim + c] = x[t, h, c] * sigmoid(gate[t, h * vdim + c]) for heads
//    stored wider than their values.
//  * ts_joint_norm_kvwrite: q and k of a token normed over all their heads at once (one weight
//    per column), optionally rotated, q to padded rows for the attention kernels, k and v to the token's cache
//    slot; v may be the k rows as they come.
//  * ts_mlstm_gates: the stabilised gates of a matrix memory with exponential input gate:
//    m_t = max(f_t + m_(t-1), i_t), keep_t = exp(f_t + m_(t-1) - m_t), write_t = exp(i_t - m_t),
//    floor_t = exp(-m_t); i and f capped by cap tanh(. / cap), f through log-sigmoid; m is state.
//  * ts_mlstm_finish: o / (max(|n . q|, floor) + 1e-6), RMS per head, weight, sigmoid gate.
//  * ts_ssm_finish: (y + D x) silu(z), RMS in groups over all heads, weight.
#include "common.cuh"

TS_DEFINE_LAST_ERROR()

namespace {

// an operand that is float or bfloat16, chosen at run time
struct Rows {
  const void* ptr;
  long long ld;
  int is_f32;
  __device__ __forceinline__ float at(size_t row, int col) const {
    return is_f32 ? static_cast<const float*>(ptr)[row * ld + col]
                  : __bfloat162float(static_cast<const __nv_bfloat16*>(ptr)[row * ld + col]);
  }
};
struct RowsOut {
  void* ptr;
  long long ld;
  int is_f32;
  __device__ __forceinline__ void put(size_t row, int col, float v) const {
    if (is_f32) static_cast<float*>(ptr)[row * ld + col] = v;
    else static_cast<__nv_bfloat16*>(ptr)[row * ld + col] = __float2bfloat16_rn(v);
  }
};

__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float log_sigmoid_f(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// ------------------------------------------------------------------ learned positions
__global__ void add_position_rows_kernel(float* __restrict__ residual, VecParam table, const int* __restrict__ positions,
                                         int num_positions, int n) {
  pdl_trigger();
  pdl_wait();
  const size_t t = blockIdx.x;
  const int p = positions[t];
  if (p < 0 || p >= num_positions) {
    if (threadIdx.x == 0) ts_raise_status(TS_STATUS_BOUNDS, TS_BAD_POSITION);
    return;
  }
  for (int i = threadIdx.x; i < n; i += blockDim.x) residual[t * n + i] += table[(size_t)p * n + i];
}

// ------------------------------------------------------------------ causal convolution over time
constexpr int CONV_TILE = 32;        // tokens of a block
constexpr int CONV_THREADS = 128;    // channels of a block
constexpr int CONV_MAX_TAPS = 8;

struct ConvParams {
  Rows x;
  RowsOut y;
  VecParam w;              // [C, taps]
  VecParam bias;           // [C] or null
  float* state;            // [slots, taps - 1, C]: a request's last inputs, oldest first
  const int* state_slots; const int* fresh; const int* cu_q;
  int C, add_input, silu;
};

// Thread = one channel over CONV_TILE tokens of one request, its last TAPS - 1 inputs in
// registers.  The block of a request's first tile also makes the request's new state: it is the
// only one that reads the old state, so nobody reads what it overwrites.
template <int TAPS>
__global__ void __launch_bounds__(CONV_THREADS) causal_conv_kernel(ConvParams p) {
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.z;
  const int t0 = p.cu_q[b], n = p.cu_q[b + 1] - t0;
  const int first = blockIdx.y * CONV_TILE;
  const int c = blockIdx.x * CONV_THREADS + threadIdx.x;
  if (first >= n || c >= p.C) return;
  constexpr int H = TAPS - 1;
  float w[TAPS];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) w[j] = p.w[(size_t)c * TAPS + j];
  const float bias = p.bias.ptr ? p.bias[c] : 0.f;
  float* st = p.state + (size_t)p.state_slots[b] * H * p.C + c;
  const bool is_fresh = p.fresh[b] != 0;
  float old[H > 0 ? H : 1];
  if (first < H) {
#pragma unroll
    for (int i = 0; i < H; ++i) old[i] = is_fresh ? 0.f : st[(size_t)i * p.C];
  }
  // hist[i] = input at token first - H + i of this portion (negative tokens: the state)
  float hist[H > 0 ? H : 1];
#pragma unroll
  for (int i = 0; i < H; ++i) {
    const int tok = first - H + i;
    hist[i] = tok >= 0 ? p.x.at(t0 + tok, c) : old[i];      // (tok < 0 only in a request's first tile)
  }
  const int last = min(n, first + CONV_TILE);
  for (int tok = first; tok < last; ++tok) {
    const float cur = p.x.at(t0 + tok, c);
    float acc = bias + w[H] * cur;
#pragma unroll
    for (int i = 0; i < H; ++i) acc = fmaf(w[i], hist[i], acc);
    if (p.silu) acc = silu_f(acc);
    if (p.add_input) acc += cur;
    p.y.put(t0 + tok, c, acc);
#pragma unroll
    for (int i = 0; i + 1 < H; ++i) hist[i] = hist[i + 1];
    if (H > 0) hist[H - 1] = cur;
  }
  if (first == 0) {
    // new state: inputs at tokens n - H .. n - 1 (tokens below 0: the old state, shifted)
#pragma unroll
    for (int i = 0; i < H; ++i) {
      const int tok = n - H + i;
      float v = 0.f;
      if (tok >= 0) v = p.x.at(t0 + tok, c);
      else {
#pragma unroll
        for (int j = 0; j < H; ++j)
          if (j == tok + H) v = old[j];
      }
      st[(size_t)i * p.C] = v;
    }
  }
}

// ------------------------------------------------------------------ causal convolution of q, k, v + cache write
// The rows x [T, H dim (q) | G dim (k) | G vdim (v)] of a fused projection pass the convolution and leave as what
// the attention kernels read: query rows [T, H, stored] (times one factor per head), keys and values at the cache
// slots of their tokens, heads padded with zeros to `stored`.  G = 0: queries only (the keys and values are
// another layer's).  A thread owns VEC neighbouring columns of a stored head over HEADS_TILE tokens of one request,
// whose loads are all in flight together (the tokens before them are read again: they come from L1 and L2);
// the block of a request's first tile also replaces the request's state, as in causal_conv_kernel.
struct ConvHeads {
  const void* x; long long ldx;
  VecParam w;                       // [TAPS, channels], so that a warp's loads are contiguous; null (TAPS 1): the rows as they are
  VecParam factor;                  // [H] or null
  float* state;                     // [slots, TAPS - 1, channels]
  const int* state_slots; const int* fresh; const int* cu_q;
  int H, G, dim, vdim, stored, page_size, page_shift, channels;     // page_shift: log2(page_size), or -1
  void* q_out; void* k_cache; void* v_cache;
  const int* slot_mapping;
};
constexpr int HEADS_TILE = 8;        // tokens of a block: at least CONV_MAX_TAPS - 1

template <typename T, int VEC> struct Pack;
template <> struct Pack<float, 1> {
  static __device__ __forceinline__ void load(const float* p, float (&v)[1]) { v[0] = *p; }
  static __device__ __forceinline__ void store(float* p, const float (&v)[1]) { *p = v[0]; }
};
template <> struct Pack<float, 2> {
  static __device__ __forceinline__ void load(const float* p, float (&v)[2]) {
    const float2 q = *reinterpret_cast<const float2*>(p);
    v[0] = q.x; v[1] = q.y;
  }
  static __device__ __forceinline__ void store(float* p, const float (&v)[2]) { *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]); }
};
template <> struct Pack<__nv_bfloat16, 1> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[1]) { v[0] = __bfloat162float(*p); }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[1]) { *p = __float2bfloat16_rn(v[0]); }
};
template <> struct Pack<__nv_bfloat16, 2> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[2]) {
    const __nv_bfloat162 q = *reinterpret_cast<const __nv_bfloat162*>(p);
    v[0] = __low2float(q); v[1] = __high2float(q);
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[2]) {
    *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v[0], v[1]);
  }
};

template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(CONV_THREADS) conv_heads_kvwrite_kernel(ConvHeads p) {
  pdl_trigger();
  constexpr int H1 = TAPS - 1;
  const int col = (blockIdx.x * CONV_THREADS + threadIdx.x) * VEC;      // over the stored heads: q, then k, then v
  const int head = col / p.stored, d = col % p.stored;
  const bool is_q = head < p.H, is_v = head >= p.H + p.G;
  const int g = is_q ? head : (is_v ? head - p.H - p.G : head - p.H);
  const bool live = head < p.H + 2 * p.G;
  const bool real = live && d < (is_v ? p.vdim : p.dim);                // else: a column of zeros
  // the projection's column, which is also the convolution's channel
  const int c = is_q ? g * p.dim + d : (is_v ? (p.H + p.G) * p.dim + g * p.vdim + d : p.H * p.dim + g * p.dim + d);
  float w[TAPS][VEC];
  float factor = 1.f;
  if (real) {      // (weights are constants: fetched while the predecessor still runs)
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const size_t at = (size_t)j * p.channels + c;
      if (p.w.ptr == nullptr) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) w[j][e] = 1.f;
      } else if (p.w.is_f32) {
        Pack<float, VEC>::load(static_cast<const float*>(p.w.ptr) + at, w[j]);
      } else {
        Pack<__nv_bfloat16, VEC>::load(static_cast<const __nv_bfloat16*>(p.w.ptr) + at, w[j]);
      }
    }
    if (is_q && p.factor.ptr) factor = p.factor[head];
  }
  pdl_wait();
  const int b = blockIdx.z;
  const int t0 = p.cu_q[b], n = p.cu_q[b + 1] - t0;
  const int first = blockIdx.y * HEADS_TILE;
  if (first >= n || !live) return;
  const int count = min(HEADS_TILE, n - first);
  const int tok = t0 + first;
  // where token k's result goes: the query row, or the token's place in the cache (null: nowhere)
  T* const q_row = static_cast<T*>(p.q_out) + ((size_t)tok * p.H + head) * p.stored + d;
  T* const cache = static_cast<T*>(is_v ? p.v_cache : p.k_cache) + d;
  auto place = [&](int k) -> T* {
    if (is_q) return q_row + (size_t)k * p.H * p.stored;
    const int slot = p.slot_mapping[tok + k];
    if (slot < 0) return nullptr;
    const int page = p.page_shift >= 0 ? slot >> p.page_shift : slot / p.page_size;
    return cache + ((size_t)(page * p.G + g) * p.page_size + (slot - page * p.page_size)) * p.stored;
  };
  if (!real) {
    const float zeros[VEC] = {};
    for (int k = 0; k < count; ++k)
      if (T* dst = place(k)) Pack<T, VEC>::store(dst, zeros);
    return;
  }
  const T* x = static_cast<const T*>(p.x) + c;
  const T* row = x + (size_t)tok * p.ldx;
  // in[i] = input at token first - H1 + i of this portion (before the portion: the state)
  float in[H1 + HEADS_TILE][VEC];
  T* dst[HEADS_TILE];
#pragma unroll
  for (int k = 0; k < HEADS_TILE; ++k)
    if (k < count) {
      Pack<T, VEC>::load(row + (size_t)k * p.ldx, in[H1 + k]);
      dst[k] = place(k);
    }
  float* st = nullptr;
  bool is_fresh = false;
  if (H1 > 0) {
    if (first == 0) {
      st = p.state + (size_t)p.state_slots[b] * H1 * p.channels + c;
      is_fresh = p.fresh[b] != 0;
#pragma unroll
      for (int i = 0; i < H1; ++i)
#pragma unroll
        for (int e = 0; e < VEC; ++e) in[i][e] = is_fresh ? 0.f : st[(size_t)i * p.channels + e];
    } else {
#pragma unroll
      for (int i = 0; i < H1; ++i) Pack<T, VEC>::load(row - (size_t)(H1 - i) * p.ldx, in[i]);
    }
  }
#pragma unroll
  for (int k = 0; k < HEADS_TILE; ++k) {
    if (k < count && dst[k] != nullptr) {
      float y[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        float acc = w[H1][e] * in[H1 + k][e];
#pragma unroll
        for (int i = 0; i < H1; ++i) acc = fmaf(w[i][e], in[k + i][e], acc);
        y[e] = acc * factor;
      }
      Pack<T, VEC>::store(dst[k], y);
    }
  }
  if (H1 > 0 && first == 0) {
    // new state: inputs at tokens n - H1 .. n - 1; tokens below 0 are the old state's row i + n, which an ascending
    // walk has not overwritten yet
#pragma unroll
    for (int i = 0; i < H1; ++i) {
      const int at = n - H1 + i;
      float v[VEC];
      if (at >= 0) {
        Pack<T, VEC>::load(x + (size_t)(t0 + at) * p.ldx, v);
      } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] = is_fresh ? 0.f : st[(size_t)(i + n) * p.channels + e];
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) st[(size_t)i * p.channels + e] = v[e];
    }
  }
}

template <typename T, int VEC>
int launch_conv_heads(const ConvHeads& p, int taps, dim3 grid, cudaStream_t stream) {
  switch (taps) {
#define TS_CONV_CASE(N) \
    case N: TS_LAUNCH("conv_heads_kvwrite", (conv_heads_kvwrite_kernel<T, VEC, N>), grid, CONV_THREADS, 0, stream, p); break;
    TS_CONV_CASE(1) TS_CONV_CASE(2) TS_CONV_CASE(3) TS_CONV_CASE(4) TS_CONV_CASE(5) TS_CONV_CASE(6) TS_CONV_CASE(7)
    TS_CONV_CASE(8)
#undef TS_CONV_CASE
  }
  return 0;
}

// ------------------------------------------------------------------ RMS norm in groups
// a block per (row, group); y = x / sqrt(mean(x^2) + eps) * w over each group of n / groups.  A thread keeps
// its first ROW_HOLD elements in registers between the sum and the scaling, and reads any further ones twice.
constexpr int ROW_HOLD = 8;

// threads of a block that walks `per` elements of a row: four elements a thread, 32 to 256 threads
inline int row_threads(int per) { return per >= 1024 ? 256 : (per >= 512 ? 128 : (per >= 256 ? 64 : 32)); }

template <bool ADD>
__global__ void group_norm_kernel(Rows x, VecParam w, const int* __restrict__ rows, int groups, int n, float eps,
                                  RowsOut out, float* __restrict__ residual) {
  __shared__ float scratch[33];
  pdl_trigger();
  pdl_wait();
  const size_t o = blockIdx.x;
  const size_t t = rows ? (size_t)rows[o] : o;
  const int per = n / groups, base = blockIdx.y * per;
  float held[ROW_HOLD], acc = 0.f;
#pragma unroll
  for (int j = 0; j < ROW_HOLD; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    held[j] = i < per ? x.at(t, base + i) : 0.f;
    acc = fmaf(held[j], held[j], acc);
  }
  for (int i = threadIdx.x + ROW_HOLD * blockDim.x; i < per; i += blockDim.x) {
    const float v = x.at(t, base + i);
    acc = fmaf(v, v, acc);
  }
  const float rstd = rsqrtf(block_sum(acc, scratch) / (float)per + eps);
  auto put = [&](int i, float v) {
    const int col = base + i;
    const float y = v * rstd * w[col];
    if (ADD) residual[t * n + col] += y;
    else out.put(o, col, y);
  };
#pragma unroll
  for (int j = 0; j < ROW_HOLD; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i < per) put(i, held[j]);
  }
  for (int i = threadIdx.x + ROW_HOLD * blockDim.x; i < per; i += blockDim.x) put(i, x.at(t, base + i));
}

// ------------------------------------------------------------------ a x + b y
__global__ void axpby_kernel(Rows x, Rows y, float a, float b, RowsOut out, long long count) {
  pdl_trigger();
  pdl_wait();
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < count; i += (long long)gridDim.x * blockDim.x)
    out.put((size_t)i, 0, a * x.at((size_t)i, 0) + b * y.at((size_t)i, 0));
}

// ------------------------------------------------------------------ heads times an element-wise sigmoid gate
__global__ void gate_columns_kernel(Rows x, Rows gate, RowsOut out, int H, int stored, int vdim) {
  pdl_trigger();
  pdl_wait();
  const size_t t = blockIdx.x;
  for (int i = threadIdx.x; i < H * vdim; i += blockDim.x) {
    const int h = i / vdim, c = i % vdim;
    out.put(t, i, x.at(t, h * stored + c) * sigmoid_f(gate.at(t, i)));
  }
}

// ------------------------------------------------------------------ q and k normed over all heads, cache write
struct JointNorm {
  Rows q, k, v;
  VecParam qw, kw;         // [H dim], [G dim]; null: no norm
  float eps;
  int H, G, dim, vdim, stored, page_size;
  void* q_out;             // [T, H, stored]
  void* k_cache; void* v_cache;     // [pages, G, page, stored]
  const int* slot_mapping;          // null: nothing is written
  int out_is_f32;
  // rotary positions after the norm, on the first `rot` columns of every head (0: none); pairs (2i, 2i + 1), or (i, i + rot / 2)
  const float* cos; const float* sin; const int* positions;
  int rot, interleaved;
};

__global__ void joint_norm_kvwrite_kernel(JointNorm p) {
  __shared__ float scratch[33];
  pdl_trigger();
  pdl_wait();
  const size_t t = blockIdx.x;
  const int nq = p.H * p.dim, nk = p.G * p.dim, half = p.rot >> 1;
  float aq = 0.f, ak = 0.f;
  if (p.qw.ptr) {
    for (int i = threadIdx.x; i < nq; i += blockDim.x) { const float v = p.q.at(t, i); aq = fmaf(v, v, aq); }
    for (int i = threadIdx.x; i < nk; i += blockDim.x) { const float v = p.k.at(t, i); ak = fmaf(v, v, ak); }
  }
  const float rq = p.qw.ptr ? rsqrtf(block_sum(aq, scratch) / (float)nq + p.eps) : 1.f;
  const float rk = p.qw.ptr ? rsqrtf(block_sum(ak, scratch) / (float)nk + p.eps) : 1.f;
  const size_t angles = p.rot > 0 ? (size_t)p.positions[t] * half : 0;
  // column d of the head at `base` of x's row, normed and rotated
  auto element = [&](const Rows& x, const VecParam& w, float r, int base, int d) {
    auto normed = [&](int e) {
      const float v = x.at(t, base + e) * r;
      return w.ptr ? v * w[base + e] : v;
    };
    const float a = normed(d);
    if (d >= p.rot) return a;
    const int j = p.interleaved ? d >> 1 : (d < half ? d : d - half);
    const bool first = p.interleaved ? !(d & 1) : d < half;
    const float b = normed(p.interleaved ? d ^ 1 : (first ? d + half : d - half));
    const float c = p.cos[angles + j], s = p.sin[angles + j];
    return first ? a * c - b * s : a * c + b * s;
  };
  RowsOut qo{p.q_out, (long long)p.H * p.stored, p.out_is_f32};
  for (int i = threadIdx.x; i < p.H * p.stored; i += blockDim.x) {
    const int h = i / p.stored, d = i % p.stored;
    qo.put(t, i, d < p.dim ? element(p.q, p.qw, rq, h * p.dim, d) : 0.f);
  }
  if (!p.slot_mapping) return;
  const int slot = p.slot_mapping[t];
  if (slot < 0) return;
  const size_t page = slot / p.page_size, in_page = slot % p.page_size;
  for (int i = threadIdx.x; i < p.G * p.stored; i += blockDim.x) {
    const int g = i / p.stored, d = i % p.stored;
    const float kv = d < p.dim ? element(p.k, p.kw, rk, g * p.dim, d) : 0.f;
    const float vv = d < p.vdim ? p.v.at(t, g * p.vdim + d) : 0.f;
    const size_t at = ((page * p.G + g) * p.page_size + in_page) * p.stored + d;
    if (p.out_is_f32) {
      static_cast<float*>(p.k_cache)[at] = kv;
      static_cast<float*>(p.v_cache)[at] = vv;
    } else {
      static_cast<__nv_bfloat16*>(p.k_cache)[at] = __float2bfloat16_rn(kv);
      static_cast<__nv_bfloat16*>(p.v_cache)[at] = __float2bfloat16_rn(vv);
    }
  }
}

// The same for sizes in multiples of 8 and neighbouring pairs: a thread keeps up to JOINT_PACKS runs of eight
// columns of q and k between the sums and the results, 16 bytes of bfloat16 each.
constexpr int JOINT_PACKS = 4, JOINT_THREADS = 256;

__device__ __forceinline__ void weight8(const VecParam& w, int c, float (&v)[8]) {
  if (w.is_f32) load8<float>(static_cast<const float*>(w.ptr) + c, v);
  else load8<__nv_bfloat16>(static_cast<const __nv_bfloat16*>(w.ptr) + c, v);
}

template <typename T>
__global__ void __launch_bounds__(JOINT_THREADS) joint_norm_kvwrite_vec_kernel(JointNorm p) {
  __shared__ float2 parts[JOINT_THREADS / 32];
  pdl_trigger();
  const int per = p.dim >> 3, packs_q = p.H * per, packs = packs_q + p.G * per;
  pdl_wait();
  const size_t t = blockIdx.x;
  const T* q = static_cast<const T*>(p.q.ptr) + t * p.q.ld;
  const T* k = static_cast<const T*>(p.k.ptr) + t * p.k.ld;
  const T* v = static_cast<const T*>(p.v.ptr) + t * p.v.ld;
  const int slot = p.slot_mapping ? p.slot_mapping[t] : -1;
  const size_t angles = p.rot > 0 ? (size_t)p.positions[t] * (p.rot >> 1) : 0;
  float x[JOINT_PACKS][8], aq = 0.f, ak = 0.f;
#pragma unroll
  for (int j = 0; j < JOINT_PACKS; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i >= packs) continue;
    const bool is_q = i < packs_q;
    load8<T>(is_q ? q + i * 8 : k + (i - packs_q) * 8, x[j]);
    float sum = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) sum = fmaf(x[j][e], x[j][e], sum);
    if (is_q) aq += sum;
    else ak += sum;
  }
  aq = warp_sum(aq);
  ak = warp_sum(ak);
  if ((threadIdx.x & 31) == 0) parts[threadIdx.x >> 5] = make_float2(aq, ak);
  __syncthreads();
  aq = ak = 0.f;
  for (int w = 0; w < (int)(blockDim.x >> 5); ++w) {
    aq += parts[w].x;
    ak += parts[w].y;
  }
  const float rq = rsqrtf(aq / (float)(packs_q * 8) + p.eps), rk = rsqrtf(ak / (float)((packs - packs_q) * 8) + p.eps);
  T* q_out = static_cast<T*>(p.q_out) + t * p.H * p.stored;
  const size_t page = slot >= 0 ? slot / p.page_size : 0, in_page = slot >= 0 ? slot % p.page_size : 0;
  auto cache = [&](void* base, int g) { return static_cast<T*>(base) + ((page * p.G + g) * p.page_size + in_page) * p.stored; };
  const bool tied = p.v.ptr == p.k.ptr && p.vdim == p.dim;      // the values are the k rows as they came
#pragma unroll
  for (int j = 0; j < JOINT_PACKS; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i >= packs) continue;
    const bool is_q = i < packs_q;
    const int col = (is_q ? i : i - packs_q) * 8, head = col / p.dim, d = col - head * p.dim;
    if (!is_q && slot < 0) continue;
    if (!is_q && tied) store8<T>(cache(p.v_cache, head) + d, x[j]);
    float w[8];
    weight8(is_q ? p.qw : p.kw, col, w);
    const float r = is_q ? rq : rk;
#pragma unroll
    for (int e = 0; e < 8; ++e) x[j][e] *= r * w[e];
    if (d < p.rot) turn_pairs8(x[j], p.cos, p.sin, angles + (d >> 1));
    store8<T>((is_q ? q_out + (size_t)head * p.stored : cache(p.k_cache, head)) + d, x[j]);
  }
  const float zeros[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
  if (p.stored > p.dim) {
    const int pad = (p.stored - p.dim) >> 3, heads = slot >= 0 ? p.H + p.G : p.H;
    for (int i = threadIdx.x; i < heads * pad; i += blockDim.x) {
      const int head = i / pad, d = p.dim + (i - head * pad) * 8;
      store8<T>((head < p.H ? q_out + (size_t)head * p.stored : cache(p.k_cache, head - p.H)) + d, zeros);
    }
  }
  if (slot < 0) return;
  const int vper = p.stored >> 3, from = tied ? p.vdim >> 3 : 0, span = vper - from;
  for (int i = threadIdx.x; i < p.G * span; i += blockDim.x) {
    const int g = i / span, d = (from + i - g * span) * 8;
    float y[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (d < p.vdim) load8<T>(v + g * p.vdim + d, y);
    store8<T>(cache(p.v_cache, g) + d, y);
  }
}

// ------------------------------------------------------------------ gates of a matrix memory with exponential input gate
// m_t = max(f_t + m_(t-1), i_t) is a chain of maps x -> max(F + x, I); two such maps compose to another one,
// (F2, I2) o (F1, I1) = (F1 + F2, max(I1 + F2, I2)), so 32 tokens are a warp scan, and a span of tokens has
// one map that can be applied before the span's own maximum is known.
//
// A warp walks the tokens [a, e) of head h 32 at a time.  EMIT: from the maximum m before token a it writes
// keep_t, write_t, exp(-m_t) and returns the maximum after the span in .x.  Otherwise it writes nothing and
// returns the span's map (F, I).
template <bool EMIT>
__device__ __forceinline__ float2 mlstm_gates_walk(const float* __restrict__ raw, long long ld, float cap, int H, int h,
                                                   int a, int e, float m, float* __restrict__ keep,
                                                   float* __restrict__ write, float* __restrict__ floor_) {
  const int lane = threadIdx.x & 31;
  const float inv_cap = 1.f / cap;
  float Fs = 0.f, Is = -INFINITY;
  for (int base = a; base < e; base += 32) {
    const int t = base + lane;
    const bool live = t < e;
    float gi = -INFINITY, gf = 0.f;      // (a lane behind the span holds the identity map)
    if (live) {
      gi = cap * tanhf(raw[(size_t)t * ld + h] * inv_cap);
      gf = log_sigmoid_f(cap * tanhf(raw[(size_t)t * ld + H + h] * inv_cap));
    }
    float F = gf, I = gi;       // the map of tokens base .. t, composed
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float pF = __shfl_up_sync(0xffffffffu, F, o), pI = __shfl_up_sync(0xffffffffu, I, o);
      if (lane >= o) {
        I = fmaxf(pI + F, I);
        F = pF + F;
      }
    }
    if (EMIT) {
      const float m_t = fmaxf(F + m, I);
      float m_prev = __shfl_up_sync(0xffffffffu, m_t, 1);
      if (lane == 0) m_prev = m;
      if (live) {
        keep[(size_t)t * H + h] = expf(gf + m_prev - m_t);
        write[(size_t)t * H + h] = expf(gi - m_t);
        floor_[(size_t)t * H + h] = expf(-m_t);
      }
      m = __shfl_sync(0xffffffffu, m_t, 31);
    } else {
      const float tF = __shfl_sync(0xffffffffu, F, 31), tI = __shfl_sync(0xffffffffu, I, 31);
      Is = fmaxf(Is + tF, tI);
      Fs += tF;
    }
  }
  return EMIT ? make_float2(m, 0.f) : make_float2(Fs, Is);
}

// a warp per (request, head): steps of few tokens a request
__global__ void mlstm_gates_kernel(const float* __restrict__ raw, long long ld, float cap, float* __restrict__ m_state,
                                   const int* __restrict__ state_slots, const int* __restrict__ fresh,
                                   const int* __restrict__ cu_q, int num_requests, int H, float* __restrict__ keep,
                                   float* __restrict__ write, float* __restrict__ floor_) {
  pdl_trigger();
  pdl_wait();
  const int pair = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (pair >= num_requests * H) return;
  const int b = pair / H, h = pair % H;
  const int t0 = cu_q[b], t1 = cu_q[b + 1];
  if (t1 <= t0) return;
  float* ms = m_state + (size_t)state_slots[b] * H + h;
  const float m = mlstm_gates_walk<true>(raw, ld, cap, H, h, t0, t1, fresh[b] ? 0.f : *ms, keep, write, floor_).x;
  if ((threadIdx.x & 31) == 0) *ms = m;
}

// a block per (request, head): every warp takes a span of the request's tokens, finds the span's map, learns
// the maximum before its span from the maps of the spans before it, and walks its span again to write
__global__ void mlstm_gates_spans_kernel(const float* __restrict__ raw, long long ld, float cap, float* __restrict__ m_state,
                                         const int* __restrict__ state_slots, const int* __restrict__ fresh,
                                         const int* __restrict__ cu_q, int H, float* __restrict__ keep,
                                         float* __restrict__ write, float* __restrict__ floor_) {
  __shared__ float span_f[32], span_i[32];
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  const int b = blockIdx.x / H, h = blockIdx.x % H;
  const int t0 = cu_q[b], t1 = cu_q[b + 1];
  if (t1 <= t0) return;
  float* ms = m_state + (size_t)state_slots[b] * H + h;
  const float m0 = fresh[b] ? 0.f : *ms;
  const int span = (((t1 - t0) + warps - 1) / warps + 31) / 32 * 32;
  const int a = min(t1, t0 + warp * span), e = min(t1, a + span);
  const float2 map = mlstm_gates_walk<false>(raw, ld, cap, H, h, a, e, 0.f, keep, write, floor_);
  if (lane == 0) {
    span_f[warp] = map.x;
    span_i[warp] = map.y;
  }
  __syncthreads();          // (also: every thread has read the old maximum before thread 0 writes the new one)
  float m = m0;
  for (int w = 0; w < warp; ++w) m = fmaxf(span_f[w] + m, span_i[w]);
  mlstm_gates_walk<true>(raw, ld, cap, H, h, a, e, m, keep, write, floor_);
  if (threadIdx.x == 0) {
    float last = m0;
    for (int w = 0; w < warps; ++w) last = fmaxf(span_f[w] + last, span_i[w]);
    *ms = last;
  }
}

// ------------------------------------------------------------------ what follows the scan of a matrix memory
// raw [T, H, wide] 32-bit: columns [0, vdim) the numerator S^T q, column vdim the product n . q
__global__ void mlstm_finish_kernel(const float* __restrict__ raw, int wide, const float* __restrict__ floor_,
                                    VecParam weight, Rows gate, float eps, RowsOut out, int H, int vdim, int num_tokens) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long pair = blockIdx.x * (long long)(blockDim.x >> 5) + (threadIdx.x >> 5);
  if (pair >= (long long)num_tokens * H) return;
  const size_t t = pair / H;
  const int h = (int)(pair % H);
  const float* o = raw + (t * H + h) * wide;
  const float den = fmaxf(fabsf(o[vdim]), floor_[t * H + h]) + 1e-6f;
  const float inv = 1.f / den;
  float acc = 0.f;
  for (int i = lane; i < vdim; i += 32) {
    const float v = o[i] * inv;
    acc = fmaf(v, v, acc);
  }
  const float rstd = rsqrtf(warp_sum(acc) / (float)vdim + eps);
  for (int i = lane; i < vdim; i += 32) {
    const int col = h * vdim + i;
    float y = o[i] * inv * rstd * weight[col];
    if (gate.ptr) y *= sigmoid_f(gate.at(t, col));
    out.put(t, col, y);
  }
}

// raw [T, H vdim] 32-bit y of the scan; x the scan's values; z the gate; a block per (token, norm group)
__global__ void ssm_finish_kernel(const float* __restrict__ raw, Rows x, VecParam skip, Rows z, VecParam weight, int groups,
                                  float eps, RowsOut out, int H, int vdim) {
  __shared__ float scratch[33];
  pdl_trigger();
  pdl_wait();
  const size_t t = blockIdx.x;
  const int n = H * vdim, per = n / groups, base = blockIdx.y * per;
  auto gated = [&](int i) {
    const int col = base + i;
    return (raw[t * n + col] + skip[col / vdim] * x.at(t, col)) * silu_f(z.at(t, col));
  };
  float held[ROW_HOLD], acc = 0.f;
#pragma unroll
  for (int j = 0; j < ROW_HOLD; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    held[j] = i < per ? gated(i) : 0.f;
    acc = fmaf(held[j], held[j], acc);
  }
  for (int i = threadIdx.x + ROW_HOLD * blockDim.x; i < per; i += blockDim.x) {
    const float y = gated(i);
    acc = fmaf(y, y, acc);
  }
  const float rstd = rsqrtf(block_sum(acc, scratch) / (float)per + eps);
#pragma unroll
  for (int j = 0; j < ROW_HOLD; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i < per) out.put(t, base + i, held[j] * rstd * weight[base + i]);
  }
  for (int i = threadIdx.x + ROW_HOLD * blockDim.x; i < per; i += blockDim.x)
    out.put(t, base + i, gated(i) * rstd * weight[base + i]);
}

}  // namespace

TS_EXPORT int ts_add_position_rows(float* residual, const void* table, int table_is_f32, const int* positions,
                                   int num_positions, int num_tokens, int n, cudaStream_t stream) {
  TS_REQUIRE(num_tokens > 0 && n > 0 && residual && table && positions, "add_position_rows: empty input");
  TS_LAUNCH("add_position_rows", add_position_rows_kernel, num_tokens, n >= 1024 ? 256 : 128, 0, stream, residual,
            VecParam{table, table_is_f32}, positions, num_positions, n);
  return 0;
}

TS_EXPORT int ts_causal_conv_max_taps() { return CONV_MAX_TAPS; }

TS_EXPORT int ts_causal_conv(const void* x, long long ldx, int x_is_f32, void* y, long long ldy, int y_is_f32,
                             const void* w, int w_is_f32, const void* bias, int taps, float* state, const int* state_slots,
                             const int* fresh, const int* cu_q, int num_requests, int max_q_len, int C, int add_input,
                             int silu, cudaStream_t stream) {
  TS_REQUIRE(num_requests > 0 && max_q_len > 0 && C > 0, "causal_conv: empty input");
  TS_REQUIRE(taps >= 1 && taps <= CONV_MAX_TAPS, "causal_conv: 1 to %d taps, got %d", CONV_MAX_TAPS, taps);
  TS_REQUIRE(x && y && w && (taps == 1 || state) && state_slots && fresh && cu_q, "causal_conv: a null operand");
  ConvParams p{Rows{x, ldx, x_is_f32}, RowsOut{y, ldy, y_is_f32}, VecParam{w, w_is_f32}, VecParam{bias, w_is_f32},
               state, state_slots, fresh, cu_q, C, add_input, silu};
  const dim3 grid((C + CONV_THREADS - 1) / CONV_THREADS, (max_q_len + CONV_TILE - 1) / CONV_TILE, num_requests);
  TS_REQUIRE(grid.y <= 65535 && grid.z <= 65535, "causal_conv: the step is too large");
  switch (taps) {
#define TS_CONV_CASE(N) \
    case N: TS_LAUNCH("causal_conv", causal_conv_kernel<N>, grid, CONV_THREADS, 0, stream, p); break;
    TS_CONV_CASE(1) TS_CONV_CASE(2) TS_CONV_CASE(3) TS_CONV_CASE(4) TS_CONV_CASE(5) TS_CONV_CASE(6) TS_CONV_CASE(7)
    TS_CONV_CASE(8)
#undef TS_CONV_CASE
  }
  return 0;
}

// x [T, H dim | G dim | G vdim]; w [taps, channels] or null (taps 1); factor [H] or null; G 0: queries only
TS_EXPORT int ts_conv_heads_kvwrite(int is_f32, const void* x, long long ldx, const void* w, int w_is_f32, int taps,
                                    const void* factor, int factor_is_f32, float* state, const int* state_slots,
                                    const int* fresh, const int* cu_q, int num_requests, int max_q_len, int H, int G, int dim,
                                    int vdim, int stored, void* q_out, void* k_cache, void* v_cache, const int* slot_mapping,
                                    int page_size, cudaStream_t stream) {
  TS_REQUIRE(num_requests > 0 && max_q_len > 0 && H > 0 && G >= 0 && dim > 0 && vdim > 0 && stored >= dim && stored >= vdim,
             "conv_heads_kvwrite: sizes do not fit");
  TS_REQUIRE(taps >= 1 && taps <= CONV_MAX_TAPS && (w || taps == 1), "conv_heads_kvwrite: 1 to %d taps, got %d", CONV_MAX_TAPS, taps);
  TS_REQUIRE(x && q_out && (taps == 1 || state) && state_slots && fresh && cu_q, "conv_heads_kvwrite: a null operand");
  TS_REQUIRE(G == 0 || (k_cache && v_cache && slot_mapping && page_size > 0), "conv_heads_kvwrite: no cache to write");
  ConvHeads p{x, ldx, VecParam{w, w_is_f32}, VecParam{factor, factor_is_f32}, state, state_slots, fresh, cu_q, H, G, dim, vdim, stored,
              page_size, -1, H * dim + G * (dim + vdim), q_out, k_cache, v_cache, slot_mapping};
  if (page_size > 0 && (page_size & (page_size - 1)) == 0)
    for (p.page_shift = 0; (1 << p.page_shift) < page_size;) ++p.page_shift;
  const bool even = dim % 2 == 0 && vdim % 2 == 0 && stored % 2 == 0 && ldx % 2 == 0 && ((uintptr_t)x | (uintptr_t)w) % 8 == 0;
  const int cols = (H + 2 * G) * stored / (even ? 2 : 1);
  const dim3 grid((cols + CONV_THREADS - 1) / CONV_THREADS, (max_q_len + HEADS_TILE - 1) / HEADS_TILE, num_requests);
  TS_REQUIRE(grid.y <= 65535 && grid.z <= 65535, "conv_heads_kvwrite: the step is too large");
  if (is_f32) return even ? launch_conv_heads<float, 2>(p, taps, grid, stream) : launch_conv_heads<float, 1>(p, taps, grid, stream);
  return even ? launch_conv_heads<__nv_bfloat16, 2>(p, taps, grid, stream) : launch_conv_heads<__nv_bfloat16, 1>(p, taps, grid, stream);
}

// rows null: every row of x [num_out, n]; else out[o] = norm(x[rows[o]])
TS_EXPORT int ts_group_norm(const void* x, long long ldx, int x_is_f32, const void* w, int w_is_f32, const int* rows,
                            int groups, int n, float eps, void* out, int out_is_f32, int num_out, cudaStream_t stream) {
  TS_REQUIRE(num_out > 0 && n > 0 && groups > 0 && groups <= 65535 && n % groups == 0, "group_norm: %d columns in %d groups", n, groups);
  TS_LAUNCH("group_norm", group_norm_kernel<false>, dim3(num_out, groups), row_threads(n / groups), 0, stream, Rows{x, ldx, x_is_f32},
            VecParam{w, w_is_f32}, rows, groups, n, eps, RowsOut{out, (long long)n, out_is_f32}, (float*)nullptr);
  return 0;
}

// residual [T, n] (float, in place) += norm(y)
TS_EXPORT int ts_group_norm_add(const void* y, long long ldy, int y_is_f32, const void* w, int w_is_f32, int groups, int n,
                                float eps, float* residual, int num_tokens, cudaStream_t stream) {
  TS_REQUIRE(num_tokens > 0 && n > 0 && groups > 0 && groups <= 65535 && n % groups == 0, "group_norm_add: %d columns in %d groups", n, groups);
  TS_LAUNCH("group_norm_add", group_norm_kernel<true>, dim3(num_tokens, groups), row_threads(n / groups), 0, stream, Rows{y, ldy, y_is_f32},
            VecParam{w, w_is_f32}, (const int*)nullptr, groups, n, eps, RowsOut{nullptr, 0, 0}, residual);
  return 0;
}

TS_EXPORT int ts_axpby(const void* x, const void* y, int in_is_f32, float a, float b, void* out, int out_is_f32,
                       long long count, cudaStream_t stream) {
  TS_REQUIRE(count > 0 && x && y && out, "axpby: empty input");
  const int blocks = (int)((count + 255) / 256 < 148 * 16 ? (count + 255) / 256 : 148 * 16);
  TS_LAUNCH("axpby", axpby_kernel, blocks, 256, 0, stream, Rows{x, 1, in_is_f32}, Rows{y, 1, in_is_f32}, a, b,
            RowsOut{out, 1, out_is_f32}, count);
  return 0;
}

TS_EXPORT int ts_gate_columns(const void* x, const void* gate, long long ldg, int is_f32, void* out, int H, int stored,
                              int vdim, int num_tokens, cudaStream_t stream) {
  TS_REQUIRE(num_tokens > 0 && H > 0 && vdim > 0 && stored >= vdim && x && gate && out, "gate_columns: operands do not fit");
  TS_LAUNCH("gate_columns", gate_columns_kernel, num_tokens, H * vdim >= 2048 ? 512 : (H * vdim >= 1024 ? 256 : 128), 0, stream,
            Rows{x, (long long)H * stored, is_f32}, Rows{gate, ldg, is_f32}, RowsOut{out, (long long)H * vdim, is_f32}, H, stored,
            vdim);
  return 0;
}

TS_EXPORT int ts_joint_norm_kvwrite(int is_f32, const void* q, long long ldq, const void* k, long long ldk, const void* v,
                                    long long ldv, const void* qw, const void* kw, int w_is_f32, float eps, int H, int G,
                                    int dim, int vdim, int stored, void* q_out, void* k_cache, void* v_cache,
                                    const int* slot_mapping, int page_size, int num_tokens, const float* cos, const float* sin,
                                    const int* positions, int rot, int interleaved, cudaStream_t stream) {
  TS_REQUIRE(num_tokens > 0 && H > 0 && G > 0 && dim > 0 && vdim > 0 && stored >= dim && stored >= vdim,
             "joint_norm_kvwrite: sizes do not fit");
  TS_REQUIRE((qw == nullptr) == (kw == nullptr), "joint_norm_kvwrite: q and k are normed together or not at all");
  TS_REQUIRE(slot_mapping == nullptr || (k_cache && v_cache && page_size > 0), "joint_norm_kvwrite: no cache to write");
  TS_REQUIRE(rot >= 0 && rot <= dim && rot % 2 == 0 && (rot == 0 || (cos && sin && positions)), "joint_norm_kvwrite: rotary size %d of %d", rot, dim);
  JointNorm p{Rows{q, ldq, is_f32}, Rows{k, ldk, is_f32}, Rows{v, ldv, is_f32}, VecParam{qw, w_is_f32},
              VecParam{kw, w_is_f32}, eps, H, G, dim, vdim, stored, page_size, q_out, k_cache, v_cache, slot_mapping, is_f32,
              cos, sin, positions, rot, interleaved};
  const int packs = (H + G) * (dim / 8);
  const uintptr_t all = (uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)qw | (uintptr_t)kw | (uintptr_t)q_out |
                        (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)cos | (uintptr_t)sin;
  if (qw && (interleaved || rot == 0) && ((dim | vdim | stored | rot) & 7) == 0 && ((ldq | ldk | ldv) & 7) == 0 && (all & 15) == 0 &&
      packs <= JOINT_PACKS * JOINT_THREADS) {
    const int threads = packs >= 512 ? 256 : (packs >= 128 ? 128 : (packs + 31) / 32 * 32);
    if (is_f32) TS_LAUNCH("joint_norm_kvwrite", joint_norm_kvwrite_vec_kernel<float>, num_tokens, threads, 0, stream, p);
    else TS_LAUNCH("joint_norm_kvwrite", joint_norm_kvwrite_vec_kernel<__nv_bfloat16>, num_tokens, threads, 0, stream, p);
    return 0;
  }
  TS_LAUNCH("joint_norm_kvwrite", joint_norm_kvwrite_kernel, num_tokens, H * dim >= 2048 ? 512 : (H * dim >= 512 ? 256 : 128), 0, stream, p);
  return 0;
}

TS_EXPORT int ts_mlstm_gates(const float* raw, long long ld, float cap, float* m_state, const int* state_slots,
                             const int* fresh, const int* cu_q, int num_requests, int max_q_len, int H, float* keep,
                             float* write, float* floor_, cudaStream_t stream) {
  TS_REQUIRE(num_requests > 0 && H > 0 && cap > 0.f, "mlstm_gates: empty input or a cap that is not positive");
  TS_REQUIRE(raw && m_state && state_slots && fresh && cu_q && keep && write && floor_, "mlstm_gates: a null operand");
  if (max_q_len >= 128) {
    const int warps = max_q_len >= 512 ? 16 : (max_q_len + 31) / 32;
    TS_LAUNCH("mlstm_gates", mlstm_gates_spans_kernel, num_requests * H, warps * 32, 0, stream, raw, ld, cap, m_state,
              state_slots, fresh, cu_q, H, keep, write, floor_);
    return 0;
  }
  const int warps = 4;
  TS_LAUNCH("mlstm_gates", mlstm_gates_kernel, (num_requests * H + warps - 1) / warps, warps * 32, 0, stream, raw, ld, cap,
            m_state, state_slots, fresh, cu_q, num_requests, H, keep, write, floor_);
  return 0;
}

TS_EXPORT int ts_mlstm_finish(const float* raw, int wide, const float* floor_, const void* weight, int w_is_f32,
                              const void* gate, long long ldg, int io_is_f32, float eps, void* out, int H, int vdim,
                              int num_tokens, cudaStream_t stream) {
  TS_REQUIRE(num_tokens > 0 && H > 0 && vdim > 0 && wide > vdim && raw && floor_ && weight && out,
             "mlstm_finish: operands do not fit");
  const int warps = 4;
  const long long pairs = (long long)num_tokens * H;
  TS_LAUNCH("mlstm_finish", mlstm_finish_kernel, (int)((pairs + warps - 1) / warps), warps * 32, 0, stream, raw, wide,
            floor_, VecParam{weight, w_is_f32}, Rows{gate, ldg, io_is_f32}, eps,
            RowsOut{out, (long long)H * vdim, io_is_f32}, H, vdim, num_tokens);
  return 0;
}

TS_EXPORT int ts_ssm_finish(const float* raw, const void* x, long long ldx, const void* skip, const void* z, long long ldz,
                            const void* weight, int w_is_f32, int io_is_f32, int groups, float eps, void* out, int H,
                            int vdim, int num_tokens, cudaStream_t stream) {
  TS_REQUIRE(num_tokens > 0 && H > 0 && vdim > 0 && groups > 0 && groups <= 65535 && (H * vdim) % groups == 0,
             "ssm_finish: %d columns in %d groups", H * vdim, groups);
  TS_REQUIRE(raw && x && skip && z && weight && out, "ssm_finish: a null operand");
  TS_LAUNCH("ssm_finish", ssm_finish_kernel, dim3(num_tokens, groups), row_threads(H * vdim / groups), 0, stream, raw, Rows{x, ldx, io_is_f32},
            VecParam{skip, w_is_f32}, Rows{z, ldz, io_is_f32}, VecParam{weight, w_is_f32}, groups, eps,
            RowsOut{out, (long long)H * vdim, io_is_f32}, H, vdim);
  return 0;
}
