// Mixers whose memory is one matrix per head: four recurrences over the tokens of a sequence on one
// kernel, what prepares their operands, and what finishes their outputs. Per head the state S is
// dim x vdim float32 numbers of a request (zero before its first token):
//
//   delta    S <- g S (g per key channel), then S <- S + k u^T with u = beta (v - S^T k), then o = S^T q; the last
//            two as o = (g S)^T q + (q . k) u, so that both sums over g S are formed together
//   bonus    o = (S + diag(u) k v^T)^T q, then S <- diag(w) S + k v^T, w = exp(-exp(z + z0))
//   memory   m' = max(f + m, i), S <- e^(f + m - m') S + e^(i - m') k v^T, the normaliser n alike with
//            k alone, o = S^T q (divided later by max(|n . q|, e^-m) + 1e-6)
//   space    S <- a S + k (t v)^T, o = S^T q + D v, with two numbers per token and head: the decay a and the step t
//
// The columns of S (one per value channel) do not meet inside a token, so a block walks the rows of one
// sequence of the step for one head and a few columns, from the state that the request's slot holds.
// LP lanes of a warp share two neighbouring columns (what a lane reads of a token then serves both); a
// lane holds V groups of four consecutive rows (group p + LP i). A sum over a column's rows is four chains
// per lane and a butterfly over the LP lanes, in an order given by dim alone. The tokens' operands are copied into shared memory a chunk ahead (cp.async, two buffers);
// the chunk is a staging unit only: every S and o is the same chain of operations wherever the step's
// rows begin and end, so a position's result does not depend on how its prompt was cut.
// Everything here is float32 in both precisions; only what enters the next product changes type.
#include "bw_act.cuh"
#include "bw_mma.cuh"

#include <math.h>

namespace {

constexpr int kThreads = 128;
constexpr int kWarps = kThreads / 32;
constexpr int kCols = 2;  // columns of a lane
enum { kDelta = 0, kBonus = 1, kMemory = 2, kSpace = 3 };

// The serving precision takes the hardware's exponential (relative error about 1e-7 times the exponent's size, far
// below that of the bfloat16 operands of the products before it).
__device__ __forceinline__ float exp_f(float x) {
#if BW_ACT_BF16
  return __expf(x);
#else
  return expf(x);
#endif
}
__device__ __forceinline__ float sigmoid_f(float z) { return __fdiv_rn(1.0f, __fadd_rn(1.0f, expf(-z))); }
// ln(1 + e^z) without overflow
__device__ __forceinline__ float softplus_f(float z) { return __fadd_rn(fmaxf(z, 0.0f), log1pf(expf(-fabsf(z)))); }

__device__ __forceinline__ void copy4_async(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(bw::smem_addr(dst)), "l"(src));
}
__device__ __forceinline__ void copy16_async(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(bw::smem_addr(dst)), "l"(src));
}

struct ScanArgs {
  const float* q;          // row r, head h / rep: q + r * q_stride + (h / rep) * dim
  const float* k;
  const float* v;          // row r, head h: v + r * v_stride + h * vdim
  int q_stride, k_stride, v_stride;
  int rep;                 // heads that share a q/k head
  const float* decay;      // delta: g; bonus: z. Row r, head h: decay + r * decay_stride + h * dim
  int decay_stride;
  const float* decay_bias;  // bonus: z0 [heads * dim]
  const float* bonus;      // bonus: u [heads * dim]; space: D [heads]
  const float* s0;         // delta: beta; memory: the forget gate's projection; space: a. Row r, head h: s0 + r * s_stride + h
  const float* s1;         // delta: q . k, one per query head (h / rep); memory: the input gate's projection; space: t; one per head
  int s_stride;
  const float* s0_bias;    // memory: [heads]
  const float* s1_bias;
  float cap;               // memory: gates are cap * tanh(. / cap)
  float* state;            // [slots, heads, columns, column]: delta, bonus, space: vdim columns of dim; memory: vdim + 1
                           // columns of dim + 4 (the last column is n; entry dim of every column is m)
  float* o;                // [n, heads * vdim]
  float* aux;              // memory: [n, heads, 2]: n . q and m
  const int* tile_seq;
  const int* tile_row0;
  const int* tile_rows;
  const int* seq_pos0;
  const int* seq_slot;
  int heads, dim, vdim, chunk, wide;
};

// Sums x[0 .. G - 1] over the LP lanes of a column at once: afterwards lane p holds the sum of x[p / (LP / G)]. Each
// sum is the butterfly over lane distances LP / 2, LP / 4, .. 1 (a + b and b + a are the same bits), as below.
template <int LP, int G>
__device__ __forceinline__ float group_sum(float (&x)[G], int p) {
  int off = LP / 2;
#pragma unroll
  for (int n = G; n > 1; n /= 2) {
    const bool up = (p & off) != 0;
#pragma unroll
    for (int i = 0; i < n / 2; ++i) {
      const float send = up ? x[i] : x[i + n / 2], keep = up ? x[i + n / 2] : x[i];
      x[i] = __fadd_rn(keep, __shfl_xor_sync(0xffffffffu, send, off));
    }
    off /= 2;
  }
#pragma unroll
  for (; off > 0; off /= 2) x[0] = __fadd_rn(x[0], __shfl_xor_sync(0xffffffffu, x[0], off));
  return x[0];
}
template <int LP>
__device__ __forceinline__ float column_sum(float x) {
#pragma unroll
  for (int off = LP / 2; off > 0; off /= 2) x = __fadd_rn(x, __shfl_xor_sync(0xffffffffu, x, off));
  return x;
}

template <int MODE, int LP, int V>
struct Shape {
  static constexpr int CB = kThreads / LP * kCols;  // columns of a block
  static constexpr int DP = LP * 4 * V;      // rows held; those from dim on are zero
  static constexpr int VECS = MODE == kMemory || MODE == kSpace ? 2 : 3;
  static constexpr int SC = VECS * DP + CB;  // where a token's scalars start
  static constexpr int W = SC + 4;           // a staged token: k | q | decay | values | scalars
  static constexpr int G = LP < 8 ? LP : 8;  // tokens whose outputs are summed together
};

template <int V>
struct Rows {
  float v[4 * V];
};
template <int LP, int V>
__device__ __forceinline__ Rows<V> load_rows(const float* at, int p) {
  Rows<V> r;
#pragma unroll
  for (int i = 0; i < V; ++i) {
    const float4 f = *reinterpret_cast<const float4*>(at + 4 * (p + LP * i));
    r.v[4 * i] = f.x, r.v[4 * i + 1] = f.y, r.v[4 * i + 2] = f.z, r.v[4 * i + 3] = f.w;
  }
  return r;
}
// Four chains (the entries of equal place in the groups of four) and their sum.
template <int V>
__device__ __forceinline__ float dot(const Rows<V>& a, const Rows<V>& b) {
  float s[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) s[e] = __fmul_rn(a.v[e], b.v[e]);
#pragma unroll
  for (int i = 4; i < 4 * V; ++i) s[i & 3] = __fmaf_rn(a.v[i], b.v[i], s[i & 3]);
  return __fadd_rn(__fadd_rn(s[0], s[1]), __fadd_rn(s[2], s[3]));
}
// What a lane reads of a staged token.
template <int V>
struct Token {
  Rows<V> k, q, d;
  float v[kCols];
  float s0, s1;
};

template <int MODE, int LP, int V>
__global__ void __launch_bounds__(kThreads) state_scan_kernel(const ScanArgs a) {
  typedef Shape<MODE, LP, V> T;
  const bool few = gridDim.x * gridDim.y * gridDim.z <= 296;
  if (few) bw::pdl_launch();
  extern __shared__ __align__(16) float sm[];
  const int dim = a.dim, vdim = a.vdim, chunk = a.chunk;
  float* stage = sm;                            // [2][chunk][W]
  float* outs = sm + 2 * chunk * T::W;          // [chunk][CB]
  const int t = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * T::CB;
  const int seq = a.tile_seq[t], row0 = a.tile_row0[t], cnt = a.tile_rows[t];
  const int tid = threadIdx.x;
  const int p = tid & (LP - 1), col = tid / LP * kCols;  // this lane's rows and its first column in the block
  constexpr bool kMem = MODE == kMemory, kRowScalars = kMem || MODE == kSpace;
  const int cols = kMem ? vdim + 1 : vdim, col_size = kMem ? dim + 4 : dim;
  float* head_state = a.state + (static_cast<size_t>(a.seq_slot[seq]) * a.heads + h) * cols * col_size;
  float* sp = head_state + static_cast<size_t>(c0 + col) * col_size;
  const bool fresh = a.seq_pos0[seq] == 0;      // a slot is handed out as its last holder left it
  // The state of this run was written by the step before, so it is asked for before the wait for this step's kernels.
  Rows<V> S[kCols];
#pragma unroll
  for (int j = 0; j < kCols; ++j) {
    const float* from = sp + j * col_size;
#pragma unroll
    for (int i = 0; i < V; ++i) {
      const int row = 4 * (p + LP * i);
      float4 f = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      if (!fresh && c0 + col + j < cols) {
        if (a.wide) {
          if (row < dim) f = *reinterpret_cast<const float4*>(from + row);
        } else {
          if (row < dim) f.x = from[row];
          if (row + 1 < dim) f.y = from[row + 1];
          if (row + 2 < dim) f.z = from[row + 2];
          if (row + 3 < dim) f.w = from[row + 3];
        }
      }
      S[j].v[4 * i] = f.x, S[j].v[4 * i + 1] = f.y, S[j].v[4 * i + 2] = f.z, S[j].v[4 * i + 3] = f.w;
    }
  }
  float m = 0.0f;  // memory: the running maximum (held by every thread of warp 0)
  if (kMem && !fresh) m = head_state[static_cast<size_t>(c0) * col_size + dim];
  Rows<V> bonus;
  if (MODE == kBonus) {
#pragma unroll
    for (int i = 0; i < V; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int row = 4 * (p + LP * i) + e;
        bonus.v[4 * i + e] = row < dim ? a.bonus[h * dim + row] : 0.0f;
      }
  }
  if (dim < T::DP)  // rows from dim on stay zero
    for (int i = tid; i < 2 * chunk * T::W; i += kThreads) stage[i] = 0.0f;
  bw::pdl_wait();
  if (!few) bw::pdl_launch();
  __syncthreads();
  const int kh = h / a.rep;
  const int warp = tid >> 5, lane = tid & 31;
  // where entry e of a staged token's vectors and values comes from: its address in row 0 and the distance between rows
  auto source = [&](int e, int& stride) -> const float* {
    if (e < T::VECS * T::DP) {
      const int d = e % T::DP;
      if (d >= dim) return nullptr;
      if (e < T::DP) return stride = a.k_stride, a.k + kh * dim + d;
      if (e < 2 * T::DP) return stride = a.q_stride, a.q + kh * dim + d;
      return stride = a.decay_stride, a.decay + h * dim + d;
    }
    const int cc = c0 + e - T::VECS * T::DP;
    if (e >= T::SC || cc >= vdim) return nullptr;
    return stride = a.v_stride, a.v + h * vdim + cc;
  };
  // A warp copies every fourth token, a lane the same 16-byte pieces of each: addresses only move on by rows.
  constexpr int NP = (T::SC / 4 + 31) / 32;
  const float* piece[NP];
  int step[NP];
  if (a.wide) {
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      step[i] = 0;
      piece[i] = source(4 * (lane + 32 * i), step[i]);
      if (piece[i]) piece[i] += static_cast<size_t>(row0 + warp) * step[i];
      step[i] *= kWarps;
    }
  }
  auto request = [&](int first, float* buf) {
    const int len = min(chunk, cnt - first);
    if (a.wide) {
      for (int tt = warp; tt < len; tt += kWarps) {
        float* dst = buf + tt * T::W + 4 * lane;
#pragma unroll
        for (int i = 0; i < NP; ++i)
          if (piece[i]) copy16_async(dst + 128 * i, piece[i]), piece[i] += step[i];
      }
    } else {
      for (int i = tid; i < len * T::SC; i += kThreads) {
        const int tt = i / T::SC, e = i - tt * T::SC;
        int stride = 0;
        const float* src = source(e, stride);
        if (src) copy4_async(buf + tt * T::W + e, src + static_cast<size_t>(row0 + first + tt) * stride);
      }
    }
    if (MODE != kBonus) {
      for (int tt = tid; tt < len; tt += kThreads) {
        const size_t r = static_cast<size_t>(row0 + first + tt);
        copy4_async(buf + tt * T::W + T::SC, a.s0 + r * a.s_stride + h);
        copy4_async(buf + tt * T::W + T::SC + 1, a.s1 + r * a.s_stride + (kRowScalars ? h : kh));
      }
    }
    bw::copies_commit();
  };
  auto load = [&](const float* tok) -> Token<V> {
    Token<V> x;
    x.k = load_rows<LP, V>(tok, p), x.q = load_rows<LP, V>(tok + T::DP, p);
    if (!kRowScalars) x.d = load_rows<LP, V>(tok + 2 * T::DP, p);
#pragma unroll
    for (int j = 0; j < kCols; ++j) x.v[j] = tok[T::VECS * T::DP + col + j];
    x.s0 = MODE == kBonus ? 0.0f : tok[T::SC], x.s1 = MODE == kBonus ? 0.0f : tok[T::SC + 1];
    return x;
  };
  // One token: S moves on; this lane's share of both columns' outputs into o (delta: one column's whole output, see below).
  auto move = [&](const Token<V>& x, float (&o)[kCols]) {
    if (MODE == kDelta) {
      // All four sums (of k and of q, both columns) in one butterfly: lane p ends up with the sum p / (LP / 4).
      float d[2 * kCols];
#pragma unroll
      for (int j = 0; j < kCols; ++j) {
#pragma unroll
        for (int i = 0; i < 4 * V; ++i) S[j].v[i] = __fmul_rn(x.d.v[i], S[j].v[i]);
        d[j] = dot<V>(x.k, S[j]);
        d[kCols + j] = dot<V>(x.q, S[j]);
      }
      const float sum = group_sum<LP, 2 * kCols>(d, p);
      const float mine = __fmul_rn(x.s0, __fsub_rn((p & (LP / 4)) ? x.v[1] : x.v[0], sum));
      const int base = lane & ~(LP - 1);
      float u[kCols];
#pragma unroll
      for (int j = 0; j < kCols; ++j) u[j] = __shfl_sync(0xffffffffu, mine, base + j * (LP / 4));
#pragma unroll
      for (int j = 0; j < kCols; ++j) {
#pragma unroll
        for (int i = 0; i < 4 * V; ++i) S[j].v[i] = __fmaf_rn(x.k.v[i], u[j], S[j].v[i]);
      }
      o[0] = __fmaf_rn(x.s1, (p & (LP / 4)) ? u[1] : u[0], sum);  // in the lanes of q's sums: a column's output
    } else {
#pragma unroll
      for (int j = 0; j < kCols; ++j) {
        if (MODE == kBonus) {
          Rows<V> seen;
#pragma unroll
          for (int i = 0; i < 4 * V; ++i) {
            const float kv = __fmul_rn(x.k.v[i], x.v[j]);
            seen.v[i] = __fmaf_rn(bonus.v[i], kv, S[j].v[i]);
            S[j].v[i] = __fmaf_rn(x.d.v[i], S[j].v[i], kv);
          }
          o[j] = dot<V>(x.q, seen);
        } else {
          const float add = __fmul_rn(x.s1, kMem && c0 + col + j == vdim ? 1.0f : x.v[j]);  // (the normaliser's column takes ones)
#pragma unroll
          for (int i = 0; i < 4 * V; ++i) S[j].v[i] = __fmaf_rn(x.k.v[i], add, __fmul_rn(x.s0, S[j].v[i]));
          o[j] = dot<V>(x.q, S[j]);
        }
      }
    }
  };
  request(0, stage);
  for (int first = 0, b = 0; first < cnt; first += chunk, b ^= 1) {
    const int len = min(chunk, cnt - first);
    float* buf = stage + b * chunk * T::W;
    if (first) __syncthreads();  // the other buffer and `outs` have been used
    if (first + chunk < cnt) {
      request(first + chunk, stage + (b ^ 1) * chunk * T::W);
      bw::copies_wait<1>();
    } else {
      bw::copies_wait<0>();
    }
    __syncthreads();
    if (MODE == kBonus) {
      constexpr int kTokens = T::DP < kThreads ? kThreads / T::DP : 1;  // tokens that the block's threads cover at a time
      for (int d = tid % T::DP; d < dim; d += kThreads) {
        const float bias = a.decay_bias[h * dim + d];
        float* at = buf + tid / T::DP * T::W + 2 * T::DP + d;
        for (int tt = tid / T::DP; tt < len; tt += kTokens, at += kTokens * T::W)
          *at = exp_f(-exp_f(__fadd_rn(*at, bias)));
      }
      __syncthreads();
    }
    if (kMem) {
      if (tid < 32) {
        // lane l forms the gates of tokens l, l + 32, ..; the maxima follow one after the other
        const float bf = a.s0_bias[h], bi = a.s1_bias[h];
        for (int t0 = 0; t0 < len; t0 += 32) {
          float f = 0.0f, g = 0.0f;
          float* sc = buf + (t0 + tid) * T::W + T::SC;
          if (t0 + tid < len) {
            // ln(sigmoid(y)) = -softplus(-y)
            f = -softplus_f(-__fmul_rn(a.cap, tanhf(__fdiv_rn(__fadd_rn(sc[0], bf), a.cap))));
            g = __fmul_rn(a.cap, tanhf(__fdiv_rn(__fadd_rn(sc[1], bi), a.cap)));
          }
          float mine = 0.0f, before = 0.0f;
          const int end = min(32, len - t0);
          for (int l = 0; l < end; ++l) {
            const float fm = __fadd_rn(__shfl_sync(0xffffffffu, f, l), m);
            m = fmaxf(fm, __shfl_sync(0xffffffffu, g, l));
            if (tid == l) mine = m, before = fm;
          }
          if (t0 + tid < len) {
            sc[0] = exp_f(__fsub_rn(before, mine));
            sc[1] = exp_f(__fsub_rn(g, mine));
            sc[2] = mine;
          }
        }
      }
      __syncthreads();
    }
    int tt = 0;
    if (MODE == kDelta) {
      // lane p = LP / 2 holds the first column's output, lane p = LP / 2 + LP / 4 the second's
      float* to = outs + col + ((p & (LP / 4)) ? 1 : 0);
      const bool stores = p == LP / 2 || p == LP / 2 + LP / 4;
      Token<V> x = load(buf);
#pragma unroll 4
      for (; tt < len; ++tt) {  // the next token's operands are asked for before this one's are used
        const Token<V> y = load(buf + min(tt + 1, len - 1) * T::W);
        float o[kCols];
        move(x, o);
        if (stores) to[tt * T::CB] = o[0];
        x = y;
      }
    }
    for (; tt + T::G <= len; tt += T::G) {
      float part[kCols][T::G];
      const float* tok = buf + tt * T::W;
      Token<V> x = load(tok);
#pragma unroll
      for (int i = 0; i < T::G; ++i) {  // the next token's operands are asked for before this one's are used
        const Token<V> y = load(tok + min(i + 1, T::G - 1) * T::W);
        float o[kCols];
        move(x, o);
#pragma unroll
        for (int j = 0; j < kCols; ++j) part[j][i] = o[j];
        x = y;
      }
#pragma unroll
      for (int j = 0; j < kCols; ++j) {
        const float s = group_sum<LP, T::G>(part[j], p);
        if (p % (LP / T::G) == 0) outs[(tt + p / (LP / T::G)) * T::CB + col + j] = s;
      }
    }
    for (; tt < len; ++tt) {
      float o[kCols];
      move(load(buf + tt * T::W), o);
#pragma unroll
      for (int j = 0; j < kCols; ++j) {
        const float s = column_sum<LP>(o[j]);
        if (p == 0) outs[tt * T::CB + col + j] = s;
      }
    }
    __syncthreads();
    const int cc = c0 + tid % T::CB;
    const float skip = MODE == kSpace ? a.bonus[h] : 0.0f;
    for (int i = tid; i < len * T::CB; i += kThreads) {
      const int ti = i / T::CB;
      const size_t r = static_cast<size_t>(row0 + first + ti);
      if (cc < vdim) {
        const float o = outs[i];
        a.o[r * a.heads * vdim + h * vdim + cc] =
            MODE == kSpace ? __fmaf_rn(skip, buf[ti * T::W + T::VECS * T::DP + tid % T::CB], o) : o;
      } else if (kMem && cc == vdim) {
        float* x = a.aux + (r * a.heads + h) * 2;
        x[0] = outs[i], x[1] = buf[ti * T::W + T::SC + 2];
      }
    }
  }
#pragma unroll
  for (int j = 0; j < kCols; ++j) {
    if (c0 + col + j >= cols) continue;
    float* to = sp + j * col_size;
#pragma unroll
    for (int i = 0; i < V; ++i) {
      const int row = 4 * (p + LP * i);
      if (a.wide) {
        if (row < dim)
          *reinterpret_cast<float4*>(to + row) = make_float4(S[j].v[4 * i], S[j].v[4 * i + 1], S[j].v[4 * i + 2], S[j].v[4 * i + 3]);
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (row + e < dim) to[row + e] = S[j].v[4 * i + e];
      }
    }
    // every column keeps the maximum of its own: the blocks of a head do not read what another one writes
    if (kMem && p == 0) {
      const int last = (cnt - 1) / chunk, slot = (cnt - 1) - last * chunk;
      to[dim] = stage[(last & 1) * chunk * T::W + slot * T::W + T::SC + 2];
    }
  }
}

// out[r, h] = y / sqrt(mean(y^2) + eps) * w * gate(g) for every head, y the recurrence's output; with `aux` y is first
// divided: y <- s y / (max(|s n.q|, e^-m) + 1e-6), s the queries' scale. A warp per row and head.
struct FinishArgs {
  const float* o;
  const float* aux;    // [n, heads, 2] or null
  float q_scale;
  const float* w;      // [vdim] (w_stride 0) or [heads * vdim] (w_stride vdim)
  int w_stride;
  const float* gate;   // row r, head h: gate + r * gate_stride + h * vdim
  int gate_stride;
  int gate_silu;       // 0: sigmoid(g); 1: g sigmoid(g)
  float eps;
  act_t* out;
  int heads, vdim;
};

__global__ void __launch_bounds__(kThreads) scan_finish_kernel(const FinishArgs a) {
  bw::pdl_enter();
  const size_t r = blockIdx.x;
  const int h = blockIdx.y * (kThreads / 32) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= a.heads) return;
  const float* o = a.o + (r * a.heads + h) * a.vdim;
  const float* g = a.gate + r * a.gate_stride + h * a.vdim;
  const float* w = a.w + static_cast<size_t>(h) * a.w_stride;
  act_t* out = a.out + (r * a.heads + h) * a.vdim;
  float f = 1.0f;
  if (a.aux) {
    const float nq = a.aux[(r * a.heads + h) * 2], m = a.aux[(r * a.heads + h) * 2 + 1];
    const float den = __fadd_rn(fmaxf(fabsf(__fmul_rn(nq, a.q_scale)), expf(-m)), 1e-6f);
    f = __fdiv_rn(a.q_scale, den);
  }
  constexpr int kKeep = 8;  // entries of a lane that stay in registers (vdim up to 256)
  float y[kKeep];
  float ss = 0.0f;
#pragma unroll
  for (int j = 0; j < kKeep; ++j) {
    const int d = lane + 32 * j;
    y[j] = d < a.vdim ? __fmul_rn(o[d], f) : 0.0f;
    ss = __fmaf_rn(y[j], y[j], ss);
  }
  for (int d = lane + 32 * kKeep; d < a.vdim; d += 32) {
    const float v = __fmul_rn(o[d], f);
    ss = __fmaf_rn(v, v, ss);
  }
  const float inv = bw::rms_scale(bw::warp_sum(ss), a.vdim, a.eps);
  auto finish = [&](int d, float v) {
    const float z = g[d];
    const float s = sigmoid_f(z);
    out[d] = bw::from_f<act_t>(__fmul_rn(bw::rms_apply(v, inv, w[d]), a.gate_silu ? __fmul_rn(z, s) : s));
  };
#pragma unroll
  for (int j = 0; j < kKeep; ++j) {
    const int d = lane + 32 * j;
    if (d < a.vdim) finish(d, y[j]);
  }
  for (int d = lane + 32 * kKeep; d < a.vdim; d += 32) finish(d, __fmul_rn(o[d], f));
}

// ---------------------------------------------------------------------------------------
// What the delta recurrence reads, row by row. q, k and v pass a causal convolution over time on
// every channel (inputs before the step's first row of a sequence from the request's state, zeros before position 0)
// and SiLU; q and k become unit vectors, q times a scale; the decays g = exp(-exp(A_h) softplus(z + bias)) replace z;
// beta = sigmoid(b); q . k per query head. With `keep` (steps of one row per sequence) the state is brought up to date here as well.
struct DeltaPrepArgs {
  const float* u;         // [n, u_stride]: q heads | k heads | v heads, beta's projections from beta_col on
  int u_stride, beta_col;
  const float* conv_t;    // [taps, channels]
  int taps;
  float* conv_state;      // [slots, taps - 1, channels] or null
  int keep;
  float* z;               // [n, z_stride]: heads * dim columns
  int z_stride;
  const float* dt_bias;   // [heads * dim]
  const float* a_log;     // [heads]
  float* out;             // [n, out_stride]: q | k | v | beta | q . k (one per query head)
  int out_stride;
  const int* pos;
  const int* row_seq;
  const int* seq_row0;
  const int* seq_slot;
  int heads, kv_heads, dim, vdim;
  float q_scale;
};

constexpr int kMaxPer = 16;  // entries of a head per lane: sizes up to 512

template <int VEC>
struct VecOf {
  typedef float4 type;
};
template <>
struct VecOf<1> {
  typedef float type;
};

// The convolution over time and SiLU of one head (`size` channels from col0 on) into the lane's registers: with VEC 4 four
// neighbouring channels at a time (128 to a warp), else channels 32 apart. The order of a channel's sum is the taps', either way.
template <int VEC>
__device__ __forceinline__ void conv_head(const DeltaPrepArgs& a, int r, int p, int row0, float* st, int channels, int lane, int col0,
                                          int size, float (&val)[kMaxPer]) {
  constexpr int NG = kMaxPer / VEC, kTapBatch = 4;  // taps whose inputs are asked for together
  typedef typename VecOf<VEC>::type vec_t;
#pragma unroll
  for (int j = 0; j < kMaxPer; ++j) val[j] = 0.0f;
  const float* u = a.u + static_cast<size_t>(r) * a.u_stride + col0;
  const bool keep = a.keep && st;
#pragma unroll
  for (int g = 0; g < NG; ++g) {
    const int e = VEC * (lane + 32 * g);
    if (e >= size) continue;
    for (int t0 = 0; t0 < a.taps; t0 += kTapBatch) {  // taps ascending
      vec_t x[kTapBatch], w[kTapBatch];
#pragma unroll
      for (int i = 0; i < kTapBatch; ++i) {
        const int t = t0 + i, back = a.taps - 1 - t;
        x[i] = vec_t{}, w[i] = vec_t{};
        if (t >= a.taps || p - back < 0) continue;
        const float* src = r - back >= row0 ? u - static_cast<ptrdiff_t>(back) * a.u_stride
                                            : st + static_cast<size_t>(a.taps - 1 - (row0 - (r - back))) * channels + col0;
        x[i] = *reinterpret_cast<const vec_t*>(src + e);
        w[i] = *reinterpret_cast<const vec_t*>(a.conv_t + static_cast<size_t>(t) * channels + col0 + e);
      }
#pragma unroll
      for (int i = 0; i < kTapBatch; ++i) {  // (a tap before the sequence's start adds 0 * 0)
        const float* xf = reinterpret_cast<const float*>(&x[i]);
        const float* wf = reinterpret_cast<const float*>(&w[i]);
#pragma unroll
        for (int c = 0; c < VEC; ++c) val[VEC * g + c] = __fmaf_rn(wf[c], xf[c], val[VEC * g + c]);
        // the sequence's only row: the inputs move up by one (row t - 1 of the state was read as tap t - 1)
        if (keep && t0 + i >= 1 && t0 + i < a.taps)
          *reinterpret_cast<vec_t*>(st + static_cast<size_t>(t0 + i - 1) * channels + col0 + e) = x[i];
      }
    }
  }
#pragma unroll
  for (int j = 0; j < kMaxPer; ++j) val[j] = __fmul_rn(val[j], sigmoid_f(val[j]));
}

template <int VEC>
__device__ __forceinline__ void store_head(float* out, int lane, int size, const float (&val)[kMaxPer], float f) {
#pragma unroll
  for (int g = 0; g < kMaxPer / VEC; ++g) {
    const int e = VEC * (lane + 32 * g);
    if (e >= size) continue;
    if (VEC == 4)
      *reinterpret_cast<float4*>(out + e) = make_float4(__fmul_rn(val[4 * g], f), __fmul_rn(val[4 * g + 1], f),
                                                        __fmul_rn(val[4 * g + 2], f), __fmul_rn(val[4 * g + 3], f));
    else
      out[e] = __fmul_rn(val[g], f);
  }
}

// A warp per query/key head (both), value head, head of decays; the last one forms beta.
template <int VEC>
__global__ void __launch_bounds__(kThreads) delta_prepare_kernel(const DeltaPrepArgs a) {
  bw::pdl_enter();
  const int r = blockIdx.x;
  const int lane = threadIdx.x & 31;
  int unit = blockIdx.y * kWarps + (threadIdx.x >> 5);
  const int G = a.kv_heads, channels = 2 * G * a.dim + a.heads * a.vdim;
  float* out = a.out + static_cast<size_t>(r) * a.out_stride;
  if (unit < G + a.heads) {
    const int p = a.pos[r], seq = a.row_seq[r], row0 = a.seq_row0[seq];
    float* st = a.conv_state ? a.conv_state + static_cast<size_t>(a.seq_slot[seq]) * (a.taps - 1) * channels : nullptr;
    float val[kMaxPer];
    if (unit >= G) {
      const int col0 = 2 * G * a.dim + (unit - G) * a.vdim;
      conv_head<VEC>(a, r, p, row0, st, channels, lane, col0, a.vdim, val);
      store_head<VEC>(out + col0, lane, a.vdim, val, 1.0f);
      return;
    }
    float other[kMaxPer];
    conv_head<VEC>(a, r, p, row0, st, channels, lane, unit * a.dim, a.dim, val);
    conv_head<VEC>(a, r, p, row0, st, channels, lane, (G + unit) * a.dim, a.dim, other);
    float qq = 0.0f, kk = 0.0f;  // (entries beyond the head are zero)
#pragma unroll
    for (int j = 0; j < kMaxPer; ++j) qq = __fmaf_rn(val[j], val[j], qq), kk = __fmaf_rn(other[j], other[j], kk);
    const float fq = __fmul_rn(__fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(bw::warp_sum(qq), 1e-6f))), a.q_scale);
    const float fk = __fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(bw::warp_sum(kk), 1e-6f)));
    float qk = 0.0f;
#pragma unroll
    for (int j = 0; j < kMaxPer; ++j) qk = __fmaf_rn(__fmul_rn(val[j], fq), __fmul_rn(other[j], fk), qk);
    qk = bw::warp_sum(qk);
    store_head<VEC>(out + unit * a.dim, lane, a.dim, val, fq);
    store_head<VEC>(out + (G + unit) * a.dim, lane, a.dim, other, fk);
    if (lane == 0) out[channels + a.heads + unit] = qk;
    return;
  }
  unit -= G + a.heads;
  if (unit < a.heads) {
    const float rate = expf(a.a_log[unit]);
    float* z = a.z + static_cast<size_t>(r) * a.z_stride + unit * a.dim;
    const float* bias = a.dt_bias + unit * a.dim;
    for (int d = lane; d < a.dim; d += 32) z[d] = exp_f(-__fmul_rn(rate, softplus_f(__fadd_rn(z[d], bias[d]))));
  } else if (unit == a.heads) {
    for (int h = lane; h < a.heads; h += 32) out[channels + h] = sigmoid_f(a.u[static_cast<size_t>(r) * a.u_stride + a.beta_col + h]);
  }
}

// What the state-space recurrence reads, row by row. The columns conv0 .. conv0 + channels - 1 of a projected row pass a causal
// convolution over time (a bias per channel; inputs before the step's first row of a sequence from the request's state, zeros
// before position 0) and SiLU; the columns step0 .. step0 + heads - 1 become steps t = ln(1 + e^(z + bias_h)) and decays
// e^(-rate_h t). With `keep` (steps of one row per sequence) the state is brought up to date here as well.
struct SpacePrepArgs {
  const float* u;         // [n, u_stride]
  int u_stride, conv0, channels, step0, heads;
  const float* conv_t;    // [taps, channels]
  const float* conv_b;    // [channels]
  int taps;
  float* conv_state;      // [slots, taps - 1, channels] or null
  int keep;
  const float* dt_bias;   // [heads]
  const float* rate;      // [heads]
  float* out;             // [n, out_stride]: the channels, from out_step on the heads' steps, then their decays
  int out_stride, out_step;
  const int* pos;
  const int* row_seq;
  const int* seq_row0;
  const int* seq_slot;
  int n;
};

// A thread walks VEC neighbouring channels down ROWS rows; with TAPS > 0 (their number known) the inputs of the rows before
// stay in registers as long as the sequence goes on, else every tap's input is fetched. The order of a channel's sum is the
// taps', either way. The blocks behind those of the channels form the steps.
template <int VEC, int TAPS, int ROWS>
__global__ void __launch_bounds__(kThreads) space_prepare_kernel(const SpacePrepArgs a, int conv_blocks) {
  bw::pdl_enter();
  typedef typename VecOf<VEC>::type vec_t;
  const int r0 = blockIdx.x * ROWS, end = min(r0 + ROWS, a.n);
  if (static_cast<int>(blockIdx.y) >= conv_blocks) {
    const int h = (blockIdx.y - conv_blocks) * kThreads + threadIdx.x;
    if (h >= a.heads) return;
    const float bias = a.dt_bias[h], rate = a.rate[h];
    for (int r = r0; r < end; ++r) {
      float* to = a.out + static_cast<size_t>(r) * a.out_stride + a.out_step + h;
      const float t = softplus_f(__fadd_rn(a.u[static_cast<size_t>(r) * a.u_stride + a.step0 + h], bias));
      to[0] = t, to[a.heads] = expf(-__fmul_rn(rate, t));
    }
    return;
  }
  const int c = (blockIdx.y * kThreads + threadIdx.x) * VEC;
  if (c >= a.channels) return;
  const vec_t bias = *reinterpret_cast<const vec_t*>(a.conv_b + c);
  constexpr int KEPT = TAPS > 0 ? TAPS : 1;
  vec_t x[KEPT], w[KEPT];  // the inputs that a row's taps see, the row's own last
#pragma unroll
  for (int t = 0; t < TAPS; ++t) w[t] = *reinterpret_cast<const vec_t*>(a.conv_t + static_cast<size_t>(t) * a.channels + c);
  const float* u = a.u + a.conv0 + c;
  int seq_before = -1;
  for (int r = r0; r < end; ++r) {
    const int p = a.pos[r], seq = a.row_seq[r], row0 = a.seq_row0[seq];
    float* st = a.conv_state ? a.conv_state + static_cast<size_t>(a.seq_slot[seq]) * (a.taps - 1) * a.channels + c : nullptr;
    auto input = [&](int back) -> vec_t {  // the input `back` rows before this one
      if (p - back < 0) return vec_t{};
      return *reinterpret_cast<const vec_t*>(r - back >= row0 ? u + static_cast<size_t>(r - back) * a.u_stride
                                                              : st + static_cast<size_t>(a.taps - 1 - (row0 - (r - back))) * a.channels);
    };
    vec_t sum = bias;
    float* sf = reinterpret_cast<float*>(&sum);
    auto add = [&](const vec_t& wt, const vec_t& xt) {
      const float* xf = reinterpret_cast<const float*>(&xt);
      const float* wf = reinterpret_cast<const float*>(&wt);
#pragma unroll
      for (int e = 0; e < VEC; ++e) sf[e] = __fmaf_rn(wf[e], xf[e], sf[e]);
    };
    if (TAPS > 0) {
      if (seq == seq_before) {
#pragma unroll
        for (int t = 0; t < TAPS - 1; ++t) x[t] = x[t + 1];
      } else {
#pragma unroll
        for (int t = 0; t < TAPS - 1; ++t) x[t] = input(TAPS - 1 - t);
      }
      x[KEPT - 1] = input(0);
#pragma unroll
      for (int t = 0; t < TAPS; ++t) add(w[t], x[t]);
      if (a.keep && st) {  // the sequence's only row: the inputs move up by one
#pragma unroll
        for (int t = 1; t < TAPS; ++t) *reinterpret_cast<vec_t*>(st + static_cast<size_t>(t - 1) * a.channels) = x[t];
      }
      seq_before = seq;
    } else {
      for (int t = 0; t < a.taps; ++t) {
        const vec_t xt = input(a.taps - 1 - t);
        add(*reinterpret_cast<const vec_t*>(a.conv_t + static_cast<size_t>(t) * a.channels + c), xt);
        if (a.keep && st && t >= 1) *reinterpret_cast<vec_t*>(st + static_cast<size_t>(t - 1) * a.channels) = xt;
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) sf[e] = __fmul_rn(sf[e], sigmoid_f(sf[e]));
    *reinterpret_cast<vec_t*>(a.out + static_cast<size_t>(r) * a.out_stride + c) = sum;
  }
}

// What follows the state-space recurrence: y = o * g sigmoid(g), then every one of the row's `groups` equal parts divided by
// sqrt(mean(y^2) + eps) of its own, times w. A block per row and part.
template <int VEC>
__global__ void __launch_bounds__(256)
gated_group_norm_kernel(const float* __restrict__ o, const float* __restrict__ gate, int gate_stride, const float* __restrict__ w,
                        float eps, act_t* out, int width, int size) {
  bw::pdl_enter();
  extern __shared__ __align__(16) float row[];
  __shared__ float red[32];
  typedef typename VecOf<VEC>::type vec_t;
  const int first = blockIdx.y * size;
  const float* src = o + static_cast<size_t>(blockIdx.x) * width + first;
  const float* g = gate + static_cast<size_t>(blockIdx.x) * gate_stride + first;
  act_t* dst = out + static_cast<size_t>(blockIdx.x) * width + first;
  float ss = 0.0f;
  for (int i = threadIdx.x * VEC; i < size; i += blockDim.x * VEC) {
    vec_t v = *reinterpret_cast<const vec_t*>(src + i);
    const vec_t z = *reinterpret_cast<const vec_t*>(g + i);
    float* vf = reinterpret_cast<float*>(&v);
    const float* zf = reinterpret_cast<const float*>(&z);
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      vf[e] = __fmul_rn(vf[e], __fmul_rn(zf[e], sigmoid_f(zf[e])));
      ss = __fmaf_rn(vf[e], vf[e], ss);
    }
    *reinterpret_cast<vec_t*>(row + i) = v;
  }
  const float inv = bw::rms_scale(bw::block_sum(ss, red), size, eps);
  for (int i = threadIdx.x * VEC; i < size; i += blockDim.x * VEC) {  // (each thread reads back only what it wrote)
    float y[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) y[e] = bw::rms_apply(row[i + e], inv, w[first + i + e]);
    if constexpr (VEC == 4) {
#if BW_ACT_BF16
      uint2 packed;
      packed.x = bw::pack_bf16(y[0], y[1]), packed.y = bw::pack_bf16(y[2], y[3]);
      *reinterpret_cast<uint2*>(dst + i) = packed;
#else
      *reinterpret_cast<float4*>(dst + i) = make_float4(y[0], y[1], y[2], y[3]);
#endif
    } else {
      dst[i] = bw::from_f<act_t>(y[0]);
    }
  }
}

// Token shift: mix_s = x + (x' - x) mu_s for `mixes` vectors mu, x' the row before of the same sequence (from the
// state for the step's first row, zero for a sequence's first token). out: [mixes, n, width], as the products read them.
// With `keep` (steps of one row per sequence) the state becomes the row.
__global__ void __launch_bounds__(256)
shift_mix_kernel(const float* __restrict__ x, const float* __restrict__ mu, int mixes, float* last, int keep, act_t* out, int n,
                 int width, const int* __restrict__ pos, const int* __restrict__ row_seq, const int* __restrict__ seq_row0,
                 const int* __restrict__ seq_slot) {
  bw::pdl_enter();
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= width) return;
  const int r = blockIdx.x;
  const int seq = row_seq[r];
  float* st = last + static_cast<size_t>(seq_slot[seq]) * width + c;
  const float v = x[static_cast<size_t>(r) * width + c];
  float before = 0.0f;
  if (r > seq_row0[seq]) before = x[static_cast<size_t>(r - 1) * width + c];
  else if (pos[r] > 0) before = *st;
  if (keep) *st = v;
  const float d = __fsub_rn(before, v);
  for (int s = 0; s < mixes; ++s)
    out[(static_cast<size_t>(s) * n + r) * width + c] = bw::from_f<act_t>(__fmaf_rn(d, mu[static_cast<size_t>(s) * width + c], v));
}

// Two sublayers side by side and the block's norm behind them, one block per row:
//   y = (a / rms(a) * wa + b / rms(b) * wb) / 2
// and either y into `y`, or x += layernorm(y) * w with the summed row rounded into `xn`.
__global__ void __launch_bounds__(256)
pair_mean_kernel(const float* __restrict__ a, const float* __restrict__ wa, const float* __restrict__ b,
                 const float* __restrict__ wb, float eps, float* y, int width, const float* __restrict__ w, float norm_eps,
                 float* x, act_t* xn) {
  bw::pdl_enter();
  extern __shared__ float row[];
  __shared__ float red[32];
  const size_t base = static_cast<size_t>(blockIdx.x) * width;
  float sa = 0.0f, sb = 0.0f;
  for (int i = threadIdx.x; i < width; i += 256) {
    const float va = a[base + i], vb = b[base + i];
    sa = __fmaf_rn(va, va, sa), sb = __fmaf_rn(vb, vb, sb);
  }
  const float ia = bw::rms_scale(bw::block_sum(sa, red), width, eps), ib = bw::rms_scale(bw::block_sum(sb, red), width, eps);
  float s = 0.0f;
  for (int i = threadIdx.x; i < width; i += 256) {
    const float v = __fmul_rn(0.5f, __fadd_rn(bw::rms_apply(a[base + i], ia, wa[i]), bw::rms_apply(b[base + i], ib, wb[i])));
    if (x) {
      row[i] = v;
      s = __fadd_rn(s, v);
    } else {
      y[base + i] = v;
    }
  }
  if (!x) return;
  const float fw = static_cast<float>(width);
  const float mean = __fdiv_rn(bw::block_sum(s, red), fw);
  float q = 0.0f;
  for (int i = threadIdx.x; i < width; i += 256) {
    const float d = __fsub_rn(row[i], mean);
    q = __fmaf_rn(d, d, q);
  }
  const float inv = __fdiv_rn(1.0f, __fsqrt_rn(__fadd_rn(__fdiv_rn(bw::block_sum(q, red), fw), norm_eps)));
  for (int i = threadIdx.x; i < width; i += 256) {
    const float v = __fadd_rn(x[base + i], __fmul_rn(__fmul_rn(__fsub_rn(row[i], mean), inv), w[i]));
    x[base + i] = v;
    if (xn) xn[base + i] = bw::from_f<act_t>(v);
  }
}

template <int MODE, int LP, int V>
int launch_scan(ScanArgs a, int tiles, int longest, cudaStream_t stream) {
  typedef Shape<MODE, LP, V> T;
  // Tokens staged at a time: no more than the longest sequence of the step can have (a step of single rows stages
  // one, so that many of its small blocks share an SM), at most 32 (a chunk is a multiple of the warps beyond that), and no more
  // than two blocks of an SM have room for.
  a.chunk = 1;
  while (a.chunk < 32 && a.chunk < longest) a.chunk *= 2;
  auto bytes = [](int chunk) { return static_cast<size_t>(2 * chunk * T::W + chunk * T::CB) * sizeof(float); };
  while (a.chunk > kWarps && bytes(a.chunk) > 108 * 1024) a.chunk /= 2;
  const size_t smem = bytes(a.chunk);
  static size_t allowed = 48 * 1024;
  if (smem > allowed) {
    cudaError_t e = cudaFuncSetAttribute(state_scan_kernel<MODE, LP, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) {
      bw::set_error("state_scan: %zu bytes of shared memory: %s", smem, cudaGetErrorString(e));
      return static_cast<int>(e);
    }
    allowed = smem;
  }
  const int cols = MODE == kMemory ? a.vdim + 1 : a.vdim;
  bw::launch_pdl(state_scan_kernel<MODE, LP, V>, dim3(tiles, a.heads, (cols + T::CB - 1) / T::CB), dim3(kThreads), smem, stream, a);
  return bw::launch_status();
}

template <int MODE>
int launch_mode(const ScanArgs& a, int tiles, int longest, cudaStream_t stream) {
  if (a.dim <= 16) return launch_scan<MODE, 4, 1>(a, tiles, longest, stream);
  if (a.dim <= 32) return launch_scan<MODE, 8, 1>(a, tiles, longest, stream);
  if (a.dim <= 64) return launch_scan<MODE, 16, 1>(a, tiles, longest, stream);
  if (a.dim <= 128) return launch_scan<MODE, 16, 2>(a, tiles, longest, stream);
  if (a.dim <= 256) return launch_scan<MODE, 32, 2>(a, tiles, longest, stream);
  if (a.dim <= 512) return launch_scan<MODE, 32, 4>(a, tiles, longest, stream);
  bw::set_error("state_scan: key size %d (up to 512)", a.dim);
  return -1;
}

bool on16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace

// mode 0: the delta rule (decay = g, s0 = beta, s1 = q . k per query head); 1: the bonus form (decay = z with decay_bias, bonus = u); 2: the matrix memory
// (s0, s1 = the projections of the forget and the input gate with their biases, cap; aux [n, heads, 2]); 3: the state-space form (s0 = the
// decays, s1 = the steps, bonus = D [heads]). q and k
// rows hold heads / rep heads. o: [n, heads * vdim]. tiles: one per sequence (sequence, first row, rows).
BW_API int BW_FN(state_scan)(int mode, const float* q, int q_stride, const float* k, int k_stride, const float* v,
                             int v_stride, int rep, const float* decay, int decay_stride, const float* decay_bias,
                             const float* bonus, const float* s0, const float* s1, int s_stride, const float* s0_bias,
                             const float* s1_bias, float cap, float* state, float* o, float* aux, const int* tile_seq,
                             const int* tile_row0, const int* tile_rows, int tiles, const int* seq_pos0, const int* seq_slot,
                             int n, int heads, int dim, int vdim, cudaStream_t stream) {
  if (tiles <= 0 || n <= 0) return 0;
  if (heads <= 0 || dim <= 0 || vdim <= 0 || rep <= 0 || heads % rep) {
    bw::set_error("state_scan: %d heads, %d to a query head, sizes %d / %d", heads, rep, dim, vdim);
    return -1;
  }
  ScanArgs a;
  a.q = q, a.k = k, a.v = v, a.q_stride = q_stride, a.k_stride = k_stride, a.v_stride = v_stride, a.rep = rep;
  a.decay = decay, a.decay_stride = decay_stride, a.decay_bias = decay_bias, a.bonus = bonus;
  a.s0 = s0, a.s1 = s1, a.s_stride = s_stride, a.s0_bias = s0_bias, a.s1_bias = s1_bias, a.cap = cap;
  a.state = state, a.o = o, a.aux = aux, a.tile_seq = tile_seq, a.tile_row0 = tile_row0, a.tile_rows = tile_rows;
  a.seq_pos0 = seq_pos0, a.seq_slot = seq_slot, a.heads = heads, a.dim = dim, a.vdim = vdim, a.chunk = 1;
  // 16 bytes at a time where every row and head starts on 16 bytes
  a.wide = dim % 4 == 0 && vdim % 4 == 0 && q_stride % 4 == 0 && k_stride % 4 == 0 && v_stride % 4 == 0 &&
           (mode == kMemory || decay_stride % 4 == 0) && on16(q) && on16(k) && on16(v) && on16(decay) && on16(state);
  const int longest = n - tiles + 1;
  switch (mode) {
    case kDelta: return launch_mode<kDelta>(a, tiles, longest, stream);
    case kBonus: return launch_mode<kBonus>(a, tiles, longest, stream);
    case kMemory: return launch_mode<kMemory>(a, tiles, longest, stream);
    case kSpace: return launch_mode<kSpace>(a, tiles, longest, stream);
  }
  bw::set_error("state_scan: unknown mode %d", mode);
  return -1;
}

// gate_kind 0: sigmoid(g); 1: g sigmoid(g). w_per_head: w holds heads * vdim numbers (else vdim). aux may be null.
BW_API int BW_FN(scan_finish)(const float* o, const float* aux, float q_scale, const float* w, int w_per_head,
                              const float* gate, int gate_stride, int gate_kind, float eps, void* out, int n, int heads,
                              int vdim, cudaStream_t stream) {
  if (n <= 0) return 0;
  FinishArgs a;
  a.o = o, a.aux = aux, a.q_scale = q_scale, a.w = w, a.w_stride = w_per_head ? vdim : 0, a.gate = gate;
  a.gate_stride = gate_stride, a.gate_silu = gate_kind, a.eps = eps, a.out = static_cast<act_t*>(out), a.heads = heads, a.vdim = vdim;
  bw::launch_pdl(scan_finish_kernel, dim3(n, (heads + kThreads / 32 - 1) / (kThreads / 32)), dim3(kThreads), 0, stream, a);
  return bw::launch_status();
}

BW_API int BW_FN(delta_prepare)(const float* u, int u_stride, int beta_col, const float* conv_t, int taps, float* conv_state,
                                int keep, float* z, int z_stride, const float* dt_bias, const float* a_log, float* out,
                                int out_stride, const int* pos, const int* row_seq, const int* seq_row0, const int* seq_slot,
                                int n, int heads, int kv_heads, int dim, int vdim, float q_scale, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (dim > 32 * kMaxPer || vdim > 32 * kMaxPer) {
    bw::set_error("delta_prepare: head sizes %d / %d (up to %d)", dim, vdim, 32 * kMaxPer);
    return -1;
  }
  if (taps > 1 && !conv_state) {
    bw::set_error("delta_prepare: a convolution of %d taps needs the requests' state", taps);
    return -1;
  }
  DeltaPrepArgs a;
  a.u = u, a.u_stride = u_stride, a.beta_col = beta_col, a.conv_t = conv_t, a.taps = taps;
  a.conv_state = taps > 1 ? conv_state : nullptr, a.keep = keep, a.z = z, a.z_stride = z_stride, a.dt_bias = dt_bias, a.a_log = a_log;
  a.out = out, a.out_stride = out_stride, a.pos = pos, a.row_seq = row_seq, a.seq_row0 = seq_row0, a.seq_slot = seq_slot;
  a.heads = heads, a.kv_heads = kv_heads, a.dim = dim, a.vdim = vdim, a.q_scale = q_scale;
  const dim3 grid(n, (kv_heads + 2 * heads + 1 + kWarps - 1) / kWarps);
  if (dim % 4 == 0 && vdim % 4 == 0 && u_stride % 4 == 0 && out_stride % 4 == 0 && on16(u) && on16(conv_t) && on16(conv_state) && on16(out))
    bw::launch_pdl(delta_prepare_kernel<4>, grid, dim3(kThreads), 0, stream, a);
  else
    bw::launch_pdl(delta_prepare_kernel<1>, grid, dim3(kThreads), 0, stream, a);
  return bw::launch_status();
}

// u's columns: conv0 .. conv0 + channels - 1 into the convolution, step0 .. step0 + heads - 1 the steps' projections. out
// [n, out_stride]: the channels, from out_step (>= channels) on the heads' steps and their decays.
BW_API int BW_FN(space_prepare)(const float* u, int u_stride, int conv0, int channels, int step0, int heads, const float* conv_t,
                                const float* conv_b, int taps, float* conv_state, int keep, const float* dt_bias,
                                const float* rate, float* out, int out_stride, int out_step, const int* pos, const int* row_seq,
                                const int* seq_row0, const int* seq_slot, int n, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (taps <= 0 || channels <= 0 || heads <= 0 || (taps > 1 && !conv_state)) {
    bw::set_error("space_prepare: %d channels, %d heads, %d taps (more than one needs the requests' state)", channels, heads, taps);
    return -1;
  }
  SpacePrepArgs a;
  a.u = u, a.u_stride = u_stride, a.conv0 = conv0, a.channels = channels, a.step0 = step0, a.heads = heads;
  a.conv_t = conv_t, a.conv_b = conv_b, a.taps = taps, a.conv_state = taps > 1 ? conv_state : nullptr, a.keep = keep;
  a.dt_bias = dt_bias, a.rate = rate, a.out = out, a.out_stride = out_stride, a.out_step = out_step;
  a.pos = pos, a.row_seq = row_seq, a.seq_row0 = seq_row0, a.seq_slot = seq_slot, a.n = n;
  const bool by_four = channels % 4 == 0 && u_stride % 4 == 0 && out_stride % 4 == 0 && conv0 % 4 == 0 && on16(u) && on16(conv_t) &&
                       on16(conv_b) && on16(conv_state) && on16(out);
  const int vec = by_four ? 4 : 1;
  const int conv_blocks = (channels / vec + kThreads - 1) / kThreads;
  const unsigned blocks = conv_blocks + (heads + kThreads - 1) / kThreads;
#define BW_SPACE(T, R)                                                                                                      \
  do {                                                                                                                      \
    if (by_four) bw::launch_pdl(space_prepare_kernel<4, T, R>, dim3((n + R - 1) / R, blocks), dim3(kThreads), 0, stream, a, conv_blocks); \
    else bw::launch_pdl(space_prepare_kernel<1, T, R>, dim3((n + R - 1) / R, blocks), dim3(kThreads), 0, stream, a, conv_blocks); \
  } while (0)
  // (a step of few rows spreads them over the machine)
  if (n <= 64) {
    switch (taps) {
      case 1: BW_SPACE(1, 1); break;
      case 2: BW_SPACE(2, 1); break;
      case 3: BW_SPACE(3, 1); break;
      case 4: BW_SPACE(4, 1); break;
      default: BW_SPACE(0, 1);
    }
  } else {
    switch (taps) {
      case 1: BW_SPACE(1, 4); break;
      case 2: BW_SPACE(2, 4); break;
      case 3: BW_SPACE(3, 4); break;
      case 4: BW_SPACE(4, 4); break;
      default: BW_SPACE(0, 1);
    }
  }
#undef BW_SPACE
  return bw::launch_status();
}

// o: [n, width], gate: float32 rows of gate_stride floats, w: [width], out: [n, width] in the activation type.
BW_API int BW_FN(gated_group_norm)(const float* o, const float* gate, int gate_stride, const float* w, float eps, void* out, int n,
                                   int width, int groups, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (groups <= 0 || width <= 0 || width % groups || width / groups > 48 * 1024 / 4 || groups > 65535) {
    bw::set_error("gated_group_norm: %d columns in %d groups (of at most 12288)", width, groups);
    return -1;
  }
  const int size = width / groups;
  const bool by_four = size % 4 == 0 && gate_stride % 4 == 0 && on16(o) && on16(gate) && on16(out);
  const int want = by_four ? size / 4 : size;
  const int threads = want >= 256 ? 256 : (want + 31) / 32 * 32;
  const size_t smem = static_cast<size_t>(size) * sizeof(float);
  act_t* dst = static_cast<act_t*>(out);
  if (by_four)
    bw::launch_pdl(gated_group_norm_kernel<4>, dim3(n, groups), dim3(threads), smem, stream, o, gate, gate_stride, w, eps, dst, width, size);
  else
    bw::launch_pdl(gated_group_norm_kernel<1>, dim3(n, groups), dim3(threads), smem, stream, o, gate, gate_stride, w, eps, dst, width, size);
  return bw::launch_status();
}

BW_API int BW_FN(shift_mix)(const float* x, const float* mu, int mixes, float* last, int keep, void* out, int n, int width,
                            const int* pos, const int* row_seq, const int* seq_row0, const int* seq_slot, cudaStream_t stream) {
  if (n <= 0) return 0;
  bw::launch_pdl(shift_mix_kernel, dim3(n, (width + 255) / 256), dim3(256), 0, stream, x, mu, mixes, last, keep,
                 static_cast<act_t*>(out), n, width, pos, row_seq, seq_row0, seq_slot);
  return bw::launch_status();
}

// x null: y = the mean of the two normed rows. Otherwise x += layernorm(that) * w, and the summed row into xn (if given).
BW_API int BW_FN(pair_mean)(const float* a, const float* wa, const float* b, const float* wb, float eps, float* y, int n,
                            int width, const float* w, float norm_eps, float* x, void* xn, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (width <= 0 || width > 48 * 1024 / 4) {
    bw::set_error("pair_mean: width %d (1 .. 12288)", width);
    return -1;
  }
  bw::launch_pdl(pair_mean_kernel, dim3(n), dim3(256), x ? static_cast<size_t>(width) * sizeof(float) : 0, stream, a, wa, b, wb,
                 eps, y, width, w, norm_eps, x, static_cast<act_t*>(xn));
  return bw::launch_status();
}
