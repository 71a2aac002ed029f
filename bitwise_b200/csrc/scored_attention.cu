// Grouped-query softmax attention over paged keys and values with optional steps around the
// scores, and the kernels that prepare its operands.
//
//   qkv_prepare        per row and head: a short causal convolution over time on every channel of
//                      the projected q, k, v (inputs before the step's first row come from the
//                      request's state slot), a root-mean-square norm per head of q and k, the
//                      rotation of the leading entries of q and k (pair i = entries 2i, 2i + 1, or i and
//                      i + pairs), q into the step's buffer, k and v into their pages
//   conv_state_update  the convolution's inputs of a request's last taps - 1 positions
//   scored_attention   s = (q . k) * scale; s <- cap * tanh(s / cap); s <- s - slope_h * (i - j);
//                      window or chunks; softmax with an optional extra one in the denominator; the values
//                      may be the keys themselves (no value pages); several maps (attentions with queries and keys
//                      of their own) may weight the same values
//   scored_difference  two maps of a head become one output: a1 - lambda a2, a norm over the head, an output gate
//
// Everything after the projection is float32 in both precisions; only what is loaded and stored
// changes type. Keys are walked in tiles of 32 at fixed absolute positions, so what a query gets
// depends on its own keys only: not on the other rows of the step, nor on where a portion began.
#include "bw_act.cuh"
#include "bw_mma.cuh"

#include <math.h>

namespace {

// ---------------------------------------------------------------------------------------
// qkv_prepare. One block per row, a warp per head of q, k or v at a time; lane l holds the
// entries l, l + 32, ... of the head (up to kMaxE * 32).
constexpr int kMaxE = 8;
constexpr int kPrepWarps = 4;

struct PrepArgs {
  const float* u;            // [n, cols] projected rows: q heads, then k heads, then v heads
  int cols;
  int u_stride;              // floats between two rows of u (cols, or more where the rows are columns of a wider product)
  const float* bias;         // [cols] added to every projected row (also to rows read from the state), or null
  const float* vmix_src;     // [n, v_heads * vdim] values that this layer's values are mixed with, or null
  const float* vmix_lambda;  // one number: v <- (1 - lambda) v + lambda vmix_src
  float* v_keep;             // [n, v_heads * vdim]: the values as stored, kept in float32 for later layers, or null
  const float* conv_w;       // [cols, taps] or null
  const float* conv_wt;      // the same transposed, [taps, cols], for the kernel that reads four channels at a time
  int taps;
  const float* conv_state;   // [slots, taps - 1, cols] or null
  const float* q_norm;       // [dim] or null
  const float* k_norm;
  float eps;
  const float* cos_t;        // [positions, pairs] or null
  const float* sin_t;
  int pairs;
  int half_layout;           // pair i is made of entries i and i + pairs instead of 2i and 2i + 1
  const int* pos;
  const int* row_seq;
  const int* seq_row0;
  const int* seq_pos0;
  const int* seq_slot;
  const int* block_table;
  int max_blocks;
  act_t* kcache;             // [pages, kv_heads, page, dim]
  act_t* vcache;             // [pages, kv_heads, page, vdim] or null
  act_t* q_out;              // [n, heads * dim]
  int heads, kv_heads /* 0: nothing is stored */, v_heads, dim, vdim, page;
};

__global__ void __launch_bounds__(kPrepWarps * 32) qkv_prepare_kernel(const PrepArgs a) {
  bw::pdl_enter();
  __shared__ float heads_sm[kPrepWarps][kMaxE * 32];  // a head at a time, for partners that other lanes hold
  const int r = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int p = a.pos[r];
  const int seq = a.row_seq[r];
  const int row0 = a.seq_row0[seq];
  const int slot = a.conv_state ? a.seq_slot[seq] : 0;
  const int total = a.heads + a.kv_heads + a.v_heads;
  for (int hs = blockIdx.y * kPrepWarps + warp; hs < total; hs += kPrepWarps * gridDim.y) {
    int size, col0;
    const float* norm_w;
    bool turns;
    if (hs < a.heads) {
      size = a.dim, col0 = hs * a.dim, norm_w = a.q_norm, turns = true;
    } else if (hs < a.heads + a.kv_heads) {
      size = a.dim, col0 = hs * a.dim, norm_w = a.k_norm, turns = true;
    } else {
      size = a.vdim, col0 = (a.heads + a.kv_heads) * a.dim + (hs - a.heads - a.kv_heads) * a.vdim, norm_w = nullptr;
      turns = false;
    }
    float val[kMaxE];
    float ss = 0.0f;
#pragma unroll
    for (int j = 0; j < kMaxE; ++j) {
      const int e = lane + 32 * j;
      float v = 0.0f;
      if (e < size) {
        const int c = col0 + e;
        if (a.conv_w) {
          // y_t = sum_j w[c][j] * u_(t - taps + 1 + j), taps ascending; inputs before position 0 are zero
          for (int t = 0; t < a.taps; ++t) {
            const int back = a.taps - 1 - t;
            if (p - back < 0) continue;
            const int rr = r - back;
            float src = rr >= row0
                            ? a.u[static_cast<size_t>(rr) * a.u_stride + c]
                            : a.conv_state[(static_cast<size_t>(slot) * (a.taps - 1) + (a.taps - 1 - (row0 - rr))) * a.cols + c];
            if (a.bias) src = __fadd_rn(src, a.bias[c]);
            v = __fmaf_rn(a.conv_w[static_cast<size_t>(c) * a.taps + t], src, v);
          }
        } else {
          v = a.u[static_cast<size_t>(r) * a.u_stride + c];
          if (a.bias) v = __fadd_rn(v, a.bias[c]);
        }
        if (!turns && (a.vmix_src || a.v_keep)) {  // a value head (keys and queries turn or are normed; values neither)
          const size_t at = static_cast<size_t>(r) * a.v_heads * a.vdim + (hs - a.heads - a.kv_heads) * a.vdim + e;
          if (a.vmix_src) {
            const float lam = a.vmix_lambda[0];
            v = __fmaf_rn(lam, a.vmix_src[at], __fmul_rn(__fsub_rn(1.0f, lam), v));
          }
          if (a.v_keep) a.v_keep[at] = v;
        }
        ss = __fmaf_rn(v, v, ss);
      }
      val[j] = v;
    }
    if (norm_w) {
      const float inv = bw::rms_scale(bw::warp_sum(ss), size, a.eps);
#pragma unroll
      for (int j = 0; j < kMaxE; ++j) {
        const int e = lane + 32 * j;
        if (e < size) val[j] = bw::rms_apply(val[j], inv, norm_w[e]);
      }
    }
    if (turns && a.pairs > 0 && a.half_layout) {
      float* hv = heads_sm[warp];
      __syncwarp();
#pragma unroll
      for (int j = 0; j < kMaxE; ++j)
        if (lane + 32 * j < size) hv[lane + 32 * j] = val[j];
      __syncwarp();
#pragma unroll
      for (int j = 0; j < kMaxE; ++j) {
        const int e = lane + 32 * j;
        if (e < 2 * a.pairs && e < size) {
          const bool second = e >= a.pairs;
          const int i = second ? e - a.pairs : e;
          const float other = hv[second ? i : i + a.pairs];
          const float c = a.cos_t[static_cast<size_t>(p) * a.pairs + i], s = a.sin_t[static_cast<size_t>(p) * a.pairs + i];
          val[j] = second ? __fadd_rn(__fmul_rn(val[j], c), __fmul_rn(other, s))
                          : __fsub_rn(__fmul_rn(val[j], c), __fmul_rn(other, s));
        }
      }
    } else if (turns && a.pairs > 0) {
#pragma unroll
      for (int j = 0; j < kMaxE; ++j) {
        const int e = lane + 32 * j;
        const float other = __shfl_xor_sync(0xffffffffu, val[j], 1);  // the partner of entry e is entry e ^ 1
        if (e < 2 * a.pairs && e < size) {
          const float c = a.cos_t[static_cast<size_t>(p) * a.pairs + (e >> 1)];
          const float s = a.sin_t[static_cast<size_t>(p) * a.pairs + (e >> 1)];
          val[j] = (e & 1) ? __fadd_rn(__fmul_rn(val[j], c), __fmul_rn(other, s))
                           : __fsub_rn(__fmul_rn(val[j], c), __fmul_rn(other, s));
        }
      }
    }
    act_t* dst;
    if (hs < a.heads) {
      dst = a.q_out + static_cast<size_t>(r) * a.heads * a.dim + hs * a.dim;
    } else {
      const int blk = a.block_table[static_cast<size_t>(seq) * a.max_blocks + p / a.page];
      if (hs < a.heads + a.kv_heads)
        dst = a.kcache + ((static_cast<size_t>(blk) * a.kv_heads + (hs - a.heads)) * a.page + p % a.page) * a.dim;
      else
        dst = a.vcache + ((static_cast<size_t>(blk) * a.v_heads + (hs - a.heads - a.kv_heads)) * a.page + p % a.page) * a.vdim;
    }
#pragma unroll
    for (int j = 0; j < kMaxE; ++j) {
      const int e = lane + 32 * j;
      if (e < size) dst[e] = bw::from_f<act_t>(val[j]);
    }
  }
}

// The same with four consecutive entries of a head per lane (head sizes and column counts that are
// multiples of 4): the projected rows, the state, the taps (transposed: [taps, cols]) and the norm
// weights are read 16 bytes at a time, a rotation's partners lie in one lane, and a lane stores its
// four results at once. Lane l holds entries 4 l .. 4 l + 3 and 128 + 4 l .. of the head.
#if BW_ACT_BF16
__device__ __forceinline__ void store4(__nv_bfloat16* dst, float4 v) {
  uint2 w;
  w.x = bw::pack_bf16(v.x, v.y), w.y = bw::pack_bf16(v.z, v.w);
  *reinterpret_cast<uint2*>(dst) = w;
}
#else
__device__ __forceinline__ void store4(float* dst, float4 v) { *reinterpret_cast<float4*>(dst) = v; }
#endif

__global__ void __launch_bounds__(kPrepWarps * 32) qkv_prepare_vec_kernel(const PrepArgs a) {
  bw::pdl_enter();
  __shared__ __align__(16) float heads_sm[kPrepWarps][kMaxE * 32];
  const int r = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int p = a.pos[r];
  const int seq = a.row_seq[r];
  const int row0 = a.seq_row0[seq];
  const int slot = a.conv_state ? a.seq_slot[seq] : 0;
  const int total = a.heads + a.kv_heads + a.v_heads;
  const float* urow = a.u + static_cast<size_t>(r) * a.u_stride;
  for (int hs = blockIdx.y * kPrepWarps + warp; hs < total; hs += kPrepWarps * gridDim.y) {
    int size, col0;
    const float* norm_w;
    bool turns;
    if (hs < a.heads + a.kv_heads) {
      size = a.dim, col0 = hs * a.dim, norm_w = hs < a.heads ? a.q_norm : a.k_norm, turns = true;
    } else {
      size = a.vdim, col0 = (a.heads + a.kv_heads) * a.dim + (hs - a.heads - a.kv_heads) * a.vdim, norm_w = nullptr;
      turns = false;
    }
    float4 val[2];
    float ss = 0.0f;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int e0 = 4 * lane + 128 * j;
      float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      if (e0 < size) {
        const int c = col0 + e0;
        if (a.conv_wt) {
          for (int t = 0; t < a.taps; ++t) {  // taps ascending, as in the kernel above
            const int back = a.taps - 1 - t;
            if (p - back < 0) continue;
            const int rr = r - back;
            const float* src = rr >= row0 ? urow - static_cast<size_t>(back) * a.u_stride + c
                                          : a.conv_state + (static_cast<size_t>(slot) * (a.taps - 1) + (a.taps - 1 - (row0 - rr))) * a.cols + c;
            float4 x = *reinterpret_cast<const float4*>(src);
            if (a.bias) {
              const float4 b = *reinterpret_cast<const float4*>(a.bias + c);
              x.x = __fadd_rn(x.x, b.x), x.y = __fadd_rn(x.y, b.y), x.z = __fadd_rn(x.z, b.z), x.w = __fadd_rn(x.w, b.w);
            }
            const float4 w = *reinterpret_cast<const float4*>(a.conv_wt + static_cast<size_t>(t) * a.cols + c);
            v.x = __fmaf_rn(w.x, x.x, v.x), v.y = __fmaf_rn(w.y, x.y, v.y), v.z = __fmaf_rn(w.z, x.z, v.z), v.w = __fmaf_rn(w.w, x.w, v.w);
          }
        } else {
          v = *reinterpret_cast<const float4*>(urow + c);
          if (a.bias) {
            const float4 b = *reinterpret_cast<const float4*>(a.bias + c);
            v.x = __fadd_rn(v.x, b.x), v.y = __fadd_rn(v.y, b.y), v.z = __fadd_rn(v.z, b.z), v.w = __fadd_rn(v.w, b.w);
          }
        }
        if (!turns && (a.vmix_src || a.v_keep)) {  // a value head
          const size_t at = static_cast<size_t>(r) * a.v_heads * a.vdim + (hs - a.heads - a.kv_heads) * a.vdim + e0;
          if (a.vmix_src) {
            const float lam = a.vmix_lambda[0], rest = __fsub_rn(1.0f, lam);
            const float4 f = *reinterpret_cast<const float4*>(a.vmix_src + at);
            v.x = __fmaf_rn(lam, f.x, __fmul_rn(rest, v.x)), v.y = __fmaf_rn(lam, f.y, __fmul_rn(rest, v.y));
            v.z = __fmaf_rn(lam, f.z, __fmul_rn(rest, v.z)), v.w = __fmaf_rn(lam, f.w, __fmul_rn(rest, v.w));
          }
          if (a.v_keep) *reinterpret_cast<float4*>(a.v_keep + at) = v;
        }
        ss = __fmaf_rn(v.x, v.x, ss), ss = __fmaf_rn(v.y, v.y, ss), ss = __fmaf_rn(v.z, v.z, ss), ss = __fmaf_rn(v.w, v.w, ss);
      }
      val[j] = v;
    }
    if (norm_w) {
      const float inv = bw::rms_scale(bw::warp_sum(ss), size, a.eps);
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int e0 = 4 * lane + 128 * j;
        if (e0 < size) {
          const float4 w = *reinterpret_cast<const float4*>(norm_w + e0);
          val[j].x = bw::rms_apply(val[j].x, inv, w.x), val[j].y = bw::rms_apply(val[j].y, inv, w.y);
          val[j].z = bw::rms_apply(val[j].z, inv, w.z), val[j].w = bw::rms_apply(val[j].w, inv, w.w);
        }
      }
    }
    if (turns && a.pairs > 0 && a.half_layout) {
      float* hv = heads_sm[warp];
      __syncwarp();
#pragma unroll
      for (int j = 0; j < 2; ++j)
        if (4 * lane + 128 * j < size) *reinterpret_cast<float4*>(hv + 4 * lane + 128 * j) = val[j];
      __syncwarp();
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        float* f = &val[j].x;
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const int e = 4 * lane + 128 * j + k;
          if (e < 2 * a.pairs && e < size) {
            const bool second = e >= a.pairs;
            const int i = second ? e - a.pairs : e;
            const float other = hv[second ? i : i + a.pairs];
            const float c = a.cos_t[static_cast<size_t>(p) * a.pairs + i], s = a.sin_t[static_cast<size_t>(p) * a.pairs + i];
            f[k] = second ? __fadd_rn(__fmul_rn(f[k], c), __fmul_rn(other, s))
                          : __fsub_rn(__fmul_rn(f[k], c), __fmul_rn(other, s));
          }
        }
      }
    } else if (turns && a.pairs > 0) {
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int e0 = 4 * lane + 128 * j;
        if (e0 >= size) continue;
        const int i0 = e0 >> 1;
        const size_t at = static_cast<size_t>(p) * a.pairs;
        if (i0 < a.pairs) {
          const float c = a.cos_t[at + i0], s = a.sin_t[at + i0];
          const float x = val[j].x, y = val[j].y;
          val[j].x = __fsub_rn(__fmul_rn(x, c), __fmul_rn(y, s)), val[j].y = __fadd_rn(__fmul_rn(y, c), __fmul_rn(x, s));
        }
        if (i0 + 1 < a.pairs) {
          const float c = a.cos_t[at + i0 + 1], s = a.sin_t[at + i0 + 1];
          const float x = val[j].z, y = val[j].w;
          val[j].z = __fsub_rn(__fmul_rn(x, c), __fmul_rn(y, s)), val[j].w = __fadd_rn(__fmul_rn(y, c), __fmul_rn(x, s));
        }
      }
    }
    act_t* dst;
    if (hs < a.heads) {
      dst = a.q_out + static_cast<size_t>(r) * a.heads * a.dim + hs * a.dim;
    } else {
      const int blk = a.block_table[static_cast<size_t>(seq) * a.max_blocks + p / a.page];
      if (hs < a.heads + a.kv_heads)
        dst = a.kcache + ((static_cast<size_t>(blk) * a.kv_heads + (hs - a.heads)) * a.page + p % a.page) * a.dim;
      else
        dst = a.vcache + ((static_cast<size_t>(blk) * a.v_heads + (hs - a.heads - a.kv_heads)) * a.page + p % a.page) * a.vdim;
    }
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int e0 = 4 * lane + 128 * j;
      if (e0 < size) store4(dst + e0, val[j]);
    }
  }
}

// state[slot][i] = the projected row of position end - (taps - 1) + i (i < taps - 1), `end` the
// request's length after this step: from the step's rows, from the old state, or zero before
// position 0. One thread per (sequence, channel) reads all it needs before it writes.
constexpr int kMaxTaps = 16;

__global__ void __launch_bounds__(128)
conv_state_update_kernel(const float* __restrict__ u, int u_stride, int cols, float* state, int taps, const int* __restrict__ tile_seq,
                         const int* __restrict__ tile_row0, const int* __restrict__ tile_rows,
                         const int* __restrict__ seq_pos0, const int* __restrict__ seq_slot) {
  bw::pdl_enter();
  const int t = blockIdx.x;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= cols) return;
  const int seq = tile_seq[t], row0 = tile_row0[t], cnt = tile_rows[t];
  const int pos0 = seq_pos0[seq];
  float* st = state + static_cast<size_t>(seq_slot[seq]) * (taps - 1) * cols + c;
  float keep[kMaxTaps];
#pragma unroll
  for (int i = 0; i < kMaxTaps; ++i) {
    if (i >= taps - 1) break;
    const int p = pos0 + cnt - (taps - 1) + i;
    float v = 0.0f;
    if (p >= pos0)
      v = u[static_cast<size_t>(row0 + p - pos0) * u_stride + c];
    else if (p >= 0)
      v = st[static_cast<size_t>(p - pos0 + taps - 1) * cols];
    keep[i] = v;
  }
#pragma unroll
  for (int i = 0; i < kMaxTaps; ++i) {
    if (i >= taps - 1) break;
    st[static_cast<size_t>(i) * cols] = keep[i];
  }
}

// ---------------------------------------------------------------------------------------
// Attention on the CUDA cores. A block takes one query tile (rows of one sequence at consecutive
// positions), one key/value head and up to `hb` of the query heads that read it; a warp works on
// one query (a row and a head) at a time, lane l on key l of the tile of 32: its score, the tile's
// maximum and sum over the warp, and the running (maximum, sum, weighted sum of values).
constexpr int kWarps = 8;
constexpr int kKeys = 32;
constexpr int kThreads = kWarps * 32;
constexpr int kQW = 4;  // queries per warp

struct ScoreArgs {
  float cap_exp;  // 2 * scale / softcap * log2(e): the exponent of the cap's exponential per unit of raw score
  float scale, softcap;
  int sink;
  const float* slopes;  // [heads] or null
  int window;
  const float* dist_a;  // [heads] or null: s <- s - dist_a[h] * ln(1 + dist_b[h] * (i - j))
  const float* dist_b;
  const float* sinks;   // [heads] or null: with `sink`, exp(sinks[h]) joins the denominator instead of exp(0)
  int keep_first;       // with a window: the keys j < keep_first stay visible to every later position
  int chunk;            // > 0: position i sees the keys j <= i with j / chunk == i / chunk (no window then)
  int maps;             // key heads that share a value head: key head g holds map g % maps of value head g / maps, and
                        // query head h is map h % maps of result head h / maps
};
// The first query head of a block's share of the heads on key head g (the others follow `maps` apart).
__device__ __forceinline__ int first_head(const ScoreArgs& sa, int g, int rep, int skip) {
  return (g / sa.maps * rep + skip) * sa.maps + g % sa.maps;
}
// The first key that a query at position pq sees (kept first keys apart). It never falls as pq grows.
__device__ __forceinline__ int first_seen(const ScoreArgs& sa, int pq) {
  if (sa.chunk > 0) return pq / sa.chunk * sa.chunk;
  return sa.window > 0 ? max(0, pq - sa.window + 1) : 0;
}

// What a query's head takes off a score by distance.
struct HeadBias {
  float slope, a, b;
};
__device__ __forceinline__ HeadBias head_bias(const ScoreArgs& sa, int h, bool ok) {
  HeadBias hb;
  hb.slope = sa.slopes && ok ? sa.slopes[h] : 0.0f;
  hb.a = sa.dist_a && ok ? sa.dist_a[h] : 0.0f;
  hb.b = sa.dist_a && ok ? sa.dist_b[h] : 0.0f;
  return hb;
}
// The first key a query at position pq sees inside its window (keys before keep_first are seen besides).
__device__ __forceinline__ bool key_seen(const ScoreArgs& sa, int pq, int lo, int kp) {
  return kp <= pq && (kp >= lo || kp < sa.keep_first);
}

#if BW_ACT_BF16
// What one of a thread's two queries (halves of its fragments) brings to a key tile, and what it carries along.
struct QueryWalk {
  HeadBias hb;
  int pq, lo;   // its position, the first key it sees
  bool ok;      // there is such a query
  float m, l;   // running maximum; this thread's share of the sum (the shares are joined at the end)
};

// The same on the serving precision's tensor-core path, where the scores come from bfloat16 operands: tanh through the hardware's
// exponential, tanh(x) = 1 - 2 / (exp(2x) + 1) (relative error of a few 1e-7, against the 4e-3 of a bfloat16 operand). A lane holds
// eight scores of a key tile per query, keys kp0, kp0 + 1, kp0 + 8, .. + 25, those of query h in the entries 2h and 2h + 1.
template <int HALVES>
__device__ __forceinline__ void modify_scores_fast(float (&sc)[4][4], const ScoreArgs& sa, const QueryWalk (&qw)[2], int kp0) {
  if (sa.softcap > 0.0f) {
    // cap * tanh(x) = cap - 2 cap / (exp(2x) + 1), x = s * scale / cap; exp(2x) = 2^(s * cap_exp)
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int h = 0; h < HALVES; ++h) {
        float& v = sc[i >> 1][2 * h + (i & 1)];
        const float e = bw::exp2_approx(__fmul_rn(v, sa.cap_exp));
        v = __fmaf_rn(__fmul_rn(-2.0f, sa.softcap), __fdividef(1.0f, __fadd_rn(e, 1.0f)), sa.softcap);
      }
  } else {
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int h = 0; h < HALVES; ++h) sc[i >> 1][2 * h + (i & 1)] = __fmul_rn(sc[i >> 1][2 * h + (i & 1)], sa.scale);
  }
  if (sa.slopes) {
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int h = 0; h < HALVES; ++h) {
        float& v = sc[i >> 1][2 * h + (i & 1)];
        v = __fsub_rn(v, __fmul_rn(qw[h].hb.slope, static_cast<float>(qw[h].pq - (kp0 + (i >> 1) * 8 + (i & 1)))));
      }
  }
  if (sa.dist_a) {
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int h = 0; h < HALVES; ++h) {
        float& v = sc[i >> 1][2 * h + (i & 1)];
        v = __fsub_rn(v, __fmul_rn(qw[h].hb.a, __logf(__fmaf_rn(qw[h].hb.b, static_cast<float>(qw[h].pq - (kp0 + (i >> 1) * 8 + (i & 1))), 1.0f))));
      }
  }
}

// Scores of a key tile into weights relative to the queries' running maxima, which move on with the sums; al: the factors of what
// was accumulated before. `whole`: every query sees every key of the tile.
template <int HALVES>
__device__ __forceinline__ void weigh_tile(float (&sc)[4][4], const ScoreArgs& sa, QueryWalk (&qw)[2], int kp0, bool whole, float (&al)[2]) {
  modify_scores_fast<HALVES>(sc, sa, qw, kp0);
  float mt[2] = {-INFINITY, -INFINITY}, sum[2] = {0.0f, 0.0f};
  if (!whole) {
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int h = 0; h < HALVES; ++h)
        if (!(qw[h].ok && key_seen(sa, qw[h].pq, qw[h].lo, kp0 + (i >> 1) * 8 + (i & 1)))) sc[i >> 1][2 * h + (i & 1)] = -INFINITY;
  }
#pragma unroll
  for (int i = 0; i < 8; ++i)
#pragma unroll
    for (int h = 0; h < HALVES; ++h) mt[h] = fmaxf(mt[h], sc[i >> 1][2 * h + (i & 1)]);
#pragma unroll
  for (int h = 0; h < HALVES; ++h) {
    mt[h] = fmaxf(mt[h], __shfl_xor_sync(0xffffffffu, mt[h], 1)), mt[h] = fmaxf(mt[h], __shfl_xor_sync(0xffffffffu, mt[h], 2));
    mt[h] = fmaxf(qw[h].m, mt[h]);
    // (a query that has seen no key yet holds zeros, which need no factor)
    al[h] = qw[h].m == -INFINITY ? (mt[h] == -INFINITY ? 1.0f : 0.0f) : __expf(__fsub_rn(qw[h].m, mt[h]));
  }
#pragma unroll
  for (int i = 0; i < 8; ++i)
#pragma unroll
    for (int h = 0; h < HALVES; ++h) {
      float& v = sc[i >> 1][2 * h + (i & 1)];
      v = v == -INFINITY ? 0.0f : __expf(__fsub_rn(v, mt[h]));
      sum[h] = __fadd_rn(sum[h], v);
    }
#pragma unroll
  for (int h = 0; h < HALVES; ++h) qw[h].l = __fmaf_rn(qw[h].l, al[h], sum[h]), qw[h].m = mt[h];
}
#endif

__device__ __forceinline__ float modify_score(float s, const ScoreArgs& sa, const HeadBias& hb, int pq, int kp) {
  s = __fmul_rn(s, sa.scale);
  if (sa.softcap > 0.0f) s = __fmul_rn(sa.softcap, tanhf(__fdiv_rn(s, sa.softcap)));
  if (sa.slopes) s = __fsub_rn(s, __fmul_rn(hb.slope, static_cast<float>(pq - kp)));
  if (sa.dist_a) s = __fsub_rn(s, __fmul_rn(hb.a, log1pf(__fmul_rn(hb.b, static_cast<float>(pq - kp)))));
  return s;
}
// Key tiles of `tile` keys that a walk from `from` visits: with kept first keys the tiles that hold
// them, then the tiles from the window's first on; the tiles between are passed over.
__device__ __forceinline__ int skip_gap(int k0, int keep_end, int win_begin) {
  return (k0 >= keep_end && k0 < win_begin) ? win_begin : k0;
}

template <int ACC>
__global__ void __launch_bounds__(kThreads)
scored_attention_kernel(const act_t* __restrict__ q, int q_stride, const act_t* __restrict__ kcache,
                        const act_t* __restrict__ vcache, const int* __restrict__ block_table, int max_blocks,
                        const int* __restrict__ tile_seq, const int* __restrict__ tile_row0,
                        const int* __restrict__ tile_rows, const int* __restrict__ seq_pos0,
                        const int* __restrict__ seq_row0, act_t* out, int o_stride, int heads, int kv_heads, int hb,
                        int dim, int vdim, int page, const ScoreArgs sa, float* partial) {
  bw::pdl_enter();
  extern __shared__ float sm[];
  const int ks = dim + 1;
  float* keys = sm;                                         // [32][dim + 1]
  float* vals = vcache ? keys + kKeys * ks : keys;          // [32][vdim], or the keys themselves
  const int vs = vcache ? vdim : ks;
  float* qs = keys + kKeys * ks + (vcache ? kKeys * vdim : 0);
  const int t = blockIdx.x, g = blockIdx.y;
  const int rep = heads / kv_heads, v_heads = kv_heads / sa.maps, gv = g / sa.maps;
  const int h0 = first_head(sa, g, rep, blockIdx.z * hb);
  const int nh = min(hb, rep - blockIdx.z * hb);
  const int seq = tile_seq[t], row0 = tile_row0[t], rows = tile_rows[t];
  const int nq = rows * nh;
  const int p0 = seq_pos0[seq] + (row0 - seq_row0[seq]);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int qi = warp; qi < nq; qi += kWarps) {
    const act_t* src = q + static_cast<size_t>(row0 + qi / nh) * q_stride + (h0 + qi % nh * sa.maps) * dim;
    for (int d = lane; d < dim; d += 32) qs[qi * dim + d] = bw::to_f(src[d]);
  }
  float m[kQW], l[kQW], acc[kQW][ACC];
#pragma unroll
  for (int j = 0; j < kQW; ++j) {
    m[j] = -INFINITY, l[j] = 0.0f;
#pragma unroll
    for (int i = 0; i < ACC; ++i) acc[j][i] = 0.0f;
  }
  const int last = p0 + rows - 1;
  const int first = first_seen(sa, p0);  // pages before it may be gone (kept first keys stay)
  const int keep = sa.window > 0 ? sa.keep_first : 0;
  const int keep_end = (keep + kKeys - 1) / kKeys * kKeys, win_begin = first / kKeys * kKeys;
  const int* bt = block_table + static_cast<size_t>(seq) * max_blocks;
  for (int k0 = skip_gap(0, keep_end, win_begin); k0 <= last; k0 = skip_gap(k0 + kKeys, keep_end, win_begin)) {
    __syncthreads();
    for (int kk = warp; kk < kKeys; kk += kWarps) {
      const int kp = k0 + kk;
      const bool have = kp <= last && (kp >= first || kp < keep);
      size_t at = 0, vat = 0;
      if (have) {
        const size_t blk = bt[kp / page];
        at = (blk * kv_heads + g) * page + kp % page, vat = (blk * v_heads + gv) * page + kp % page;
      }
      for (int d = lane; d < dim; d += 32) keys[kk * ks + d] = have ? bw::to_f(kcache[at * dim + d]) : 0.0f;
      if (vcache)
        for (int d = lane; d < vdim; d += 32) vals[kk * vs + d] = have ? bw::to_f(vcache[vat * vdim + d]) : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < kQW; ++j) {
      const int qi = warp + kWarps * j;
      if (qi >= nq) continue;
      const int pq = p0 + qi / nh;
      const int lo = first_seen(sa, pq);
      if (k0 > pq || (k0 + kKeys <= lo && k0 >= keep)) continue;  // no key of the tile is seen: the state stays
      const int kp = k0 + lane;
      const float* qv = qs + qi * dim;
      const float* kv = keys + lane * ks;
      float s = 0.0f;
      for (int d = 0; d < dim; ++d) s = __fmaf_rn(qv[d], kv[d], s);
      s = modify_score(s, sa, head_bias(sa, h0 + qi % nh * sa.maps, true), pq, kp);
      const bool seen = key_seen(sa, pq, lo, kp);
      if (!seen) s = -INFINITY;
      const float mt = bw::warp_max(s);
      const float mn = fmaxf(m[j], mt);
      const float alpha = m[j] == -INFINITY ? 0.0f : expf(__fsub_rn(m[j], mn));
      const float pw = seen ? expf(__fsub_rn(s, mn)) : 0.0f;
      l[j] = __fmaf_rn(l[j], alpha, bw::warp_sum(pw));
#pragma unroll
      for (int i = 0; i < ACC; ++i) acc[j][i] = __fmul_rn(acc[j][i], alpha);
      for (int kk = 0; kk < kKeys; ++kk) {
        const float pk = __shfl_sync(0xffffffffu, pw, kk);
        if (pk == 0.0f) continue;
        const float* vrow = vals + kk * vs;
#pragma unroll
        for (int i = 0; i < ACC; ++i) {
          const int d = i * 32 + lane;
          if (d < vdim) acc[j][i] = __fmaf_rn(pk, vrow[d], acc[j][i]);
        }
      }
      m[j] = mn;
    }
  }
#pragma unroll
  for (int j = 0; j < kQW; ++j) {
    const int qi = warp + kWarps * j;
    if (qi >= nq) continue;
    const int h = h0 + qi % nh * sa.maps;
    if (partial) {  // a record for the kernel that joins the maps: maximum, sum, weighted values relative to that maximum
      float* rec = partial + (static_cast<size_t>(row0 + qi / nh) * heads + h) * (vdim + 2);
      if (lane == 0) rec[0] = m[j], rec[1] = l[j];
#pragma unroll
      for (int i = 0; i < ACC; ++i)
        if (i * 32 + lane < vdim) rec[2 + i * 32 + lane] = acc[j][i];
      continue;
    }
    float den = l[j];
    if (sa.sink) den = __fadd_rn(den, expf(__fsub_rn(sa.sinks ? sa.sinks[h] : 0.0f, m[j])));  // the extra key (score 0 unless given)
    const float inv = __fdiv_rn(1.0f, den);
    act_t* dst = out + static_cast<size_t>(row0 + qi / nh) * o_stride + h * vdim;
#pragma unroll
    for (int i = 0; i < ACC; ++i) {
      const int d = i * 32 + lane;
      if (d < vdim) dst[d] = bw::from_f<act_t>(__fmul_rn(acc[j][i], inv));
    }
  }
}

template <int ACC>
int launch_scored(dim3 grid, size_t smem, cudaStream_t stream, const act_t* q, int q_stride, const act_t* kcache,
                  const act_t* vcache, const int* block_table, int max_blocks, const int* tile_seq, const int* tile_row0,
                  const int* tile_rows, const int* seq_pos0, const int* seq_row0, act_t* out, int o_stride, int heads,
                  int kv_heads, int hb, int dim, int vdim, int page, const ScoreArgs& sa, float* partial) {
  static size_t allowed = 48 * 1024;
  if (smem > allowed) {
    cudaError_t e = cudaFuncSetAttribute(scored_attention_kernel<ACC>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         static_cast<int>(smem));
    if (e != cudaSuccess) {
      bw::set_error("scored_attention: %zu bytes of shared memory: %s", smem, cudaGetErrorString(e));
      return static_cast<int>(e);
    }
    allowed = smem;
  }
  bw::launch_pdl(scored_attention_kernel<ACC>, grid, dim3(kThreads), smem, stream, q, q_stride, kcache, vcache, block_table,
                 max_blocks, tile_seq, tile_row0, tile_rows, seq_pos0, seq_row0, out, o_stride, heads, kv_heads, hb, dim,
                 vdim, page, sa, partial);
  return bw::launch_status();
}

// ---------------------------------------------------------------------------------------
// Two maps of a result head joined: the spans' records of query heads 2h and 2h + 1 merged in ascending order of the spans, as
// scored_attention_merge does, then o = a1 - lambda a2, o <- o / sqrt(mean(o^2) + eps) * keep, and the output gate. Two
// warps per row and result head, one for each map.
struct DifferenceArgs {
  const float* partial;  // [n, 2 * heads, spans, vdim + 2]
  int spans, queries /* n * heads */, heads, vdim;
  const float* lambda;   // one number
  float keep, eps;
  const float* gate;     // row r, head h: gate + r * gate_stride + (h * vdim + d) / gate_group, or null
  int gate_stride, gate_group;
  act_t* out;            // [n, heads * vdim]
};

// The records of one query joined in ascending order of the spans by a warp: m and l of the sum, and the weighted values, lane l's
// entries l, l + 32, ... of them. A lane looks at one span's maximum and sum, and the values of four spans are asked for together;
// spans in which the query saw no key hold nothing but their -infinity.
__device__ __forceinline__ void merge_spans(const float* __restrict__ rec, int spans, int vdim, int lane, float& m, float& l, float (&acc)[8]) {
  const int stride = vdim + 2;
  m = -INFINITY;
  for (int s0 = 0; s0 < spans; s0 += 32)
    if (s0 + lane < spans) m = fmaxf(m, rec[static_cast<size_t>(s0 + lane) * stride]);
  m = bw::warp_max(m);
  l = 0.0f;
#pragma unroll
  for (int i = 0; i < 8; ++i) acc[i] = 0.0f;
  for (int s0 = 0; s0 < spans; s0 += 32) {
    const float* r = rec + static_cast<size_t>(s0) * stride;
    const bool have = s0 + lane < spans;
    const float ms = have ? r[static_cast<size_t>(lane) * stride] : -INFINITY;
    const float ls = have ? r[static_cast<size_t>(lane) * stride + 1] : 0.0f;
    const float fs = ms == -INFINITY ? 0.0f : expf(__fsub_rn(ms, m));
    unsigned live = __ballot_sync(0xffffffffu, ms != -INFINITY);
    while (live) {
      constexpr int kBatch = 4;
      float v[kBatch][8], f[kBatch], lp[kBatch];
      bool take[kBatch];
#pragma unroll
      for (int b = 0; b < kBatch; ++b) {
        take[b] = live != 0;
        const int at = take[b] ? __ffs(live) - 1 : 0;
        live &= live - 1;
        f[b] = __shfl_sync(0xffffffffu, fs, at), lp[b] = __shfl_sync(0xffffffffu, ls, at);
        const float* src = r + static_cast<size_t>(at) * stride + 2 + lane;
#pragma unroll
        for (int i = 0; i < 8; ++i) v[b][i] = take[b] && i * 32 + lane < vdim ? src[i * 32] : 0.0f;
      }
#pragma unroll
      for (int b = 0; b < kBatch; ++b) {
        if (!take[b]) break;
        l = __fmaf_rn(lp[b], f[b], l);
#pragma unroll
        for (int i = 0; i < 8; ++i) acc[i] = __fmaf_rn(v[b][i], f[b], acc[i]);
      }
    }
  }
}

__global__ void __launch_bounds__(128) scored_difference_kernel(const DifferenceArgs a) {
  bw::pdl_enter();
  __shared__ float second[2][256];  // the second map's outputs of the block's two result heads
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, map = warp & 1;
  const int qi = blockIdx.x * 2 + (warp >> 1);
  const bool have = qi < a.queries;
  float o[8], m, l;
  if (have) {
    merge_spans(a.partial + (2 * static_cast<size_t>(qi) + map) * a.spans * (a.vdim + 2), a.spans, a.vdim, lane, m, l, o);
    const float inv = __fdiv_rn(1.0f, l);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      o[i] = __fmul_rn(o[i], inv);
      if (map) second[warp >> 1][i * 32 + lane] = o[i];
    }
  }
  __syncthreads();
  if (!have || map) return;
  const float lam = a.lambda[0];
  float ss = 0.0f;
#pragma unroll
  for (int i = 0; i < 8; ++i) {  // (entries beyond the head are zero)
    o[i] = __fmaf_rn(-lam, second[warp >> 1][i * 32 + lane], o[i]);
    ss = __fmaf_rn(o[i], o[i], ss);
  }
  const float f = __fmul_rn(bw::rms_scale(bw::warp_sum(ss), a.vdim, a.eps), a.keep);
  const int r = qi / a.heads, h = qi - r * a.heads;
  const float* gate = a.gate ? a.gate + static_cast<size_t>(r) * a.gate_stride : nullptr;
  act_t* dst = a.out + static_cast<size_t>(qi) * a.vdim;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int d = i * 32 + lane;
    if (d >= a.vdim) continue;
    float v = __fmul_rn(o[i], f);
    if (gate) v = __fdiv_rn(v, __fadd_rn(1.0f, expf(-gate[(h * a.vdim + d) / a.gate_group])));
    dst[d] = bw::from_f<act_t>(v);
  }
}

#if BW_ACT_BF16
// ---------------------------------------------------------------------------------------
// Attention on the tensor cores (bfloat16 operands, float32 accumulators; mma.sync m16n8k16).
// A block of four warps takes 64 stacked queries (rows of one query tile x the query heads of one
// key/value head), 16 per warp, and walks the keys in tiles of 32 at fixed absolute positions.
// Scores stay in the accumulators as float32: scale, cap, distance slope, mask, the running
// maximum and the weights exp(s - m) are formed there. The weights enter the second product as
// two bfloat16 parts (p = hi + lo), so the values are weighted with 16 bits of p. A query's
// result depends on its own keys and the fixed tiles only.
constexpr int kMmaWarps = 4;
constexpr int kMmaRows = 16 * kMmaWarps;
constexpr int kMmaKeys = 32;
__host__ __device__ constexpr int mma_q_rows(bool single) { return single ? 16 : kMmaRows; }  // queries that a block has room for
__host__ __device__ constexpr int mma_bufs(bool single) { return single ? 4 : 2; }            // buffers of key tiles
constexpr int kTableSlice = 264;  // page numbers of a block's keys that are staged in shared memory

// SINGLE: a step of single rows, whose blocks have at most 16 queries. All warps of a block take them then: each forms all scores and
// weights, and every fourth part of 16 value columns is its own (the sums are the same either way); and as the block's time is the way
// of the keys to it, more tiles are asked for ahead.
template <int VD16 /* value size / 16 */, bool SINGLE>
__global__ void __launch_bounds__(kMmaWarps * 32)
scored_attention_mma_kernel(const __nv_bfloat16* __restrict__ q, int q_stride, const __nv_bfloat16* __restrict__ kcache,
                            const __nv_bfloat16* __restrict__ vcache, const int* __restrict__ block_table, int max_blocks,
                            const int* __restrict__ tile_seq, const int* __restrict__ tile_row0,
                            const int* __restrict__ tile_rows, const int* __restrict__ seq_pos0,
                            const int* __restrict__ seq_row0, __nv_bfloat16* out, int o_stride, int heads, int kv_heads,
                            int hb, int dim, int page, const ScoreArgs sa, int span_tiles, int spans, float* partial) {
  constexpr int q_rows = mma_q_rows(SINGLE), bufs = mma_bufs(SINGLE);
  bw::pdl_enter();
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __shared__ int table_slice[kTableSlice];
  constexpr int vdim = VD16 * 16;
  constexpr int VT = VD16 * 2;  // accumulator tiles of 8 value columns
  const int kst = dim + 8;      // row strides in elements: 16 bytes more than a row, so that
  const int vst_own = vdim + 8; // ldmatrix reads eight rows from eight different banks
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(smem_raw);  // [q_rows][kst]
  __nv_bfloat16* ks_all = qs + q_rows * kst;                        // [bufs][32][kst]: the tile in use and the next ones
  __nv_bfloat16* vs_all = vcache ? ks_all + bufs * kMmaKeys * kst : ks_all;  // [bufs][32][vst]; the keys where values are keys
  const int vst = vcache ? vst_own : kst;
  const int t = blockIdx.x, g = blockIdx.y;
  const int rep = heads / kv_heads, v_heads = kv_heads / sa.maps, gv = g / sa.maps;
  const int zh = blockIdx.z / spans, span = blockIdx.z - zh * spans;  // the block's share of heads and of keys
  const int h0 = first_head(sa, g, rep, zh * hb), hstep = sa.maps;
  const int nh = min(hb, rep - zh * hb);
  const int seq = tile_seq[t], row0 = tile_row0[t], rows = tile_rows[t];
  const int nq = rows * nh;
  const int p0 = seq_pos0[seq] + (row0 - seq_row0[seq]);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int dparts = dim >> 3, vparts = vdim >> 3;
  const int wr = SINGLE ? 0 : warp * 16;
  // this thread's two queries: stacked rows sa_ and sb_ of the block
  const int sr_a = wr + (lane >> 2), sr_b = sr_a + 8;
  const bool ok_a = sr_a < nq, ok_b = sr_b < nq;
  const int pq_a = p0 + (ok_a ? sr_a / nh : 0), pq_b = p0 + (ok_b ? sr_b / nh : 0);
  QueryWalk qw[2] = {{head_bias(sa, h0 + sr_a % nh * hstep, ok_a), pq_a, first_seen(sa, pq_a), ok_a, -INFINITY, 0.0f},
                     {head_bias(sa, h0 + sr_b % nh * hstep, ok_b), pq_b, first_seen(sa, pq_b), ok_b, -INFINITY, 0.0f}};
  const int keep = sa.window > 0 ? sa.keep_first : 0;
  // the positions that this warp's queries span: tiles outside are skipped by the whole warp
  const int w_first = min(wr, max(nq - 1, 0)) / nh, w_last = min(wr + 15, max(nq - 1, 0)) / nh;
  const int w_lo = first_seen(sa, p0 + w_first), w_hi = p0 + w_last;
  const bool warp_has_rows = wr < nq;
  const bool warp_full = wr + 15 < nq;  // all 16 stacked rows of the warp are queries
  const int w_seen_to = p0 + w_first;           // keys up to here are seen by every query of the warp ...
  const int w_seen_from = first_seen(sa, p0 + w_last);  // ... from here on
  float acc[VT][4];
#pragma unroll
  for (int j = 0; j < VT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.0f;
  const int last = p0 + rows - 1;
  const int first = first_seen(sa, p0);  // pages before it may be gone (kept first keys stay)
  const int keep_end = (keep + kMmaKeys - 1) / kMmaKeys * kMmaKeys, win_begin = first / kMmaKeys * kMmaKeys;
  const int* bt = block_table + static_cast<size_t>(seq) * max_blocks;
  // With spans the block walks the key tiles at * span_tiles .. + span_tiles - 1 only (fixed absolute positions
  // again) and leaves a record for the merge instead of the result. Where the tile's queries see nothing before
  // their first key, the spans are counted from the one that holds it.
  int k_begin = skip_gap(0, keep_end, win_begin), k_end = last;
  if (span_tiles > 0) {
    const int at = span + (keep > 0 ? 0 : first / (span_tiles * kMmaKeys));
    k_begin = skip_gap(max(k_begin, at * span_tiles * kMmaKeys), keep_end, win_begin);
    k_end = min(k_end, (at + 1) * span_tiles * kMmaKeys - 1);
    if (k_begin > k_end) {
      // none of the block's queries reaches into this span: records that say so, nothing else
      for (int sr = tid; sr < nq; sr += kMmaWarps * 32) {
        float* rec = partial + ((static_cast<size_t>(row0 + sr / nh) * heads + h0 + sr % nh * hstep) * spans + span) * (vdim + 2);
        rec[0] = -INFINITY, rec[1] = 0.0f;
      }
      return;
    }
  }
  // The page numbers of the block's keys, looked up once (a block walks 256 keys at most where spans are used as they are meant;
  // longer walks look them up key by key).
  const int slice0 = k_begin / page, slice_n = (min(k_end, last) / page) - slice0 + 1;
  const bool staged = slice_n <= kTableSlice;
  if (staged) {
    for (int i = tid; i < slice_n; i += kMmaWarps * 32) table_slice[i] = bt[slice0 + i];
    __syncthreads();
  }
  // the queries' rows (a block with keys to walk only)
  for (int c = tid; c < q_rows * dparts; c += kMmaWarps * 32) {
    const int sr = c / dparts, part = c - sr * dparts;
    const bool valid = sr < nq;
    const __nv_bfloat16* src = valid ? q + static_cast<size_t>(row0 + sr / nh) * q_stride + (h0 + sr % nh * hstep) * dim + part * 8 : q;
    bw::copy16_async(bw::smem_addr(qs + sr * kst + part * 8), src, valid);
  }
  bw::copies_commit();
  // The threads are laid over a tile's 16-byte parts as (key, part) with the parts rounded up to a
  // power of two, so that every thread keeps its part and steps through the keys.
  int pk = 1, pv = 1;
  while (pk < dparts) pk <<= 1;
  while (pv < vparts) pv <<= 1;
  const int part_k = tid & (pk - 1), kk0_k = tid / pk, kstep_k = max(1, kMmaWarps * 32 / pk);
  const int part_v = tid & (pv - 1), kk0_v = tid / pv, kstep_v = max(1, kMmaWarps * 32 / pv);
  const int page_shift = (page & (page - 1)) == 0 ? 31 - __clz(page) : -1;
  auto request_tile = [&](int k0, int buf) {
    __nv_bfloat16* kd = ks_all + buf * kMmaKeys * kst;
    __nv_bfloat16* vd = vs_all + buf * kMmaKeys * vst;
    // a thread copies one 16-byte part of the keys kk0, kk0 + kstep, ...: its part and first key are fixed
    for (int kk = kk0_k; kk < kMmaKeys; kk += kstep_k) {
      const int kp = k0 + kk;
      const bool have = kp <= last && (kp >= first || kp < keep) && part_k < dparts;
      const __nv_bfloat16* src = kcache;
      if (have) {
        const int blk = page_shift >= 0 ? kp >> page_shift : kp / page, slot = kp - blk * page;
        src = kcache + ((static_cast<size_t>(staged ? table_slice[blk - slice0] : bt[blk]) * kv_heads + g) * page + slot) * dim + part_k * 8;
      }
      if (part_k < dparts) bw::copy16_async(bw::smem_addr(kd + kk * kst + part_k * 8), src, have);
    }
    if (vcache) {
      for (int kk = kk0_v; kk < kMmaKeys; kk += kstep_v) {
        const int kp = k0 + kk;
        const bool have = kp <= last && (kp >= first || kp < keep) && part_v < vparts;
        const __nv_bfloat16* src = vcache;
        if (have) {
          const int blk = page_shift >= 0 ? kp >> page_shift : kp / page, slot = kp - blk * page;
          src = vcache + ((static_cast<size_t>(staged ? table_slice[blk - slice0] : bt[blk]) * v_heads + gv) * page + slot) * vdim + part_v * 8;
        }
        if (part_v < vparts) bw::copy16_async(bw::smem_addr(vd + kk * vst + part_v * 8), src, have);
      }
    }
  };
  // the first tiles; every step commits one group of copies, so that waiting for all but the youngest bufs - 1 groups means
  // that the step's tile is there
  int k_req = k_begin, b_req = 0;
  for (int i = 0; i < bufs - 1; ++i) {
    if (k_req <= k_end) request_tile(k_req, b_req), k_req = skip_gap(k_req + kMmaKeys, keep_end, win_begin), ++b_req;
    bw::copies_commit();
  }
  for (int k0 = k_begin, buf = 0; k0 <= k_end; k0 = skip_gap(k0 + kMmaKeys, keep_end, win_begin), buf = (buf + 1) & (bufs - 1)) {
    // the next tiles are requested while this one is used; the buffer that the youngest takes was released by the
    // barrier at the end of the step before
    if (k_req <= k_end) {
      request_tile(k_req, b_req & (bufs - 1));
      k_req = skip_gap(k_req + kMmaKeys, keep_end, win_begin), ++b_req;
    }
    bw::copies_commit();
    bw::copies_wait<bufs - 1>();
    __syncthreads();
    const __nv_bfloat16* ks = ks_all + buf * kMmaKeys * kst;
    const __nv_bfloat16* vs = vs_all + buf * kMmaKeys * vst;
    if (warp_has_rows && k0 <= w_hi && (k0 + kMmaKeys > w_lo || k0 < keep)) {
    // scores of 16 queries x 32 keys
    float sc[4][4];
#pragma unroll
    for (int j = 0; j < 4; ++j) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.0f;
    for (int kk = 0; kk < dim; kk += 16) {
      uint32_t a[4], b[4];
      bw::ldsm4(a, bw::smem_addr(qs + (wr + (lane & 7) + ((lane >> 3) & 1) * 8) * kst + kk + (lane >> 4) * 8));
#pragma unroll
      for (int jp = 0; jp < 2; ++jp) {  // 16 keys at a time
        bw::ldsm4(b, bw::smem_addr(ks + (jp * 16 + (lane >> 4) * 8 + (lane & 7)) * kst + kk + ((lane >> 3) & 1) * 8));
        bw::mma16816(sc[2 * jp], a, b[0], b[1]);
        bw::mma16816(sc[2 * jp + 1], a, b[2], b[3]);
      }
    }
    // a tile that every query of the warp sees whole needs no mask
    const bool whole = warp_full && k0 + kMmaKeys - 1 <= w_seen_to && (k0 >= w_seen_from || k0 + kMmaKeys <= keep);
    const int kp0 = k0 + 2 * (lane & 3);
    float al[2] = {1.0f, 1.0f};
    if (!SINGLE || nq > 8) {
      weigh_tile<2>(sc, sa, qw, kp0, whole, al);
    } else {  // (a block of at most 8 queries has none in the fragments' second halves)
      weigh_tile<1>(sc, sa, qw, kp0, whole, al);
#pragma unroll
      for (int i = 0; i < 8; ++i) sc[i >> 1][2 + (i & 1)] = 0.0f;
    }
    // (a maximum that stayed gives the factor exp(0) = 1 exactly: nothing to rescale then)
    if (__any_sync(0xffffffffu, al[0] != 1.0f || al[1] != 1.0f)) {
#pragma unroll
      for (int j = 0; j < VT; ++j) {
        acc[j][0] = __fmul_rn(acc[j][0], al[0]), acc[j][1] = __fmul_rn(acc[j][1], al[0]);
        acc[j][2] = __fmul_rn(acc[j][2], al[1]), acc[j][3] = __fmul_rn(acc[j][3], al[1]);
      }
    }
    // weighted values: 16 keys at a time, the weights as hi + lo
#pragma unroll
    for (int kb = 0; kb < 2; ++kb) {
      uint32_t hi[4], lw[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float x0 = sc[2 * kb + (i >> 1)][(i & 1) * 2], x1 = sc[2 * kb + (i >> 1)][(i & 1) * 2 + 1];
        const __nv_bfloat16 h0b = __float2bfloat16_rn(x0), h1b = __float2bfloat16_rn(x1);
        hi[i] = bw::pack_bf16(x0, x1);
        lw[i] = bw::pack_bf16(__fsub_rn(x0, __bfloat162float(h0b)), __fsub_rn(x1, __bfloat162float(h1b)));
      }
#pragma unroll
      for (int jp = 0; jp < VD16; ++jp) {  // 16 value columns at a time
        if (SINGLE && (jp & 3) != warp) continue;
        uint32_t b[4];
        bw::ldsm4_trans(b, bw::smem_addr(vs + (kb * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * vst + jp * 16 + (lane >> 4) * 8));
        bw::mma16816(acc[2 * jp], hi, b[0], b[1]);
        bw::mma16816(acc[2 * jp], lw, b[0], b[1]);
        bw::mma16816(acc[2 * jp + 1], hi, b[2], b[3]);
        bw::mma16816(acc[2 * jp + 1], lw, b[2], b[3]);
      }
    }
    }
    __syncthreads();  // every warp has used the tile: its buffer may be filled again
  }
  bw::copies_wait<0>();  // (a block without a key tile has not waited for its queries' copies yet)
  const float m_a = qw[0].m, m_b = qw[1].m;
  float l_a = qw[0].l, l_b = qw[1].l;
  l_a = __fadd_rn(l_a, __shfl_xor_sync(0xffffffffu, l_a, 1)), l_a = __fadd_rn(l_a, __shfl_xor_sync(0xffffffffu, l_a, 2));
  l_b = __fadd_rn(l_b, __shfl_xor_sync(0xffffffffu, l_b, 1)), l_b = __fadd_rn(l_b, __shfl_xor_sync(0xffffffffu, l_b, 2));
  if (span_tiles > 0) {
    // the span's record per query: maximum, sum, weighted values relative to that maximum
    const int colp = 2 * (lane & 3);
    if (ok_a) {
      float* rec = partial + ((static_cast<size_t>(row0 + sr_a / nh) * heads + h0 + sr_a % nh * hstep) * spans + span) * (vdim + 2);
      if ((lane & 3) == 0 && (warp == 0 || !SINGLE)) rec[0] = m_a, rec[1] = l_a;
#pragma unroll
      for (int j = 0; j < VT; ++j)
        if (!SINGLE || ((j >> 1) & 3) == warp) rec[2 + j * 8 + colp] = acc[j][0], rec[2 + j * 8 + colp + 1] = acc[j][1];
    }
    if (ok_b) {
      float* rec = partial + ((static_cast<size_t>(row0 + sr_b / nh) * heads + h0 + sr_b % nh * hstep) * spans + span) * (vdim + 2);
      if ((lane & 3) == 0 && (warp == 0 || !SINGLE)) rec[0] = m_b, rec[1] = l_b;
#pragma unroll
      for (int j = 0; j < VT; ++j)
        if (!SINGLE || ((j >> 1) & 3) == warp) rec[2 + j * 8 + colp] = acc[j][2], rec[2 + j * 8 + colp + 1] = acc[j][3];
    }
    return;
  }
  if (sa.sink) {  // the extra key (score 0 unless the head has a number of its own)
    const float sk_a = sa.sinks && ok_a ? sa.sinks[h0 + sr_a % nh * hstep] : 0.0f, sk_b = sa.sinks && ok_b ? sa.sinks[h0 + sr_b % nh * hstep] : 0.0f;
    l_a = __fadd_rn(l_a, expf(__fsub_rn(sk_a, m_a))), l_b = __fadd_rn(l_b, expf(__fsub_rn(sk_b, m_b)));
  }
  const float inv_a = __fdiv_rn(1.0f, l_a), inv_b = __fdiv_rn(1.0f, l_b);
  const int col = 2 * (lane & 3);
  if (ok_a) {
    __nv_bfloat16* dst = out + static_cast<size_t>(row0 + sr_a / nh) * o_stride + (h0 + sr_a % nh * hstep) * vdim + col;
#pragma unroll
    for (int j = 0; j < VT; ++j)
      if (!SINGLE || ((j >> 1) & 3) == warp)
        *reinterpret_cast<__nv_bfloat162*>(dst + j * 8) = __floats2bfloat162_rn(__fmul_rn(acc[j][0], inv_a), __fmul_rn(acc[j][1], inv_a));
  }
  if (ok_b) {
    __nv_bfloat16* dst = out + static_cast<size_t>(row0 + sr_b / nh) * o_stride + (h0 + sr_b % nh * hstep) * vdim + col;
#pragma unroll
    for (int j = 0; j < VT; ++j)
      if (!SINGLE || ((j >> 1) & 3) == warp)
        *reinterpret_cast<__nv_bfloat162*>(dst + j * 8) = __floats2bfloat162_rn(__fmul_rn(acc[j][2], inv_b), __fmul_rn(acc[j][3], inv_b));
  }
}

// The spans' records of a query joined in ascending order of the spans: a warp per query.
__global__ void __launch_bounds__(128)
scored_attention_merge_kernel(const float* __restrict__ partial, __nv_bfloat16* out, int o_stride, int queries, int heads,
                              int vdim, int spans, int sink, const float* __restrict__ sinks) {
  bw::pdl_enter();
  const int qi = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (qi >= queries) return;
  float m, l, acc[8];
  merge_spans(partial + static_cast<size_t>(qi) * spans * (vdim + 2), spans, vdim, lane, m, l, acc);
  if (sink) l = __fadd_rn(l, expf(__fsub_rn(sinks ? sinks[qi % heads] : 0.0f, m)));
  const float inv = __fdiv_rn(1.0f, l);
  __nv_bfloat16* dst = out + static_cast<size_t>(qi / heads) * o_stride + (qi % heads) * vdim;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int d = i * 32 + lane;
    if (d < vdim) dst[d] = __float2bfloat16_rn(__fmul_rn(acc[i], inv));
  }
}

template <int VD16, bool SINGLE>
int launch_scored_mma(dim3 grid, size_t smem, cudaStream_t stream, const __nv_bfloat16* q, int q_stride,
                      const __nv_bfloat16* kcache, const __nv_bfloat16* vcache, const int* block_table, int max_blocks,
                      const int* tile_seq, const int* tile_row0, const int* tile_rows, const int* seq_pos0,
                      const int* seq_row0, __nv_bfloat16* out, int o_stride, int heads, int kv_heads, int hb, int dim,
                      int page, const ScoreArgs& sa, int span_tiles, int spans, float* partial) {
  static size_t allowed = 48 * 1024;
  if (smem > allowed) {
    cudaError_t e = cudaFuncSetAttribute(scored_attention_mma_kernel<VD16, SINGLE>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         static_cast<int>(smem));
    if (e != cudaSuccess) {
      bw::set_error("scored_attention: %zu bytes of shared memory: %s", smem, cudaGetErrorString(e));
      return static_cast<int>(e);
    }
    allowed = smem;
  }
  bw::launch_pdl(scored_attention_mma_kernel<VD16, SINGLE>, grid, dim3(kMmaWarps * 32), smem, stream, q, q_stride, kcache, vcache,
                 block_table, max_blocks, tile_seq, tile_row0, tile_rows, seq_pos0, seq_row0, out, o_stride, heads, kv_heads,
                 hb, dim, page, sa, span_tiles, spans, partial);
  return bw::launch_status();
}

bool g_force_plain = false;
constexpr int kSpanTiles = 8;  // key tiles per span: 256 keys, whatever the step
#endif  // BW_ACT_BF16

}  // namespace

// Rows of one sequence per query tile for `group` query heads on a key/value head.
BW_API int BW_FN(scored_attention_tile_rows)(int group) {
  const int hb = group < kWarps * kQW ? group : kWarps * kQW;
  return (kWarps * kQW) / (hb > 0 ? hb : 1);
}

BW_API int BW_FN(qkv_prepare)(const float* u, int cols, const float* conv_w, const float* conv_wt, int taps,
                              const float* conv_state,
                              const float* q_norm, const float* k_norm, float eps, const float* cos_t, const float* sin_t,
                              int pairs, const int* pos, const int* row_seq, const int* seq_row0, const int* seq_pos0,
                              const int* seq_slot, const int* block_table, int max_blocks, void* kcache, void* vcache,
                              void* q_out, int n, int heads, int kv_heads, int dim, int vdim, int page,
                              const float* bias, const float* vmix_src, const float* vmix_lambda, float* v_keep,
                              int u_stride, int half_layout, int v_heads, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (u_stride < cols) {
    bw::set_error("qkv_prepare: rows %d floats apart do not hold %d columns", u_stride, cols);
    return -1;
  }
  if (dim > kMaxE * 32 || vdim > kMaxE * 32) {
    bw::set_error("qkv_prepare: head sizes %d / %d (up to %d)", dim, vdim, kMaxE * 32);
    return -1;
  }
  if (conv_w && taps > 1 && !conv_state) {
    bw::set_error("qkv_prepare: a convolution of %d taps needs the requests' state", taps);
    return -1;
  }
  PrepArgs a;
  a.bias = bias, a.vmix_src = vmix_src, a.vmix_lambda = vmix_lambda, a.v_keep = v_keep;
  a.u = u, a.cols = cols, a.u_stride = u_stride, a.conv_w = conv_w, a.conv_wt = conv_w ? conv_wt : nullptr, a.taps = taps;
  a.conv_state = taps > 1 ? conv_state : nullptr;
  a.q_norm = q_norm, a.k_norm = k_norm, a.eps = eps, a.cos_t = cos_t, a.sin_t = sin_t, a.pairs = cos_t ? pairs : 0;
  a.half_layout = half_layout;
  a.pos = pos, a.row_seq = row_seq, a.seq_row0 = seq_row0, a.seq_pos0 = seq_pos0, a.seq_slot = seq_slot;
  a.block_table = block_table, a.max_blocks = max_blocks;
  a.kcache = static_cast<act_t*>(kcache), a.vcache = static_cast<act_t*>(vcache), a.q_out = static_cast<act_t*>(q_out);
  a.heads = heads, a.kv_heads = kv_heads, a.v_heads = vcache ? v_heads : 0, a.dim = dim, a.vdim = vdim, a.page = page;
  const int total = heads + kv_heads + a.v_heads;
  // four entries per lane where every head and row starts on 16 bytes (and the taps came transposed)
  const bool by_four = dim % 4 == 0 && vdim % 4 == 0 && cols % 4 == 0 && u_stride % 4 == 0 && (!conv_w || conv_wt) &&
                       ((reinterpret_cast<uintptr_t>(u) | reinterpret_cast<uintptr_t>(conv_state) |
                         reinterpret_cast<uintptr_t>(conv_wt) | reinterpret_cast<uintptr_t>(q_norm) |
                         reinterpret_cast<uintptr_t>(k_norm) | reinterpret_cast<uintptr_t>(bias) |
                         reinterpret_cast<uintptr_t>(vmix_src) | reinterpret_cast<uintptr_t>(v_keep)) & 15) == 0;
  // (with many rows a warp takes three heads one after the other: what it looks up about the row serves them all)
  const int per_block = kPrepWarps * (n >= 256 ? 3 : 1);
  const dim3 grid(n, (total + per_block - 1) / per_block);
  if (by_four)
    bw::launch_pdl(qkv_prepare_vec_kernel, grid, dim3(kPrepWarps * 32), 0, stream, a);
  else
    bw::launch_pdl(qkv_prepare_kernel, grid, dim3(kPrepWarps * 32), 0, stream, a);
  return bw::launch_status();
}

// u_stride: floats between two rows of u (at least cols).
BW_API int BW_FN(conv_state_update)(const float* u, int cols, float* state, int taps, const int* tile_seq,
                                    const int* tile_row0, const int* tile_rows, int tiles, const int* seq_pos0,
                                    const int* seq_slot, int u_stride, cudaStream_t stream) {
  if (tiles <= 0 || taps <= 1) return 0;
  if (u_stride < cols) {
    bw::set_error("conv_state_update: rows %d floats apart do not hold %d columns", u_stride, cols);
    return -1;
  }
  if (taps - 1 > kMaxTaps) {
    bw::set_error("conv_state_update: %d taps (up to %d)", taps, kMaxTaps + 1);
    return -1;
  }
  bw::launch_pdl(conv_state_update_kernel, dim3(tiles, (cols + 127) / 128), dim3(128), 0, stream, u, u_stride, cols, state, taps,
                 tile_seq, tile_row0, tile_rows, seq_pos0, seq_slot);
  return bw::launch_status();
}

BW_API int BW_FN(scored_attention)(const void* q, int q_stride, const void* kcache, const void* vcache,
                                   const int* block_table, int max_blocks, const int* tile_seq, const int* tile_row0,
                                   const int* tile_rows, int tiles, const int* seq_pos0, const int* seq_row0, void* out,
                                   int o_stride, int heads, int kv_heads, int dim, int vdim, int page, float scale,
                                   float softcap, int sink, const float* slopes, int window, const float* dist_a,
                                   const float* dist_b, const float* sinks, int keep_first, int chunk, int maps,
                                   float* partial, cudaStream_t stream) {
  // maps > 1: kv_heads key heads, of which `maps` neighbours share a value head. partial: [n, heads, vdim + 2] records for
  // scored_difference instead of `out`.
  if (tiles <= 0) return 0;
  if (kv_heads <= 0 || heads % kv_heads || maps <= 0 || kv_heads % maps || (maps > 1 && !vcache)) {
    bw::set_error("scored_attention: %d heads on %d key/value heads, %d maps", heads, kv_heads, maps);
    return -1;
  }
  const int acc = (vdim + 31) / 32;
  if (acc > 8) {
    bw::set_error("scored_attention: value size %d (up to 256)", vdim);
    return -1;
  }
  const int rep = heads / kv_heads;
  const int hb = rep < kWarps * kQW ? rep : kWarps * kQW;
  const size_t smem = (static_cast<size_t>(kKeys) * (dim + 1) + (vcache ? static_cast<size_t>(kKeys) * vdim : 0) +
                       static_cast<size_t>(kWarps * kQW) * dim) * sizeof(float);
  if (smem > 200 * 1024) {
    bw::set_error("scored_attention: head sizes %d / %d need %zu bytes of shared memory", dim, vdim, smem);
    return -1;
  }
  ScoreArgs sa;
  sa.scale = scale, sa.softcap = softcap, sa.sink = sink, sa.slopes = slopes, sa.window = window;
  sa.dist_a = dist_a, sa.dist_b = dist_a ? dist_b : nullptr, sa.sinks = sinks, sa.keep_first = window > 0 ? keep_first : 0;
  sa.chunk = chunk, sa.maps = maps;
  sa.cap_exp = 0.0f;  // (the tensor-core kernel's)
  const dim3 grid(tiles, kv_heads, (rep + hb - 1) / hb);
#define BW_SCORED(A)                                                                                                      \
  case A:                                                                                                                 \
    return launch_scored<A>(grid, smem, stream, static_cast<const act_t*>(q), q_stride, static_cast<const act_t*>(kcache), \
                            static_cast<const act_t*>(vcache), block_table, max_blocks, tile_seq, tile_row0, tile_rows,   \
                            seq_pos0, seq_row0, static_cast<act_t*>(out), o_stride, heads, kv_heads, hb, dim, vdim, page, \
                            sa, partial);
  switch (acc) {
    BW_SCORED(1) BW_SCORED(2) BW_SCORED(3) BW_SCORED(4) BW_SCORED(5) BW_SCORED(6) BW_SCORED(7) BW_SCORED(8)
  }
#undef BW_SCORED
  return -1;
}

#if BW_ACT_BF16
// Tests: keep attention on the CUDA-core kernel also where the tensor-core kernel takes the shape.
BW_API int bw_bf16_scored_attention_force_plain(int on) {
  g_force_plain = on != 0;
  return 0;
}

// Rows of one sequence per query tile of the tensor-core kernel, 0 where it does not take the
// shape: key size a multiple of 16, value size 16 .. 128 in steps of 16, or 256.
BW_API int bw_bf16_scored_attention_mma_tile_rows(int group, int dim, int vdim) {
  if (g_force_plain || dim % 16 || vdim % 16 || dim > 256 || !(vdim <= 128 || vdim == 256)) return 0;
  const int hb = group < kMmaRows ? group : kMmaRows;
  return kMmaRows / (hb > 0 ? hb : 1);
}

BW_API int bw_bf16_scored_attention_mma(const void* q, int q_stride, const void* kcache, const void* vcache,
                                        const int* block_table, int max_blocks, const int* tile_seq, const int* tile_row0,
                                        const int* tile_rows, int tiles, const int* seq_pos0, const int* seq_row0, void* out,
                                        int o_stride, int heads, int kv_heads, int dim, int vdim, int page, float scale,
                                        float softcap, int sink, const float* slopes, int window, int n, int spans,
                                        float* partial, const float* dist_a, const float* dist_b, const float* sinks,
                                        int keep_first, int chunk, int maps, cudaStream_t stream) {
  // maps > 1 (maps as for scored_attention): the spans' records (one span at least) stay in `partial` for scored_difference.
  // spans > 1 (`partial` holding n * heads * spans * (vdim + 2) floats): every query's keys are spread
  // over blocks of kSpanTiles key tiles each, at fixed absolute positions, and a second kernel joins
  // the spans' records in ascending order.
  if (tiles <= 0) return 0;
  if (kv_heads <= 0 || heads % kv_heads || maps <= 0 || kv_heads % maps || (maps > 1 && (!vcache || !partial)) ||
      !bw_bf16_scored_attention_mma_tile_rows(heads / kv_heads, dim, vdim)) {
    bw::set_error("scored_attention (tensor cores): %d heads on %d, %d maps, sizes %d / %d", heads, kv_heads, maps, dim, vdim);
    return -1;
  }
  const int rep = heads / kv_heads;
  const int hb = rep < kMmaRows ? rep : kMmaRows;
  const bool single = tiles == n && hb <= 16;
  const int q_rows = mma_q_rows(single), bufs = mma_bufs(single);
  const size_t smem = (static_cast<size_t>(q_rows + bufs * kMmaKeys) * (dim + 8) +
                       (vcache ? static_cast<size_t>(bufs * kMmaKeys) * (vdim + 8) : 0)) * sizeof(__nv_bfloat16);
  ScoreArgs sa;
  sa.scale = scale, sa.softcap = softcap, sa.sink = sink, sa.slopes = slopes, sa.window = window;
  sa.dist_a = dist_a, sa.dist_b = dist_a ? dist_b : nullptr, sa.sinks = sinks, sa.keep_first = window > 0 ? keep_first : 0;
  sa.chunk = chunk, sa.maps = maps;
  sa.cap_exp = softcap > 0.0f ? 2.0f * scale / softcap * 1.4426950408889634f : 0.0f;
  const bool split = (spans > 1 || maps > 1) && partial != nullptr;
  if (!split) spans = 1;
  const dim3 grid(tiles, kv_heads, (rep + hb - 1) / hb * spans);
  typedef const __nv_bfloat16* in_t;
  int rc = -1;
#define BW_SCORED_MMA_AS(V, S)                                                                                             \
  launch_scored_mma<V, S>(grid, smem, stream, static_cast<in_t>(q), q_stride, static_cast<in_t>(kcache),                   \
                          static_cast<in_t>(vcache), block_table, max_blocks, tile_seq, tile_row0, tile_rows, seq_pos0,     \
                          seq_row0, static_cast<__nv_bfloat16*>(out), o_stride, heads, kv_heads, hb, dim, page, sa,         \
                          split ? kSpanTiles : 0, spans, partial)
#define BW_SCORED_MMA(V)                                                                                                   \
  case V:                                                                                                                  \
    rc = single ? BW_SCORED_MMA_AS(V, true) : BW_SCORED_MMA_AS(V, false);                                                  \
    break;
  switch (vdim / 16) {
    BW_SCORED_MMA(1) BW_SCORED_MMA(2) BW_SCORED_MMA(3) BW_SCORED_MMA(4) BW_SCORED_MMA(5) BW_SCORED_MMA(6) BW_SCORED_MMA(7)
    BW_SCORED_MMA(8) BW_SCORED_MMA(16)
  }
#undef BW_SCORED_MMA
#undef BW_SCORED_MMA_AS
  if (rc != 0 || !split || maps > 1) return rc;
  bw::launch_pdl(scored_attention_merge_kernel, dim3((n * heads + 3) / 4), dim3(128), 0, stream,
                 static_cast<const float*>(partial), static_cast<__nv_bfloat16*>(out), o_stride, n * heads, heads, vdim, spans, sink, sinks);
  return bw::launch_status();
}

// Spans that the queries of a step with contexts of up to max_keys keys are spread over. `reach` > 0: a query sees at
// most that many keys, itself the last; query tiles hold `tile_rows` rows. (A tile then spans reach + tile_rows - 1 keys, which
// touch at most one span more than they would fill.)
BW_API int bw_bf16_scored_attention_spans(int max_keys, int reach, int tile_rows) {
  const int per = kSpanTiles * kMmaKeys;
  const int all = (max_keys + per - 1) / per;
  if (reach <= 0) return all;
  const long long keys = static_cast<long long>(reach) + tile_rows - 1;
  const long long near = (keys + per - 2) / per + 1;
  return near < all ? static_cast<int>(near) : all;
}
#endif  // BW_ACT_BF16

// Two maps per head become one output (see scored_difference_kernel). partial: [n, 2 * heads, spans, vdim + 2] records of
// scored_attention; gate: float32 rows of `gate_stride` floats with heads * vdim / gate_group numbers each, or null.
BW_API int BW_FN(scored_difference)(const float* partial, int spans, const float* lambda, float keep, float eps,
                                    const float* gate, int gate_stride, int gate_group, void* out, int n, int heads, int vdim,
                                    cudaStream_t stream) {
  if (n <= 0) return 0;
  if (spans <= 0 || heads <= 0 || vdim <= 0 || vdim > 256 || gate_group <= 0) {
    bw::set_error("scored_difference: %d spans, %d heads of %d (up to 256)", spans, heads, vdim);
    return -1;
  }
  DifferenceArgs a;
  a.partial = partial, a.spans = spans, a.queries = n * heads, a.heads = heads, a.vdim = vdim, a.lambda = lambda;
  a.keep = keep, a.eps = eps, a.gate = gate, a.gate_stride = gate_stride, a.gate_group = gate_group;
  a.out = static_cast<act_t*>(out);
  bw::launch_pdl(scored_difference_kernel, dim3((a.queries + 1) / 2), dim3(128), 0, stream, a);
  return bw::launch_status();
}
