// Row kernels that look at a row's neighbours in its own sequence, and the layer norm:
//
//   sb_embed_pair:      embedding row plus a row of a second table chosen by a hash of the
//                       previous and the current token (the previous token of a step's first
//                       row comes from per-slot state)
//   sb_keep_last_token: a step's last token of every sequence into that state
//   sb_layernorm:       (x - mean) / sqrt(var + eps) * w [+ b]
//   sb_causal_conv:     a short causal convolution over time on every channel, reading the
//                       taps before a step's first row from per-slot state
//   sb_conv_heads:      the same convolution over a fused q|k|v projection, its results going straight to
//                       the query rows and the cache pages
//
// All arithmetic is float32; sums over a row are fixed trees.
#include <math.h>

#include "common.cuh"

namespace {

template <int NT>
__device__ __forceinline__ float block_sum(float s, float* red) {
  s = sb_warp_sum(s);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  __syncthreads();
  if (lane == 0) red[warp] = s;
  __syncthreads();
  if (threadIdx.x == 0) {
    float total = 0.0f;
    for (int i = 0; i < NT / 32; ++i) total += red[i];
    red[NT / 32] = total;
  }
  __syncthreads();
  return red[NT / 32];
}

template <typename T>
__global__ void embed_pair_kernel(const int32_t* tokens, const int32_t* row_seq, const int32_t* row_pos,
                                  const int32_t* seq_row0, const int32_t* seq_slot, const int32_t* prev_token,
                                  const T* __restrict__ table, int vocab, const T* __restrict__ pair, int buckets,
                                  int mul_prev, int mul_cur, int width, float scale, float* out) {
  sb_pdl_launch();
  sb_pdl_wait();
  const int r = blockIdx.x;
  const int tok = tokens[r];
  float* o = out + (size_t)r * width;
  if (tok < 0 || tok >= vocab) {
    for (int i = threadIdx.x; i < width; i += blockDim.x) o[i] = NAN;
    return;
  }
  const int s = row_seq[r];
  long long idx = buckets;                       // a sequence's first token: the table's last row
  if (row_pos[r] > 0) {
    const int prev = r > seq_row0[s] ? tokens[r - 1] : prev_token[seq_slot[s]];
    idx = ((long long)prev * mul_prev + (long long)tok * mul_cur) % buckets;
    if (idx < 0) idx += buckets;
  }
  const T* a = table + (size_t)tok * width;
  const T* b = pair + (size_t)idx * width;
  for (int i = threadIdx.x; i < width; i += blockDim.x)
    o[i] = sb_to_f32<T>(a[i]) * scale + sb_to_f32<T>(b[i]);
}

__global__ void keep_last_token_kernel(const int32_t* tokens, const int32_t* seq_row0, const int32_t* seq_slot,
                                       int n_seqs, int32_t* prev_token) {
  sb_pdl_launch();
  sb_pdl_wait();
  const int s = blockIdx.x * blockDim.x + threadIdx.x;
  if (s < n_seqs) prev_token[seq_slot[s]] = tokens[seq_row0[s + 1] - 1];
}

template <int NT, typename TW, typename TO>
__global__ void __launch_bounds__(NT)
layernorm_kernel(const float* x, const int32_t* rows, int width, const TW* __restrict__ w,
                 const TW* __restrict__ b, float eps, TO* out) {
  __shared__ float red[NT / 32 + 1];
  sb_pdl_launch();
  sb_pdl_wait();
  const size_t r = rows ? (size_t)rows[blockIdx.x] : (size_t)blockIdx.x;
  const float* xr = x + r * width;
  float s = 0.0f;
  for (int i = threadIdx.x; i < width; i += NT) s += xr[i];
  const float mean = block_sum<NT>(s, red) / (float)width;
  float q = 0.0f;
  for (int i = threadIdx.x; i < width; i += NT) {
    const float d = xr[i] - mean;
    q = fmaf(d, d, q);
  }
  const float inv = 1.0f / sqrtf(block_sum<NT>(q, red) / (float)width + eps);
  TO* o = out + (size_t)blockIdx.x * width;
  for (int i = threadIdx.x; i < width; i += NT) {
    const float v = ((xr[i] - mean) * inv) * sb_to_f32<TW>(w[i]);
    o[i] = sb_from_f32<TO>(b ? v + sb_to_f32<TW>(b[i]) : v);
  }
}

// y_t = [x_t +] [bias +] sum_j w[c, j] x_(t - taps + 1 + j), optionally through silu.  A tap before
// the step's first row of the sequence is read from state[slot, taps - 1, channels] (the inputs at
// the taps - 1 positions before the step), one before the sequence's start is zero.  OWN: every
// sequence brings exactly one row, and the thread that computes a channel also shifts its state.
template <typename TW, typename TO, bool OWN>
__global__ void causal_conv_kernel(const float* x, int ld, int x_off, int channels, int taps,
                                   const TW* __restrict__ w, const TW* __restrict__ bias, int act, int add_input,
                                   const int32_t* row_seq, const int32_t* row_pos, const int32_t* seq_row0,
                                   const int32_t* seq_pos0, const int32_t* seq_slot, float* state, TO* out,
                                   int ld_out, int out_off) {
  sb_pdl_launch();
  sb_pdl_wait();
  const int r = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= channels) return;
  const int s = row_seq[r], pos = row_pos[r];
  const int pos0 = OWN ? pos : seq_pos0[s], r0 = OWN ? r : seq_row0[s];
  float* st = state ? state + (size_t)seq_slot[s] * (taps - 1) * channels + c : nullptr;
  const float cur = x[(size_t)r * ld + x_off + c];
  float acc = bias ? sb_to_f32<TW>(bias[c]) : 0.0f;
  for (int j = 0; j < taps; ++j) {
    const int p = pos - (taps - 1) + j;
    float v = 0.0f;
    if (p >= pos0) v = x[(size_t)(r0 + (p - pos0)) * ld + x_off + c];
    else if (p >= 0) v = st[(size_t)(p - pos0 + taps - 1) * channels];
    acc = fmaf(sb_to_f32<TW>(w[(size_t)c * taps + j]), v, acc);
  }
  if (add_input) acc += cur;
  if (act) acc = sb_silu(acc);
  out[(size_t)r * ld_out + out_off + c] = sb_from_f32<TO>(acc);
  if (OWN) {
    for (int i = 0; i + 1 < taps - 1; ++i) st[(size_t)i * channels] = st[(size_t)(i + 1) * channels];
    if (taps > 1) st[(size_t)(taps - 2) * channels] = cur;
  }
}

// The same sums for a step with several rows a sequence and at most CONV_MAXT taps: a thread walks
// CONV_RUN consecutive rows of its channel and keeps the last taps - 1 inputs in registers, so a row
// is read once instead of once per tap.  Every sum has the order of the kernel above.
constexpr int CONV_MAXT = 8, CONV_RUN = 8;
constexpr int CONV_HEADS_TAPS = 5;      // most taps of sb_conv_heads
template <typename TW, typename TO>
__global__ void causal_conv_run_kernel(const float* x, int n_rows, int ld, int x_off, int channels, int taps,
                                       const TW* __restrict__ w, const TW* __restrict__ bias, int act, int add_input,
                                       const int32_t* row_seq, const int32_t* row_pos, const int32_t* seq_pos0,
                                       const int32_t* seq_slot, const float* state, TO* out, int ld_out, int out_off) {
  sb_pdl_launch();
  sb_pdl_wait();
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= channels) return;
  const int r_begin = blockIdx.x * CONV_RUN, r_end = min(n_rows, r_begin + CONV_RUN);
  float wd[CONV_MAXT], hist[CONV_MAXT];     // by distance d: the weight of x_(t - d); hist[d] = x of the row d before
#pragma unroll
  for (int d = 0; d < CONV_MAXT; ++d) {
    wd[d] = d < taps ? sb_to_f32<TW>(w[(size_t)c * taps + (taps - 1 - d)]) : 0.0f;
    hist[d] = (d >= 1 && d < taps && r_begin - d >= 0) ? x[(size_t)(r_begin - d) * ld + x_off + c] : 0.0f;
  }
  const float b = bias ? sb_to_f32<TW>(bias[c]) : 0.0f;
  for (int r = r_begin; r < r_end; ++r) {
    const int s = row_seq[r], pos = row_pos[r], pos0 = seq_pos0[s];
    const float* st = state ? state + (size_t)seq_slot[s] * (taps - 1) * channels + c : nullptr;
    const float cur = x[(size_t)r * ld + x_off + c];
    hist[0] = cur;
    float acc = b;
#pragma unroll
    for (int d = CONV_MAXT - 1; d >= 0; --d) {
      if (d < taps) {
        const int p = pos - d;
        float v = 0.0f;
        if (p >= pos0) v = hist[d];
        else if (p >= 0) v = st[(size_t)(p - pos0 + taps - 1) * channels];
        acc = fmaf(wd[d], v, acc);
      }
    }
    if (add_input) acc += cur;
    if (act) acc = sb_silu(acc);
    out[(size_t)r * ld_out + out_off + c] = sb_from_f32<TO>(acc);
#pragma unroll
    for (int d = CONV_MAXT - 1; d >= 1; --d) hist[d] = hist[d - 1];
  }
}

// The convolution of a fused projection row [q heads x dim | k heads x dim | v heads x vdim] whose
// results are attention's operands: query channels go to q_out [row][head][hd], key and value channels
// to the position's cache row (key plane, value plane), both padded with zeros to hd.  A thread takes V
// neighbouring channels of one head and CONV_RUN consecutive rows (one row with OWN: every sequence
// brings one, and the thread shifts its channels' state).  The sums are those of the kernels above.
struct HeadsArgs {
  const float* proj;
  int n_rows, ld;
  int hq, hkv, dim, vdim, hd;          // channels: hq * dim, hkv * dim, hkv * vdim
  const void* w;                       // [channels, taps]
  const int32_t* row_seq;
  const int32_t* row_pos;
  const int32_t* seq_pos0;
  const int32_t* seq_slot;
  const int32_t* page_off;
  const int32_t* page_ids;
  int page_size;
  float* state;                        // [slot, taps - 1, channels] or null (one tap)
  void* cache;
  void* q_out;
};

template <int V, typename T>
__device__ __forceinline__ void put_lanes(T* p, const float (&v)[V]) {
  if constexpr (V == 4 && sizeof(T) == 2) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 u;
    u.x = *reinterpret_cast<uint32_t*>(&a);
    u.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = u;
  } else if constexpr (V == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  } else {
    p[0] = sb_from_f32<T>(v[0]);
  }
}
template <int V>
__device__ __forceinline__ void get_lanes(const float* p, float (&v)[V]) {
  if constexpr (V == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  } else {
    v[0] = p[0];
  }
}

template <int TAPS, int V, typename TW, typename T, bool OWN>
__global__ void __launch_bounds__(128) conv_heads_kernel(const HeadsArgs p) {
  sb_pdl_launch();
  const int qw = p.hq * p.dim, kw = p.hkv * p.dim, vw = p.hkv * p.vdim, channels = qw + kw + vw;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (c >= channels) return;
  const int part = c < qw ? 0 : (c < qw + kw ? 1 : 2);
  const int local = part == 0 ? c : (part == 1 ? c - qw : c - qw - kw);
  const int size = part == 2 ? p.vdim : p.dim, head = local / size, d = local % size;
  float wd[TAPS][V];                   // by distance: the weight of the input `i` rows before
#pragma unroll
  for (int i = 0; i < TAPS; ++i)
#pragma unroll
    for (int j = 0; j < V; ++j) wd[i][j] = sb_to_f32<TW>(((const TW*)p.w)[(size_t)(c + j) * TAPS + (TAPS - 1 - i)]);
  sb_pdl_wait();
  const int r_begin = blockIdx.x * (OWN ? 1 : CONV_RUN), r_end = OWN ? r_begin + 1 : min(p.n_rows, r_begin + CONV_RUN);
  float hist[TAPS][V];
  if (!OWN) {
#pragma unroll
    for (int i = 1; i < TAPS; ++i) {
      if (r_begin - i >= 0) {
        get_lanes<V>(p.proj + (size_t)(r_begin - i) * p.ld + c, hist[i]);
      } else {
#pragma unroll
        for (int j = 0; j < V; ++j) hist[i][j] = 0.0f;
      }
    }
  }
  for (int r = r_begin; r < r_end; ++r) {
    const int s = p.row_seq[r], pos = p.row_pos[r], pos0 = OWN ? pos : p.seq_pos0[s];
    float* st = p.state ? p.state + (size_t)p.seq_slot[s] * (TAPS - 1) * channels + c : nullptr;
    get_lanes<V>(p.proj + (size_t)r * p.ld + c, hist[0]);
    float acc[V];
#pragma unroll
    for (int j = 0; j < V; ++j) acc[j] = 0.0f;
#pragma unroll
    for (int i = TAPS - 1; i >= 0; --i) {
      const int at = pos - i;                      // before the step's first row: the state; before the start: zero
      float v[V];
      if (at >= pos0) {
#pragma unroll
        for (int j = 0; j < V; ++j) v[j] = hist[i][j];
      } else if (at >= 0) {
        get_lanes<V>(st + (size_t)(at - pos0 + TAPS - 1) * channels, v);
        if (OWN)
#pragma unroll
          for (int j = 0; j < V; ++j) hist[i][j] = v[j];
      } else {
#pragma unroll
        for (int j = 0; j < V; ++j) {
          v[j] = 0.0f;
          if (OWN) hist[i][j] = 0.0f;
        }
      }
#pragma unroll
      for (int j = 0; j < V; ++j) acc[j] = fmaf(wd[i][j], v[j], acc[j]);
    }
    T* dst = nullptr;
    if (part == 0) {
      dst = (T*)p.q_out + ((size_t)r * p.hq + head) * p.hd;
    } else {
      const int first = p.page_off[s], pi = pos / p.page_size;
      const int page = pos >= 0 && pi < p.page_off[s + 1] - first ? p.page_ids[first + pi] : -1;
      if (page >= 0)                               // else no page of its own there: nothing is written
        dst = (T*)p.cache + ((((size_t)page * 2 + (part == 2)) * p.hkv + head) * p.page_size + pos % p.page_size) * p.hd;
    }
    if (dst) {
      put_lanes<V>(dst + d, acc);
      if (d == 0)
        for (int e = size; e < p.hd; ++e) dst[e] = sb_from_f32<T>(0.0f);
    }
    if (OWN) {
      if (TAPS > 1 && st) {
#pragma unroll
        for (int i = 0; i + 1 < TAPS; ++i) put_lanes<V>(st + (size_t)i * channels, hist[TAPS - 2 - i]);   // place i: input TAPS - 2 - i rows back
      }
    } else {
#pragma unroll
      for (int i = TAPS - 1; i >= 1; --i)
#pragma unroll
        for (int j = 0; j < V; ++j) hist[i][j] = hist[i - 1][j];
    }
  }
}

template <int TAPS, typename TW, typename T>
void launch_conv_heads(const HeadsArgs& a, bool own, bool vec, cudaStream_t stream) {
  const int channels = a.hq * a.dim + a.hkv * (a.dim + a.vdim), per = 128 * (vec ? 4 : 1);
  const dim3 grid(own ? a.n_rows : (a.n_rows + CONV_RUN - 1) / CONV_RUN, (channels + per - 1) / per);
  if (own && vec) sb_launch<SB_K_ELEMENTWISE>(conv_heads_kernel<TAPS, 4, TW, T, true>, grid, dim3(128), 0, stream, a);
  else if (own) sb_launch<SB_K_ELEMENTWISE>(conv_heads_kernel<TAPS, 1, TW, T, true>, grid, dim3(128), 0, stream, a);
  else if (vec) sb_launch<SB_K_ELEMENTWISE>(conv_heads_kernel<TAPS, 4, TW, T, false>, grid, dim3(128), 0, stream, a);
  else sb_launch<SB_K_ELEMENTWISE>(conv_heads_kernel<TAPS, 1, TW, T, false>, grid, dim3(128), 0, stream, a);
}

__global__ void conv_state_kernel(const float* x, int ld, int x_off, int channels, int taps,
                                  const int32_t* seq_row0, const int32_t* seq_slot, float* state) {
  sb_pdl_launch();
  sb_pdl_wait();
  const int s = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= channels) return;
  const int r0 = seq_row0[s], n = seq_row0[s + 1] - r0;
  float* st = state + (size_t)seq_slot[s] * (taps - 1) * channels + c;
  for (int i = 0; i < taps - 1; ++i) {
    const int rel = n - (taps - 1) + i;              // the position kept at i, counted from the step's first
    st[(size_t)i * channels] = rel >= 0 ? x[(size_t)(r0 + rel) * ld + x_off + c]
                                        : st[(size_t)(i + n) * channels];      // i + n > i: not yet overwritten
  }
}

}  // namespace

extern "C" int sb_embed_pair(const int32_t* tokens, int n_rows, const int32_t* row_seq, const int32_t* row_pos,
                             const int32_t* seq_row0, const int32_t* seq_slot, const int32_t* prev_token,
                             const void* table, int table_dtype, int vocab, const void* pair, int buckets,
                             int mul_prev, int mul_cur, int width, float scale, float* out, cudaStream_t stream) {
  if (n_rows <= 0 || width <= 0 || vocab <= 0 || buckets <= 0 || !tokens || !table || !pair || !out || !prev_token)
    SB_FAIL(SB_ERR_ARG, "sb_embed_pair: rows=%d width=%d vocab=%d buckets=%d", n_rows, width, vocab, buckets);
  if (!sb_valid_dtype(table_dtype)) SB_FAIL(SB_ERR_ARG, "sb_embed_pair: dtype code %d", table_dtype);
  SB_DISPATCH_DTYPE(table_dtype, T, {
    sb_launch<SB_K_ELEMENTWISE>(embed_pair_kernel<T>, dim3(n_rows), dim3(width >= 1024 ? 256 : 128), 0, stream, tokens,
                                row_seq, row_pos, seq_row0, seq_slot, prev_token, (const T*)table, vocab,
                                (const T*)pair, buckets, mul_prev, mul_cur, width, scale, out);
  });
  SB_CHECK_LAUNCH("sb_embed_pair");
  return SB_OK;
}

extern "C" int sb_keep_last_token(const int32_t* tokens, const int32_t* seq_row0, const int32_t* seq_slot,
                                  int n_seqs, int32_t* prev_token, cudaStream_t stream) {
  if (n_seqs <= 0 || !tokens || !seq_row0 || !seq_slot || !prev_token)
    SB_FAIL(SB_ERR_ARG, "sb_keep_last_token: seqs=%d", n_seqs);
  sb_launch<SB_K_ELEMENTWISE>(keep_last_token_kernel, dim3((n_seqs + 127) / 128), dim3(128), 0, stream, tokens, seq_row0,
                              seq_slot, n_seqs, prev_token);
  SB_CHECK_LAUNCH("sb_keep_last_token");
  return SB_OK;
}

extern "C" int sb_layernorm(const float* x, const int32_t* rows, int n_rows, int width, const void* weight,
                            const void* bias, int weight_dtype, float eps, void* out, int out_dtype, cudaStream_t stream) {
  if (n_rows <= 0 || width <= 0 || !x || !weight || !out) SB_FAIL(SB_ERR_ARG, "sb_layernorm: rows=%d width=%d", n_rows, width);
  if (!sb_valid_dtype(weight_dtype) || !sb_valid_dtype(out_dtype))
    SB_FAIL(SB_ERR_ARG, "sb_layernorm: dtype codes %d %d", weight_dtype, out_dtype);
  SB_DISPATCH_DTYPE(weight_dtype, TW, {
    SB_DISPATCH_DTYPE(out_dtype, TO, {
      if (n_rows >= 512 || width <= 1024)
        sb_launch<SB_K_ELEMENTWISE>(layernorm_kernel<256, TW, TO>, dim3(n_rows), dim3(256), 0, stream, x, rows, width,
                                    (const TW*)weight, (const TW*)bias, eps, (TO*)out);
      else
        sb_launch<SB_K_ELEMENTWISE>(layernorm_kernel<1024, TW, TO>, dim3(n_rows), dim3(1024), 0, stream, x, rows, width,
                                    (const TW*)weight, (const TW*)bias, eps, (TO*)out);
    });
  });
  SB_CHECK_LAUNCH("sb_layernorm");
  return SB_OK;
}

extern "C" int sb_causal_conv(const float* x, int n_rows, int ld, int x_off, int channels, int taps, const void* w,
                              const void* bias, int w_dtype, int act, int add_input, int n_seqs,
                              const int32_t* row_seq, const int32_t* row_pos, const int32_t* seq_row0,
                              const int32_t* seq_pos0, const int32_t* seq_slot, float* state, void* out,
                              int out_dtype, int ld_out, int out_off, cudaStream_t stream) {
  if (n_rows <= 0 || channels <= 0 || taps <= 0 || n_seqs <= 0 || !x || !w || !out || (taps > 1 && !state))
    SB_FAIL(SB_ERR_ARG, "sb_causal_conv: rows=%d channels=%d taps=%d seqs=%d", n_rows, channels, taps, n_seqs);
  if (x_off < 0 || x_off + channels > ld || out_off < 0 || out_off + channels > ld_out)
    SB_FAIL(SB_ERR_ARG, "sb_causal_conv: %d channels at %d of %d, out at %d of %d", channels, x_off, ld, out_off, ld_out);
  if (!sb_valid_dtype(w_dtype) || !sb_valid_dtype(out_dtype))
    SB_FAIL(SB_ERR_ARG, "sb_causal_conv: dtype codes %d %d", w_dtype, out_dtype);
  if ((const void*)x == (const void*)out) SB_FAIL(SB_ERR_ARG, "sb_causal_conv: in place");
  const int nt = channels >= 256 ? 256 : 128;
  const dim3 grid(n_rows, (channels + nt - 1) / nt);
  const bool own = n_rows == n_seqs;        // one row a sequence: the row's threads shift the state themselves
  SB_DISPATCH_DTYPE(w_dtype, TW, {
    SB_DISPATCH_DTYPE(out_dtype, TO, {
      if (!own && taps <= CONV_MAXT)
        sb_launch<SB_K_ELEMENTWISE>(causal_conv_run_kernel<TW, TO>, dim3((n_rows + CONV_RUN - 1) / CONV_RUN, grid.y), dim3(nt),
                                    0, stream, x, n_rows, ld, x_off, channels, taps, (const TW*)w, (const TW*)bias, act,
                                    add_input, row_seq, row_pos, seq_pos0, seq_slot, (const float*)state, (TO*)out, ld_out,
                                    out_off);
      else if (own)
        sb_launch<SB_K_ELEMENTWISE>(causal_conv_kernel<TW, TO, true>, grid, dim3(nt), 0, stream, x, ld, x_off, channels,
                                    taps, (const TW*)w, (const TW*)bias, act, add_input, row_seq, row_pos, seq_row0,
                                    seq_pos0, seq_slot, state, (TO*)out, ld_out, out_off);
      else
        sb_launch<SB_K_ELEMENTWISE>(causal_conv_kernel<TW, TO, false>, grid, dim3(nt), 0, stream, x, ld, x_off, channels,
                                    taps, (const TW*)w, (const TW*)bias, act, add_input, row_seq, row_pos, seq_row0,
                                    seq_pos0, seq_slot, state, (TO*)out, ld_out, out_off);
    });
  });
  SB_CHECK_LAUNCH("sb_causal_conv");
  if (!own && taps > 1) {
    sb_launch<SB_K_ELEMENTWISE>(conv_state_kernel, dim3(n_seqs, (channels + nt - 1) / nt), dim3(nt), 0, stream, x, ld,
                                x_off, channels, taps, seq_row0, seq_slot, state);
    SB_CHECK_LAUNCH("sb_causal_conv (state)");
  }
  return SB_OK;
}

extern "C" int sb_conv_heads_max_taps(void) { return CONV_HEADS_TAPS; }

extern "C" int sb_conv_heads(const float* proj, int n_rows, int ld, int n_q_heads, int n_kv_heads, int dim, int vdim,
                             int hd, int taps, const void* w, int w_dtype, int n_seqs, const int32_t* row_seq,
                             const int32_t* row_pos, const int32_t* seq_row0, const int32_t* seq_pos0,
                             const int32_t* seq_slot, const int32_t* page_off, const int32_t* page_ids,
                             int page_size, float* state, void* cache, void* q_out, int dtype, cudaStream_t stream) {
  if (n_rows <= 0 || n_seqs <= 0 || n_q_heads <= 0 || n_kv_heads <= 0 || dim <= 0 || vdim <= 0 || hd < dim || hd < vdim)
    SB_FAIL(SB_ERR_ARG, "sb_conv_heads: rows=%d seqs=%d heads=%d/%d dim=%d vdim=%d hd=%d", n_rows, n_seqs, n_q_heads,
            n_kv_heads, dim, vdim, hd);
  if (taps < 1 || taps > CONV_HEADS_TAPS)
    SB_FAIL(SB_ERR_UNSUPPORTED, "sb_conv_heads: %d taps (1 to %d)", taps, CONV_HEADS_TAPS);
  if (!proj || !w || !row_seq || !row_pos || !seq_row0 || !seq_pos0 || !seq_slot || !page_off || !page_ids || page_size <= 0 ||
      (taps > 1 && !state) || !cache || !q_out)
    SB_FAIL(SB_ERR_ARG, "sb_conv_heads: arguments missing");
  if (!sb_valid_dtype(w_dtype) || !sb_valid_dtype(dtype)) SB_FAIL(SB_ERR_ARG, "sb_conv_heads: dtype codes %d %d", w_dtype, dtype);
  const int channels = n_q_heads * dim + n_kv_heads * (dim + vdim);
  if (channels > ld) SB_FAIL(SB_ERR_ARG, "sb_conv_heads: %d channels in rows of %d", channels, ld);
  HeadsArgs a;
  a.proj = proj; a.n_rows = n_rows; a.ld = ld; a.hq = n_q_heads; a.hkv = n_kv_heads; a.dim = dim; a.vdim = vdim; a.hd = hd;
  a.w = w; a.row_seq = row_seq; a.row_pos = row_pos; a.seq_pos0 = seq_pos0; a.seq_slot = seq_slot; a.page_off = page_off;
  a.page_ids = page_ids; a.page_size = page_size; a.state = taps > 1 ? state : nullptr; a.cache = cache; a.q_out = q_out;
  const bool own = n_rows == n_seqs;
  const bool vec = dim % 4 == 0 && vdim % 4 == 0 && hd % 4 == 0 && ld % 4 == 0 &&
                   (((uintptr_t)proj | (uintptr_t)state | (uintptr_t)cache | (uintptr_t)q_out) & 15) == 0;
  SB_DISPATCH_DTYPE(w_dtype, TW, {
    SB_DISPATCH_DTYPE(dtype, T, {
      switch (taps) {
        case 1: launch_conv_heads<1, TW, T>(a, own, vec, stream); break;
        case 2: launch_conv_heads<2, TW, T>(a, own, vec, stream); break;
        case 3: launch_conv_heads<3, TW, T>(a, own, vec, stream); break;
        case 4: launch_conv_heads<4, TW, T>(a, own, vec, stream); break;
        default: launch_conv_heads<5, TW, T>(a, own, vec, stream); break;
      }
    });
  });
  SB_CHECK_LAUNCH("sb_conv_heads");
  if (!own && taps > 1) {
    sb_launch<SB_K_ELEMENTWISE>(conv_state_kernel, dim3(n_seqs, (channels + 255) / 256), dim3(256), 0, stream, proj, ld, 0,
                                channels, taps, seq_row0, seq_slot, state);
    SB_CHECK_LAUNCH("sb_conv_heads (state)");
  }
  return SB_OK;
}
