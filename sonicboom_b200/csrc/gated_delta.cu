// The gated delta rule: a recurrence over a matrix state with one decay per token and head and an update
// that replaces what the state holds under the unit key,
//
//     S <- g_t S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t,
//
// per head, S = 0 at a sequence's start.  q and k have `dim` values per key head, v and o `vdim` per head; head h
// reads key head h / (heads / kv_heads).  Every channel of q, k and v passes a short causal convolution over time
// and silu first; q and k are then divided by sqrt(sum of squares over the head + unit_eps), and q is
// multiplied by q_scale.  beta = sigmoid(b), g = exp(-exp(a_log) * softplus(a + dt_bias)) per head.  All float32.
//
// A projection row holds [q: kv_heads * dim | k: kv_heads * dim | v: heads * vdim] from column q_off (C values:
// the convolution's channels) and a, b [heads each] at a_off, b_off.  State of a sequence's slot: memory
// [heads, vdim, dim] (column by column) and the convolution's last inputs as a ring [taps, C] in which the input
// of position p lies in row p mod taps: a step of one token writes a row that it does not read.
//
//   sb_gdelta_step:   every sequence brings one row: convolution, silu, unit vectors, decay, update, read-out, the
//                     norm over a head's outputs and the gate in one kernel, a block per (head, sequence)
//   sb_gdelta_prep:   several rows: the convolved rows [rows, C] (q and k as unit vectors), and per chunk of 16
//                     tokens and head the matrices below
//   sb_gdelta_scan:   the recurrence chunk by chunk from and to the state
//
// A chunk.  With G_i = g_0 ... g_i, D_ij = g_(j+1) ... g_i (products, so that small decays lose nothing to
// differences of logarithms) and S the state before the chunk, the updates of a chunk's tokens solve a triangular system:
//
//     u_i + beta_i sum_(j<i) D_ij (k_i . k_j) u_j = beta_i (v_i - G_i S^T k_i)
//
// so u = T (v - G * (S^T k)) with T = (I + M)^(-1) diag(beta), M_ij = beta_i D_ij (k_i . k_j) below the diagonal, and
//
//     o_i = G_i S^T q_i + sum_(j<=i) P_ij u_j,  P_ij = D_ij (q_i . k_j);     S <- G_15 S + sum_j D_15,j k_j u_j^T.
//
// T and P depend on the key head and head, not on the value channel: they are made once per head, and what is
// left per column of the state are three passes over it for 16 tokens (S^T k, S^T q, the update), none of
// which waits for the token before.  Chunks start at a step's first row of a sequence; tokens past its last row have
// beta 0, g 1 and zero vectors.
#include <math.h>

#include "common.cuh"

namespace {

constexpr int TB = 16;                          // tokens of a chunk
constexpr int MATS = 2 * TB * TB + 2 * TB;      // floats of a chunk and head: T, P, G, D_15

__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }

// Where the chunks of sequence b start in the chunk matrices: never overlapping, at most n_rows / 16 + n_seqs in all.
__device__ __forceinline__ int chunk_base(int row0, int b) { return row0 / TB + b; }

template <int N>
__device__ __forceinline__ float lanes_sum(float v) {
#pragma unroll
  for (int o = N / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// Lane `sub` of LANES keeps NPL channels of a column in runs of R = min(NPL, 4): run j holds channels
// j * LANES R + sub R ... + R - 1, so that the lanes' loads of a run are one contiguous stretch.
constexpr int LANES = 8;
template <int NPL>
struct Runs {
  static constexpr int R = NPL < 4 ? NPL : 4;
  __device__ static __forceinline__ int channel(int sub, int i) { return (i / R) * (LANES * R) + sub * R + i % R; }
};

// ------------------------------------------------------------------------------------------- one token
struct StepArgs {
  const float* proj;
  int ld, q_off, a_off, b_off, g_off;
  int n_heads, n_kv_heads, dim, vdim, taps;
  const float* conv_w;                 // [C, taps]
  const float* a_log;
  const float* dt_bias;
  const int32_t* row_pos;
  const int32_t* seq_slot;
  float* ring;                         // [slot, taps, C], or null (one tap)
  float* memory;                       // [slot, heads, vdim, dim]
  const float* norm_w;                 // [vdim]
  float q_scale, unit_eps, eps, out_scale;
  void* out;
  int ld_out, out_off;
};

constexpr int STEP_THREADS = 256;

template <int NPL, bool VEC, typename TO>
__global__ void __launch_bounds__(STEP_THREADS) gdelta_step_kernel(const StepArgs p) {
  extern __shared__ __align__(16) float sm[];
  constexpr int PAD = NPL * LANES, R = Runs<NPL>::R, COLS = STEP_THREADS / LANES;
  float* qs = sm;                      // [PAD]
  float* ks = qs + PAD;                // [PAD]
  float* vs = ks + PAD;                // [vdim]
  float* os = vs + p.vdim;             // [vdim]
  __shared__ float inv[2], red[STEP_THREADS / 32];
  sb_pdl_launch();
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int per = p.n_heads / p.n_kv_heads, kv = h / per;
  const int dim = p.dim, vdim = p.vdim, taps = p.taps;
  const int kw = p.n_kv_heads * dim, C = 2 * kw + p.n_heads * vdim;
  const int slot = p.seq_slot[b], pos = p.row_pos[b];
  float* memory = p.memory + ((size_t)slot * p.n_heads + h) * vdim * dim;
  // the head's state is on its way into L2 while the product before this kernel ends (a hint: nothing is read yet)
  for (size_t e = (size_t)tid * 32; e < (size_t)vdim * dim; e += STEP_THREADS * 32)
    asm volatile("prefetch.global.L2 [%0];\n" ::"l"(memory + e));
  for (int c = dim + tid; c < PAD; c += STEP_THREADS) qs[c] = ks[c] = 0.0f;
  sb_pdl_wait();
  const float* row = p.proj + (size_t)b * p.ld;
  float* ring = p.ring ? p.ring + (size_t)slot * taps * C : nullptr;
  const float* w = p.conv_w;
  for (int i = tid; i < 2 * dim + vdim; i += STEP_THREADS) {
    const int c = i < dim ? kv * dim + i : (i < 2 * dim ? kw + kv * dim + i - dim : 2 * kw + h * vdim + i - 2 * dim);
    const float cur = row[p.q_off + c];
    float acc = 0.0f;
    for (int j = 0; j + 1 < taps; ++j) {
      const int at = pos - (taps - 1) + j;
      acc = fmaf(w[(size_t)c * taps + j], at >= 0 ? ring[(size_t)(at % taps) * C + c] : 0.0f, acc);
    }
    acc = fmaf(w[(size_t)c * taps + taps - 1], cur, acc);
    (i < dim ? qs[i] : (i < 2 * dim ? ks[i - dim] : vs[i - 2 * dim])) = sb_silu(acc);
    // the group's first head keeps the inputs of q and k, every head those of its own values
    if (taps > 1 && (i >= 2 * dim || h == kv * per)) ring[(size_t)(pos % taps) * C + c] = cur;
  }
  const float beta = sigmoid(row[p.b_off + h]);
  const float g = expf(-expf(p.a_log[h]) * softplus(row[p.a_off + h] + p.dt_bias[h]));
  __syncthreads();
  if (warp < 2) {
    const float* x = warp == 0 ? qs : ks;
    float s = 0.0f;
    for (int c = lane; c < dim; c += 32) s = fmaf(x[c], x[c], s);
    s = sb_warp_sum(s);
    if (lane == 0) inv[warp] = 1.0f / sqrtf(s + p.unit_eps) * (warp == 0 ? p.q_scale : 1.0f);
  }
  __syncthreads();
  const int sub = tid % LANES, cl = tid / LANES;
  float kr[NPL], qr[NPL];
#pragma unroll
  for (int i = 0; i < NPL; ++i) {
    const int c = Runs<NPL>::channel(sub, i);
    qr[i] = qs[c] * inv[0];
    kr[i] = ks[c] * inv[1];
  }
  auto load = [&](int col, float (&S)[NPL]) {
#pragma unroll
    for (int j = 0; j < NPL / R; ++j) {
      const int c = j * (LANES * R) + sub * R;
      if (VEC && R == 4) {
        const float4 f = col < vdim && c < dim ? *reinterpret_cast<const float4*>(memory + (size_t)col * dim + c)
                                               : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        S[j * R] = f.x; S[j * R + 1 % R] = f.y; S[j * R + 2 % R] = f.z; S[j * R + 3 % R] = f.w;
      } else {
#pragma unroll
        for (int u = 0; u < R; ++u) S[j * R + u] = col < vdim && c + u < dim ? memory[(size_t)col * dim + c + u] : 0.0f;
      }
    }
  };
  float S[NPL], next[NPL];
  load(cl, S);
  for (int c0 = 0; c0 < vdim; c0 += COLS) {
    const int col = c0 + cl;
    load(col + COLS, next);            // the columns of the next turn, while this turn's are worked on
    float d = 0.0f;
#pragma unroll
    for (int i = 0; i < NPL; ++i) {
      S[i] *= g;
      d = fmaf(kr[i], S[i], d);
    }
    d = lanes_sum<LANES>(d);
    const float u = col < vdim ? beta * (vs[col] - d) : 0.0f;
    float o = 0.0f;
#pragma unroll
    for (int i = 0; i < NPL; ++i) {
      S[i] = fmaf(kr[i], u, S[i]);
      o = fmaf(qr[i], S[i], o);
    }
    o = lanes_sum<LANES>(o);
    if (col < vdim) {
      if (sub == 0) os[col] = o;
#pragma unroll
      for (int j = 0; j < NPL / R; ++j) {
        const int c = j * (LANES * R) + sub * R;
        if (VEC && R == 4) {
          if (c < dim)
            *reinterpret_cast<float4*>(memory + (size_t)col * dim + c) =
                make_float4(S[j * R], S[j * R + 1 % R], S[j * R + 2 % R], S[j * R + 3 % R]);
        } else {
#pragma unroll
          for (int u2 = 0; u2 < R; ++u2)
            if (c + u2 < dim) memory[(size_t)col * dim + c + u2] = S[j * R + u2];
        }
      }
    }
#pragma unroll
    for (int i = 0; i < NPL; ++i) S[i] = next[i];
  }
  __syncthreads();
  float s = 0.0f;
  for (int j = tid; j < vdim; j += STEP_THREADS) s = fmaf(os[j], os[j], s);
  s = sb_warp_sum(s);
  if (lane == 0) red[warp] = s;
  __syncthreads();
  float total = 0.0f;
#pragma unroll
  for (int i = 0; i < STEP_THREADS / 32; ++i) total += red[i];
  const float r = 1.0f / sqrtf(total / (float)vdim + p.eps);
  const float* gate = row + p.g_off + (size_t)h * vdim;
  TO* out = (TO*)p.out + (size_t)b * p.ld_out + p.out_off + (size_t)h * vdim;
  for (int j = tid; j < vdim; j += STEP_THREADS)
    out[j] = sb_from_f32<TO>((os[j] * r) * p.norm_w[j] * sb_silu(gate[j]) * p.out_scale);
}

// ------------------------------------------------------------------------------------- a chunk's inputs
struct PrepArgs {
  const float* proj;
  int ld, q_off, a_off, b_off;
  int n_heads, n_kv_heads, dim, vdim, taps;
  const float* conv_w;
  const float* a_log;
  const float* dt_bias;
  const int32_t* seq_row0;
  const int32_t* seq_pos0;
  const int32_t* seq_slot;
  const float* ring;
  float q_scale, unit_eps;
  float* act;                          // [rows, C]
  float* mats;                         // [chunks, heads, MATS]
};

constexpr int PREP_THREADS = 128;

// The convolution and silu of channel c over a chunk's tokens t0 ... t0 + cnt - 1 (rows of the sequence's stretch of the
// step, whose first row is row0 at position pos0); put(token, value).  MAXT > 0: at most MAXT taps, whose last
// inputs stay in registers; 0: any number, read again for every tap.
template <int MAXT, typename Put>
__device__ __forceinline__ void conv_walk(const float* x, int ld, int row0, int pos0, int t0, int cnt, int taps, int C, int c,
                                          const float* __restrict__ w, const float* ring, Put put) {
  auto before = [&](int t) {            // the input of the sequence's token pos0 + t, t < 0: the ring, or zero
    const int at = pos0 + t;
    return at >= 0 ? ring[(size_t)(at % taps) * C + c] : 0.0f;
  };
  if constexpr (MAXT > 0) {
    float wd[MAXT], hist[MAXT];         // by distance: the weight of the input d tokens back, and that input
#pragma unroll
    for (int d = 0; d < MAXT; ++d) {
      wd[d] = d < taps ? w[(size_t)c * taps + taps - 1 - d] : 0.0f;
      hist[d] = 0.0f;
      if (d >= 1 && d < taps) hist[d] = t0 - d >= 0 ? x[(size_t)(row0 + t0 - d) * ld + c] : before(t0 - d);
    }
#pragma unroll 4
    for (int i = 0; i < cnt; ++i) {
      hist[0] = x[(size_t)(row0 + t0 + i) * ld + c];
      float acc = 0.0f;
#pragma unroll
      for (int d = MAXT - 1; d >= 0; --d) acc = fmaf(wd[d], hist[d], acc);
      put(i, sb_silu(acc));
#pragma unroll
      for (int d = MAXT - 1; d >= 1; --d) hist[d] = hist[d - 1];
    }
  } else {
    for (int i = 0; i < cnt; ++i) {
      float acc = 0.0f;
      for (int d = taps - 1; d >= 0; --d) {
        const int t = t0 + i - d;
        acc = fmaf(w[(size_t)c * taps + taps - 1 - d], t >= 0 ? x[(size_t)(row0 + t) * ld + c] : before(t), acc);
      }
      put(i, sb_silu(acc));
    }
  }
}

template <int MAXT>
__global__ void __launch_bounds__(PREP_THREADS) gdelta_prep_kernel(const PrepArgs p) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float qk[TB][TB + 1], kk[TB][TB + 1], ms[PREP_THREADS / 32][TB][TB + 1];
  sb_pdl_launch();
  const int b = blockIdx.z, kv = blockIdx.y, t0 = blockIdx.x * TB;
  const int row0 = p.seq_row0[b], n = p.seq_row0[b + 1] - row0;
  if (t0 >= n) return;
  const int cnt = min(TB, n - t0), pos0 = p.seq_pos0[b];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int dim = p.dim, vdim = p.vdim, taps = p.taps, per = p.n_heads / p.n_kv_heads;
  const int kw = p.n_kv_heads * dim, C = 2 * kw + p.n_heads * vdim;
  const int pitch = (dim + 3) / 4 * 4 + 4;
  float* qs = sm;                       // [TB, pitch], then the keys
  float* ks = sm + TB * pitch;
  for (int i = tid; i < 2 * TB * pitch; i += PREP_THREADS) sm[i] = 0.0f;
  __syncthreads();
  sb_pdl_wait();
  const float* x = p.proj + p.q_off;
  const float* ring = p.ring ? p.ring + (size_t)p.seq_slot[b] * taps * C : nullptr;
  const float* w = p.conv_w;
  for (int i = tid; i < 2 * dim; i += PREP_THREADS) {
    const int c = i < dim ? i : i - dim;
    float* dst = (i < dim ? qs : ks) + c;
    conv_walk<MAXT>(x, p.ld, row0, pos0, t0, cnt, taps, C, (i < dim ? 0 : kw) + kv * dim + c, w, ring,
                    [&](int t, float v) { dst[t * pitch] = v; });
  }
  float* act = p.act + (size_t)(row0 + t0) * C;
  for (int i = tid; i < per * vdim; i += PREP_THREADS) {
    const int c = 2 * kw + kv * per * vdim + i;
    conv_walk<MAXT>(x, p.ld, row0, pos0, t0, cnt, taps, C, c, w, ring, [&](int t, float v) { act[(size_t)t * C + c] = v; });
  }
  __syncthreads();
  for (int i = warp; i < 2 * TB; i += PREP_THREADS / 32) {            // unit vectors, a warp each
    const int t = i % TB, is_k = i / TB;
    float* v = (is_k ? ks : qs) + t * pitch;
    float s = 0.0f;
    for (int c = lane; c < dim; c += 32) s = fmaf(v[c], v[c], s);
    const float inv = 1.0f / sqrtf(sb_warp_sum(s) + p.unit_eps) * (is_k ? 1.0f : p.q_scale);
    for (int c = lane; c < dim; c += 32) {
      const float y = v[c] * inv;
      v[c] = y;
      if (t < cnt) act[(size_t)t * C + is_k * kw + kv * dim + c] = y;
    }
  }
  __syncthreads();
  {  // q_i . k_j and k_i . k_j: a thread has row i and columns j, j + 8
    const int i = tid / 8, j = tid % 8;
    float a0 = 0.0f, a1 = 0.0f, c0 = 0.0f, c1 = 0.0f;
    for (int c = 0; c < dim; c += 4) {
      const float4 q4 = *reinterpret_cast<const float4*>(qs + i * pitch + c), k4 = *reinterpret_cast<const float4*>(ks + i * pitch + c);
      const float4 u = *reinterpret_cast<const float4*>(ks + j * pitch + c), v = *reinterpret_cast<const float4*>(ks + (j + 8) * pitch + c);
      a0 = fmaf(q4.x, u.x, fmaf(q4.y, u.y, fmaf(q4.z, u.z, fmaf(q4.w, u.w, a0))));
      a1 = fmaf(q4.x, v.x, fmaf(q4.y, v.y, fmaf(q4.z, v.z, fmaf(q4.w, v.w, a1))));
      c0 = fmaf(k4.x, u.x, fmaf(k4.y, u.y, fmaf(k4.z, u.z, fmaf(k4.w, u.w, c0))));
      c1 = fmaf(k4.x, v.x, fmaf(k4.y, v.y, fmaf(k4.z, v.z, fmaf(k4.w, v.w, c1))));
    }
    qk[i][j] = a0; qk[i][j + 8] = a1; kk[i][j] = c0; kk[i][j + 8] = c1;
  }
  __syncthreads();
  // per head: lane j (and j + 16, which repeats its work) has column j of the matrices
  const int j = lane % TB;
  float (*M)[TB + 1] = ms[warp];
  for (int hh = warp; hh < per; hh += PREP_THREADS / 32) {
    const int h = kv * per + hh;
    float beta = 0.0f, g = 1.0f;
    if (j < cnt) {
      const float* row = p.proj + (size_t)(row0 + t0 + j) * p.ld;
      beta = sigmoid(row[p.b_off + h]);
      g = expf(-expf(p.a_log[h]) * softplus(row[p.a_off + h] + p.dt_bias[h]));
    }
    float* out = p.mats + ((size_t)(chunk_base(row0, b) + blockIdx.x) * p.n_heads + h) * MATS;
    float d = 1.0f, run = 1.0f, mine = 1.0f;
#pragma unroll
    for (int i = 0; i < TB; ++i) {
      const float gi = __shfl_sync(0xffffffffu, g, i), bi = __shfl_sync(0xffffffffu, beta, i);
      run *= gi;
      if (i == j) mine = run;
      if (i > j) d *= gi;
      if (lane < TB) {
        M[i][j] = i > j ? bi * d * kk[i][j] : 0.0f;
        out[TB * TB + i * TB + j] = i >= j ? d * qk[i][j] : 0.0f;
      }
    }
    __syncwarp();
    float xcol[TB];                     // column j of (I + M)^(-1), forward substitution
#pragma unroll
    for (int i = 0; i < TB; ++i) {
      float s = 0.0f;
#pragma unroll
      for (int m = 0; m < TB; ++m)
        if (m < i) s = fmaf(M[i][m], xcol[m], s);
      xcol[i] = i == j ? 1.0f : (i < j ? 0.0f : -s);
    }
    if (lane < TB) {
#pragma unroll
      for (int i = 0; i < TB; ++i) out[i * TB + j] = xcol[i] * beta;
      out[2 * TB * TB + j] = mine;
      out[2 * TB * TB + TB + j] = d;
    }
    __syncwarp();
  }
}

// ------------------------------------------------------------------------------------------- the scan
__device__ __forceinline__ void cp_async4(float* dst, const float* src, bool ok) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(ok ? 4 : 0));
}
__device__ __forceinline__ void cp_async16(float* dst, const float* src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(ok ? 16 : 0));
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;\n"); }
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N)); }

struct ScanArgs {
  const float* act;
  const float* mats;
  const float* proj;
  int ld, q_off;
  int n_heads, n_kv_heads, dim, vdim, taps;
  const int32_t* seq_row0;
  const int32_t* seq_pos0;
  const int32_t* seq_slot;
  float* ring;
  float* memory;
  float* out;                          // [rows, heads, vdim]
};

constexpr int SCAN_THREADS = 128, SCAN_LANES = 16, SCAN_GROUPS = SCAN_THREADS / SCAN_LANES;
constexpr int TP = TB + 4;                      // pitch of a staged matrix row
constexpr int MAT_SM = 2 * TB * TP + 2 * TB;    // T, P, G, D_15
constexpr int HALF = TB / 2;

template <int NPL, int CPT>
struct ScanShape {
  static constexpr int PAD = NPL * SCAN_LANES, COLS = SCAN_GROUPS * CPT;
  static constexpr int VP = COLS + 4;                                   // pitch of a token's values
  static constexpr int STAGE = 2 * TB * PAD + TB * VP + MAT_SM;         // q, k, values, matrices
  static constexpr int XP = TB + 4;                                     // pitch of a column's exchange buffer
  static constexpr int EXTRA = SCAN_GROUPS * CPT * XP;
  static constexpr size_t bytes(int stages) { return ((size_t)stages * STAGE + EXTRA) * sizeof(float); }
};

template <int N>
struct Size {
  static constexpr int value = N;
};

// Two float32 values side by side: one fma instruction works on both, each rounded as a fma of its own.
struct Two {
  unsigned long long v;
};
__device__ __forceinline__ Two two(float lo, float hi) {
  Two r;
  asm("mov.b64 %0, {%1, %2};\n" : "=l"(r.v) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ float2 parts(Two a) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;\n" : "=f"(r.x), "=f"(r.y) : "l"(a.v));
  return r;
}
__device__ __forceinline__ Two fma2(Two a, Two b, Two c) {
  Two r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;\n" : "=l"(r.v) : "l"(a.v), "l"(b.v), "l"(c.v));
  return r;
}

// The lanes of a column add their parts of eight tokens' sums, halving what a lane keeps each time: lane `sub` ends with the
// sum of token sub % 8, by the same tree of additions for every token.
__device__ __forceinline__ float share_sums(float (&a)[HALF], int sub) {
#pragma unroll
  for (int w = HALF / 2; w > 0; w >>= 1) {
    const bool up = sub & w;
#pragma unroll
    for (int i = 0; i < w; ++i) {
      const float keep = up ? a[i + w] : a[i], give = up ? a[i] : a[i + w];
      a[i] = keep + __shfl_xor_sync(0xffffffffu, give, w);
    }
  }
  return a[0] + __shfl_xor_sync(0xffffffffu, a[0], HALF);
}

// A lane keeps NPL channels (in pairs) of CPT neighbouring columns for the whole step: what it reads of a token's q
// and k from shared memory serves CPT columns, and shared memory's bandwidth, a value a lane and cycle, is what
// the kernel runs against.  With up to 8 channels a lane also keeps the chunk's keys in registers from the first pass (S^T k)
// to the last (the update).
template <int NPL, int CPT, bool VEC, int STAGES>
__global__ void __launch_bounds__(SCAN_THREADS) gdelta_scan_kernel(const ScanArgs p) {
  using Sh = ScanShape<NPL, CPT>;
  constexpr int PAD = Sh::PAD, COLS = Sh::COLS, V = VEC ? 4 : 1;
  constexpr int R = NPL < 4 ? NPL : 4, N2 = NPL / 2;      // values of a run; pairs of a lane
  constexpr bool KEEP = NPL <= 8;
  extern __shared__ __align__(16) float sm[];
  float* xbuf = sm + STAGES * Sh::STAGE;
  sb_pdl_launch();
  const int b = blockIdx.z, h = blockIdx.y, tid = threadIdx.x, sub = tid % SCAN_LANES, cl = tid / SCAN_LANES;
  const int dim = p.dim, vdim = p.vdim, taps = p.taps, per = p.n_heads / p.n_kv_heads, kv = h / per;
  const int kw = p.n_kv_heads * dim, C = 2 * kw + p.n_heads * vdim;
  const int col0 = blockIdx.x * COLS, col = col0 + cl * CPT;
  const int row0 = p.seq_row0[b], n = p.seq_row0[b + 1] - row0, slot = p.seq_slot[b];
  // lane `sub`'s channel i: runs of R, as far apart as the lanes' runs are long together
  auto channel = [&](int i) { return (i / R) * (SCAN_LANES * R) + sub * R + i % R; };
  if (PAD > dim || vdim - col0 < COLS) {          // channels and columns past the sizes stay zero for good
    for (int i = tid; i < STAGES * Sh::STAGE; i += SCAN_THREADS) sm[i] = 0.0f;
    __syncthreads();
  }
  sb_pdl_wait();
  const float* act = p.act + (size_t)row0 * C;
  const float* mats = p.mats + ((size_t)chunk_base(row0, b) * p.n_heads + h) * MATS;
  // Staging: a thread keeps to its pieces (V values) of a token's row and takes tokens STEP apart; every division is by a
  // constant, and a chunk's source addresses follow from the first one's.
  const int n_vals = min(COLS, vdim - col0);
  auto copy = [&](float* to, int pitch, const float* from, int t0, int width, auto padded) {   // `width` values of 16 tokens' rows
    constexpr int PIECES = decltype(padded)::value / V, W = PIECES < SCAN_THREADS ? PIECES : SCAN_THREADS, STEP = SCAN_THREADS / W;
    const int first = tid / W, piece = tid % W;
    if (W * STEP < SCAN_THREADS && first >= STEP) return;
#pragma unroll
    for (int t = first; t < TB; t += STEP) {
      const bool ok = t0 + t < n;
      const float* row = ok ? from + (size_t)(t0 + t) * C : act;
#pragma unroll
      for (int i = piece; i < PIECES; i += W)
        if (i * V < width) {
          if (VEC) cp_async16(to + t * pitch + i * V, row + (ok ? i * V : 0), ok);
          else cp_async4(to + t * pitch + i, row + (ok ? i : 0), ok);
        }
    }
  };
  const float* q_src = act + kv * dim;
  const float* k_src = q_src + kw;
  const float* v_src = act + 2 * kw + h * vdim + col0;
  auto stage = [&](int st, int ch) {
    float* dst = sm + (size_t)st * Sh::STAGE;
    copy(dst, PAD, q_src, ch * TB, dim, Size<PAD>());
    copy(dst + TB * PAD, PAD, k_src, ch * TB, dim, Size<PAD>());
    copy(dst + 2 * TB * PAD, Sh::VP, v_src, ch * TB, n_vals, Size<COLS>());
    float* m = dst + 2 * TB * PAD + TB * Sh::VP;
    const float* src = mats + (size_t)ch * p.n_heads * MATS;
#pragma unroll
    for (int i = tid; i < MATS / 4; i += SCAN_THREADS) {
      const int e = i * 4;
      cp_async16(m + (e < 2 * TB * TB ? (e / TB) * TP + e % TB : 2 * TB * TP + e - 2 * TB * TB), src + e, true);
    }
  };
  const int n_chunks = (n + TB - 1) / TB;
#pragma unroll
  for (int s = 0; s < STAGES - 1; ++s) {
    if (s < n_chunks) stage(s, s);
    cp_commit();
  }
  float* memory = p.memory + ((size_t)slot * p.n_heads + h) * vdim * dim;
  Two S[CPT][N2];
#pragma unroll
  for (int x = 0; x < CPT; ++x)
#pragma unroll
    for (int i = 0; i < N2; ++i) {
      float v[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int c = channel(2 * i + e);
        v[e] = col + x < vdim && c < dim ? memory[(size_t)(col + x) * dim + c] : 0.0f;
      }
      S[x][i] = two(v[0], v[1]);
    }
  float* xb = xbuf + cl * CPT * Sh::XP;
  auto load_row = [&](const float* row, Two (&r)[N2]) {   // this lane's channels of a token's q or k
#pragma unroll
    for (int j = 0; j < NPL / R; ++j) {
      const float* at = row + j * (SCAN_LANES * R) + sub * R;
      if constexpr (R == 4) {
        const float4 f = *reinterpret_cast<const float4*>(at);
        r[2 * j] = two(f.x, f.y);
        r[2 * j + 1] = two(f.z, f.w);
      } else {
        const float2 f = *reinterpret_cast<const float2*>(at);
        r[j] = two(f.x, f.y);
      }
    }
  };

  for (int ch = 0; ch < n_chunks; ++ch) {
    cp_wait<STAGES - 2>();
    __syncthreads();                    // the chunk has landed, and every thread is done with the buffer staged next
    if (ch + STAGES - 1 < n_chunks) stage((ch + STAGES - 1) % STAGES, ch + STAGES - 1);
    cp_commit();
    const float* q = sm + (size_t)(ch % STAGES) * Sh::STAGE;
    const float* k = q + TB * PAD;
    const float* v = k + TB * PAD;
    const float* T = v + TB * Sh::VP;
    const float* P = T + TB * TP;
    const float* G = P + TB * TP;
    const float* D = G + TB;
    Two kr[KEEP ? TB : 1][N2];
    // S^T k_t and S^T q_t of the chunk's tokens: lane `sub` ends with those of token `sub`
    float d[CPT], o[CPT];
#pragma unroll
    for (int pass = 0; pass < 2; ++pass)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        float acc[CPT][HALF];
#pragma unroll
        for (int t = 0; t < HALF; ++t) {
          Two r[N2];
          load_row((pass == 0 ? k : q) + (half * HALF + t) * PAD, r);
#pragma unroll
          for (int x = 0; x < CPT; ++x) {
            Two a = two(0.0f, 0.0f);
#pragma unroll
            for (int i = 0; i < N2; ++i) a = fma2(r[i], S[x][i], a);
            const float2 f = parts(a);
            acc[x][t] = f.x + f.y;
          }
          if (KEEP && pass == 0)
#pragma unroll
            for (int i = 0; i < N2; ++i) kr[half * HALF + t][i] = r[i];
        }
#pragma unroll
        for (int x = 0; x < CPT; ++x) {
          const float y = share_sums(acc[x], sub);
          if (half == 0 || (sub & HALF)) (pass == 0 ? d : o)[x] = y;
        }
      }
    // w = v - G * (S^T k), to the column's other lanes; u = T w
    const float g_own = G[sub], g_all = G[TB - 1];
    float own[CPT];
    if constexpr (CPT == 4) {
      const float4 f = *reinterpret_cast<const float4*>(v + sub * Sh::VP + cl * CPT);
      own[0] = f.x; own[1] = f.y; own[2] = f.z; own[3] = f.w;
    } else {
#pragma unroll
      for (int x = 0; x < CPT; ++x) own[x] = v[sub * Sh::VP + cl * CPT + x];
    }
    __syncwarp();
#pragma unroll
    for (int x = 0; x < CPT; ++x) xb[x * Sh::XP + sub] = own[x] - g_own * d[x];
    __syncwarp();
#pragma unroll
    for (int x = 0; x < CPT; ++x) d[x] = 0.0f, o[x] *= g_own;
#pragma unroll
    for (int i = 0; i < TB; i += 4) {
      const float4 m = *reinterpret_cast<const float4*>(T + sub * TP + i);
#pragma unroll
      for (int x = 0; x < CPT; ++x) {
        const float4 w = *reinterpret_cast<const float4*>(xb + x * Sh::XP + i);
        d[x] = fmaf(m.x, w.x, d[x]); d[x] = fmaf(m.y, w.y, d[x]); d[x] = fmaf(m.z, w.z, d[x]); d[x] = fmaf(m.w, w.w, d[x]);
      }
    }
    __syncwarp();
#pragma unroll
    for (int x = 0; x < CPT; ++x) xb[x * Sh::XP + sub] = d[x];
    __syncwarp();
    const Two gg = two(g_all, g_all), zero = two(0.0f, 0.0f);
#pragma unroll
    for (int x = 0; x < CPT; ++x)
#pragma unroll
      for (int i = 0; i < N2; ++i) S[x][i] = fma2(S[x][i], gg, zero);
    // o += P u;  S += sum_j D_15,j k_j u_j
#pragma unroll
    for (int i = 0; i < TB; i += 4) {
      const float4 m = *reinterpret_cast<const float4*>(P + sub * TP + i), f = *reinterpret_cast<const float4*>(D + i);
      const float dd[4] = {f.x, f.y, f.z, f.w};
      float u[CPT][4];
#pragma unroll
      for (int x = 0; x < CPT; ++x) {
        const float4 w = *reinterpret_cast<const float4*>(xb + x * Sh::XP + i);
        o[x] = fmaf(m.x, w.x, o[x]); o[x] = fmaf(m.y, w.y, o[x]); o[x] = fmaf(m.z, w.z, o[x]); o[x] = fmaf(m.w, w.w, o[x]);
        u[x][0] = w.x; u[x][1] = w.y; u[x][2] = w.z; u[x][3] = w.w;
      }
#pragma unroll
      for (int t = 0; t < 4; ++t) {
        Two r[N2];
        if (KEEP) {
#pragma unroll
          for (int e = 0; e < N2; ++e) r[e] = kr[KEEP ? i + t : 0][e];
        } else {
          load_row(k + (i + t) * PAD, r);
        }
#pragma unroll
        for (int x = 0; x < CPT; ++x) {
          const float e = dd[t] * u[x][t];
          const Two ee = two(e, e);
#pragma unroll
          for (int j = 0; j < N2; ++j) S[x][j] = fma2(r[j], ee, S[x][j]);
        }
      }
    }
    const int t = ch * TB + sub;
    if (t < n) {
      float* to = p.out + ((size_t)(row0 + t) * p.n_heads + h) * vdim + col;
      if (VEC && CPT == 4) {            // vdim is a multiple of four, so four columns are all there or none is
        if (col < vdim) *reinterpret_cast<float4*>(to) = make_float4(o[0], o[1 % CPT], o[2 % CPT], o[3 % CPT]);
      } else {
#pragma unroll
        for (int x = 0; x < CPT; ++x)
          if (col + x < vdim) to[x] = o[x];
      }
    }
  }
  cp_wait<0>();
#pragma unroll
  for (int x = 0; x < CPT; ++x)
#pragma unroll
    for (int i = 0; i < N2; ++i) {
      const float2 f = parts(S[x][i]);
      const int c = channel(2 * i);
      if (col + x < vdim && c < dim) memory[(size_t)(col + x) * dim + c] = f.x;
      if (col + x < vdim && c + 1 < dim) memory[(size_t)(col + x) * dim + c + 1] = f.y;
    }
  // the convolution's last inputs (the kernel before this one has read the old ones): a head keeps its own values'
  // channels, a group's first head those of q and k too
  if (taps > 1 && blockIdx.x == 0) {
    float* ring = p.ring + (size_t)slot * taps * C;
    const int pos0 = p.seq_pos0[b], keep = min(n, taps), n_ch = vdim + (h == kv * per ? 2 * dim : 0);
    for (int i = tid; i < n_ch; i += SCAN_THREADS) {
      const int c = i < vdim ? 2 * kw + h * vdim + i : (i < vdim + dim ? kv * dim + i - vdim : kw + kv * dim + i - vdim - dim);
      for (int t = n - keep; t < n; ++t) ring[(size_t)((pos0 + t) % taps) * C + c] = p.proj[(size_t)(row0 + t) * p.ld + p.q_off + c];
    }
  }
}

int sm_count() {
  static int n = 0;
  if (n == 0) {
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess)
      n = 1;
  }
  return n;
}

template <int NPL, int CPT, bool VEC>
cudaError_t launch_scan_columns(const ScanArgs& a, int n_seqs, cudaStream_t stream) {
  constexpr int STAGES = ScanShape<NPL, CPT>::bytes(3) <= 112 * 1024 ? 3 : 2;
  constexpr size_t smem = ScanShape<NPL, CPT>::bytes(STAGES);
  static bool configured = false;
  if (!configured && smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(gdelta_scan_kernel<NPL, CPT, VEC, STAGES>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  configured = true;
  const dim3 grid((a.vdim + ScanShape<NPL, CPT>::COLS - 1) / ScanShape<NPL, CPT>::COLS, a.n_heads, n_seqs);
  return sb_launch<SB_K_OTHER>(gdelta_scan_kernel<NPL, CPT, VEC, STAGES>, grid, dim3(SCAN_THREADS), smem, stream, a);
}

int g_force_cpt = 0;

// Four columns a thread where that still gives every SM a block, else two; the largest key sizes keep fewer.  Measured on
// B200, 2,048 tokens of one sequence, heads of 128 x 128: 56 heads (224 blocks of four columns a thread) 525 us against
// 603 us with two, 32 heads (128 blocks) 325 against 312 us, 16 heads 324 against 202 us.
template <int NPL, bool VEC>
cudaError_t launch_scan(const ScanArgs& a, int n_seqs, cudaStream_t stream) {
  if constexpr (NPL > 16) {
    return launch_scan_columns<NPL, 1, VEC>(a, n_seqs, stream);
  } else if constexpr (NPL > 8 || !VEC) {
    return launch_scan_columns<NPL, 2, VEC>(a, n_seqs, stream);
  } else {
    const long blocks4 = (long)((a.vdim + 4 * SCAN_GROUPS - 1) / (4 * SCAN_GROUPS)) * a.n_heads * n_seqs;
    if (g_force_cpt ? g_force_cpt == 4 : blocks4 >= sm_count()) return launch_scan_columns<NPL, 4, VEC>(a, n_seqs, stream);
    return launch_scan_columns<NPL, 2, VEC>(a, n_seqs, stream);
  }
}

int check_sizes(const char* what, int n_heads, int n_kv_heads, int dim, int vdim, int taps) {
  if (n_heads <= 0 || n_kv_heads <= 0 || n_heads % n_kv_heads || dim <= 0 || vdim <= 0 || taps <= 0)
    SB_FAIL(SB_ERR_ARG, "%s: heads=%d/%d dim=%d vdim=%d taps=%d", what, n_heads, n_kv_heads, dim, vdim, taps);
  if (dim > 64 * LANES) SB_FAIL(SB_ERR_UNSUPPORTED, "%s: key size %d is above %d", what, dim, 64 * LANES);
  if (vdim > 8192) SB_FAIL(SB_ERR_UNSUPPORTED, "%s: value size %d is above 8192", what, vdim);
  return SB_OK;
}

}  // namespace

extern "C" int sb_gdelta_step(const float* proj, int n_seqs, int ld, int q_off, int a_off, int b_off, int g_off, int n_heads,
                              int n_kv_heads, int dim, int vdim, int taps, const float* conv_w, const float* a_log,
                              const float* dt_bias, const int32_t* row_pos, const int32_t* seq_slot, float* ring,
                              float* memory, float q_scale, float unit_eps, const float* norm_w, float eps, float out_scale,
                              void* out, int out_dtype, int ld_out, int out_off, cudaStream_t stream) {
  if (int rc = check_sizes("sb_gdelta_step", n_heads, n_kv_heads, dim, vdim, taps)) return rc;
  if (n_seqs <= 0 || !proj || !conv_w || !a_log || !dt_bias || !row_pos || !seq_slot || (taps > 1 && !ring) || !memory ||
      !norm_w || !out)
    SB_FAIL(SB_ERR_ARG, "sb_gdelta_step: arguments missing (seqs=%d)", n_seqs);
  if (!sb_valid_dtype(out_dtype)) SB_FAIL(SB_ERR_ARG, "sb_gdelta_step: dtype code %d", out_dtype);
  if (n_seqs > 65535) SB_FAIL(SB_ERR_UNSUPPORTED, "sb_gdelta_step: %d sequences", n_seqs);
  StepArgs a;
  a.proj = proj; a.ld = ld; a.q_off = q_off; a.a_off = a_off; a.b_off = b_off; a.g_off = g_off;
  a.n_heads = n_heads; a.n_kv_heads = n_kv_heads; a.dim = dim; a.vdim = vdim; a.taps = taps; a.conv_w = conv_w;
  a.a_log = a_log; a.dt_bias = dt_bias; a.row_pos = row_pos; a.seq_slot = seq_slot; a.ring = taps > 1 ? ring : nullptr;
  a.memory = memory; a.norm_w = norm_w; a.q_scale = q_scale; a.unit_eps = unit_eps; a.eps = eps; a.out_scale = out_scale;
  a.out = out; a.ld_out = ld_out; a.out_off = out_off;
  const int need = (dim + LANES - 1) / LANES;
  const int npl = need <= 2 ? 2 : need <= 4 ? 4 : need <= 8 ? 8 : need <= 16 ? 16 : need <= 32 ? 32 : 64;
  const size_t smem = ((size_t)2 * npl * LANES + 2 * vdim) * sizeof(float);        // at most 68 KiB
  const bool vec = dim % 4 == 0 && !((uintptr_t)memory & 15);
  const dim3 grid(n_heads, n_seqs);
  cudaError_t e = cudaSuccess;
#define SB_GD_STEP(N, VEC)                                                                                                      \
  do {                                                                                                                          \
    if (smem > 48 * 1024) e = cudaFuncSetAttribute(gdelta_step_kernel<N, VEC, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    if (e == cudaSuccess) e = sb_launch<SB_K_OTHER>(gdelta_step_kernel<N, VEC, TO>, grid, dim3(STEP_THREADS), smem, stream, a); \
  } while (0)
#define SB_GD_PICK(N)            \
  do {                           \
    if (vec) SB_GD_STEP(N, true); \
    else SB_GD_STEP(N, false);   \
  } while (0)
  SB_DISPATCH_DTYPE(out_dtype, TO, {
    switch (npl) {
      case 2: SB_GD_PICK(2); break;
      case 4: SB_GD_PICK(4); break;
      case 8: SB_GD_PICK(8); break;
      case 16: SB_GD_PICK(16); break;
      case 32: SB_GD_PICK(32); break;
      default: SB_GD_PICK(64); break;
    }
  });
#undef SB_GD_PICK
#undef SB_GD_STEP
  if (e != cudaSuccess) SB_FAIL(SB_ERR_CUDA, "sb_gdelta_step: launch failed: %s", cudaGetErrorString(e));
  return SB_OK;
}

extern "C" size_t sb_gdelta_mats_floats(int n_rows, int n_seqs, int n_heads) {
  return ((size_t)n_rows / TB + n_seqs) * n_heads * MATS;
}

extern "C" int sb_gdelta_prep(const float* proj, int n_rows, int ld, int q_off, int a_off, int b_off, int n_heads,
                              int n_kv_heads, int dim, int vdim, int taps, const float* conv_w, const float* a_log,
                              const float* dt_bias, int n_seqs, int max_new, const int32_t* seq_row0,
                              const int32_t* seq_pos0, const int32_t* seq_slot, const float* ring, float q_scale,
                              float unit_eps, float* act, float* mats, cudaStream_t stream) {
  if (int rc = check_sizes("sb_gdelta_prep", n_heads, n_kv_heads, dim, vdim, taps)) return rc;
  if (n_rows <= 0 || n_seqs <= 0 || max_new <= 0 || !proj || !conv_w || !a_log || !dt_bias || !seq_row0 || !seq_pos0 ||
      !seq_slot || (taps > 1 && !ring) || !act || !mats)
    SB_FAIL(SB_ERR_ARG, "sb_gdelta_prep: arguments missing (rows=%d seqs=%d)", n_rows, n_seqs);
  if (n_seqs > 65535 || n_kv_heads > 65535) SB_FAIL(SB_ERR_UNSUPPORTED, "sb_gdelta_prep: %d sequences, %d key heads", n_seqs, n_kv_heads);
  PrepArgs a;
  a.proj = proj; a.ld = ld; a.q_off = q_off; a.a_off = a_off; a.b_off = b_off; a.n_heads = n_heads; a.n_kv_heads = n_kv_heads;
  a.dim = dim; a.vdim = vdim; a.taps = taps; a.conv_w = conv_w; a.a_log = a_log; a.dt_bias = dt_bias; a.seq_row0 = seq_row0;
  a.seq_pos0 = seq_pos0; a.seq_slot = seq_slot; a.ring = taps > 1 ? ring : nullptr; a.q_scale = q_scale;
  a.unit_eps = unit_eps; a.act = act; a.mats = mats;
  const size_t smem = (size_t)2 * TB * ((dim + 3) / 4 * 4 + 4) * sizeof(float);
  const dim3 grid((max_new + TB - 1) / TB, n_kv_heads, n_seqs);
  cudaError_t e = cudaSuccess;
#define SB_GD_PREP(MAXT)                                                                                                        \
  do {                                                                                                                          \
    if (smem > 32 * 1024) e = cudaFuncSetAttribute(gdelta_prep_kernel<MAXT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    if (e == cudaSuccess) e = sb_launch<SB_K_ELEMENTWISE>(gdelta_prep_kernel<MAXT>, grid, dim3(PREP_THREADS), smem, stream, a); \
  } while (0)
  if (taps <= 4) SB_GD_PREP(4);
  else if (taps <= 8) SB_GD_PREP(8);
  else SB_GD_PREP(0);
#undef SB_GD_PREP
  if (e != cudaSuccess) SB_FAIL(SB_ERR_CUDA, "sb_gdelta_prep: launch failed: %s", cudaGetErrorString(e));
  return SB_OK;
}

extern "C" int sb_gdelta_scan(const float* act, const float* mats, const float* proj, int ld, int q_off, int n_heads,
                              int n_kv_heads, int dim, int vdim, int taps, int n_seqs, const int32_t* seq_row0,
                              const int32_t* seq_pos0, const int32_t* seq_slot, float* ring, float* memory, float* out,
                              cudaStream_t stream) {
  if (int rc = check_sizes("sb_gdelta_scan", n_heads, n_kv_heads, dim, vdim, taps)) return rc;
  if (n_seqs <= 0 || !act || !mats || !proj || !seq_row0 || !seq_pos0 || !seq_slot || (taps > 1 && !ring) || !memory || !out)
    SB_FAIL(SB_ERR_ARG, "sb_gdelta_scan: arguments missing (seqs=%d)", n_seqs);
  if (((uintptr_t)mats) & 15) SB_FAIL(SB_ERR_ARG, "sb_gdelta_scan: the chunk matrices must be 16-byte aligned");
  if (n_heads > 65535 || n_seqs > 65535) SB_FAIL(SB_ERR_UNSUPPORTED, "sb_gdelta_scan: %d heads, %d sequences", n_heads, n_seqs);
  ScanArgs a;
  a.act = act; a.mats = mats; a.proj = proj; a.ld = ld; a.q_off = q_off; a.n_heads = n_heads; a.n_kv_heads = n_kv_heads;
  a.dim = dim; a.vdim = vdim; a.taps = taps; a.seq_row0 = seq_row0; a.seq_pos0 = seq_pos0; a.seq_slot = seq_slot;
  a.ring = taps > 1 ? ring : nullptr; a.memory = memory; a.out = out;
  const bool vec = dim % 4 == 0 && vdim % 4 == 0 && !(((uintptr_t)act | (uintptr_t)out) & 15);
  const int need = (dim + SCAN_LANES - 1) / SCAN_LANES;
  cudaError_t e;
#define SB_GD_SCAN(N) e = vec ? launch_scan<N, true>(a, n_seqs, stream) : launch_scan<N, false>(a, n_seqs, stream)
  if (need <= 2) SB_GD_SCAN(2);
  else if (need <= 4) SB_GD_SCAN(4);
  else if (need <= 8) SB_GD_SCAN(8);
  else if (need <= 16) SB_GD_SCAN(16);
  else SB_GD_SCAN(32);
#undef SB_GD_SCAN
  if (e != cudaSuccess) SB_FAIL(SB_ERR_CUDA, "sb_gdelta_scan: launch failed: %s", cudaGetErrorString(e));
  return SB_OK;
}

// For measurements and tests: 2 or 4 columns per thread for every call (where the sizes allow four), 0 by the sizes again.
extern "C" void sb_gdelta_force_columns(int cpt) { g_force_cpt = cpt == 2 || cpt == 4 ? cpt : 0; }
