// The gated delta rule of the decoder models around its recurrence: short convolutions with silu, unit-norm factors
// and gates of a step's rows (prepare), the recurrence in fp32 arithmetic for any head size (scan), and the whole
// mixer of a single token in one launch (step).
//
// The convolutions' state is a table of raw inputs by position mod taps: a token's own slot is the one of the token
// `taps` places back, which nobody reads any more, so in the step kernel every CTA of a sequence may read the state
// while one of them stores the new input.  A sequence's first token needs nothing cleared: positions before zero are
// not read.
#include "common.cuh"
#include "../../include/atma_decoder.h"
#include "delta_rule.cuh"

namespace atma {

namespace {

__device__ __forceinline__ float silu(float x) { return x / (1.0f + expf(-x)); }
// for results that are rounded to 16 bits anyway: the fast exponential and division (a few fp32 units in the last place)
template <typename T>
__device__ __forceinline__ float silu_for(float x) {
  if constexpr (sizeof(T) == 2) {
    float e, r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(-1.4426950408889634f * x));
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.0f + e));        // infinity -> 0
    return x * r;
  } else {
    return silu(x);
  }
}
__device__ __forceinline__ float sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplus(float x) { return x > 0.f ? x + log1pf(expf(-x)) : log1pf(expf(x)); }


// ---- prepare: one warp = one head of q, k or v (or the gates of all heads) over a run of rows -------------
constexpr int kRunShort = 16, kRunLong = 64;           // rows per warp: short steps need the parallelism
constexpr int kLongRows = 16384;

template <typename T, int CPL, int KT>
__global__ void __launch_bounds__(128)
delta_prepare_kernel(const atma_delta_args a, T* __restrict__ qo, T* __restrict__ ko, T* __restrict__ vo, float* __restrict__ q_inv,
                     float* __restrict__ k_inv, float* __restrict__ log_decay, float* __restrict__ beta, int run) {
  const int lane = threadIdx.x & 31;
  const int units = 2 * a.G + a.H + 1;
  const int64_t wid = (int64_t)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int u = (int)(wid % units);
  const int64_t row0 = wid / units * run;
  if (row0 >= a.total_rows) return;
  const int row1 = (int)min((int64_t)a.total_rows, row0 + run);
  const T* Z = static_cast<const T*>(a.z);
  const int nq = a.G * a.dim, nv = a.H * a.vdim;
  if (u == units - 1) {                        // gates
    const int off = 2 * nq + 2 * nv;
    for (int64_t i = row0 * a.H + lane; i < (int64_t)row1 * a.H; i += 32) {
      const int64_t row = i / a.H;
      const int h = (int)(i - row * a.H);
      const T* zr = Z + row * a.z_rs + off;
      log_decay[i] = -expf(a.A_log[h]) * softplus(to_f32(zr[h]) + a.dt_bias[h]);
      beta[i] = sigmoid(to_f32(zr[a.H + h]));
    }
    return;
  }
  const int part = u < a.G ? 0 : (u < 2 * a.G ? 1 : 2);
  const int head = part == 0 ? u : (part == 1 ? u - a.G : u - 2 * a.G);
  const int dim = part == 2 ? a.vdim : a.dim;
  const int heads = part == 2 ? a.H : a.G;
  const int zoff = part * nq + head * dim;                    // channel inside a z row = channel inside the conv table
  const T* W = static_cast<const T*>(part == 0 ? a.conv_q : (part == 1 ? a.conv_k : a.conv_v)) + (int64_t)head * dim * a.taps;
  T* dst = part == 0 ? qo : (part == 1 ? ko : vo);
  const int ctot = 2 * nq + nv;
  const T* table = static_cast<const T*>(a.conv_table);
  const int c0 = lane * CPL;
  const bool full = c0 + CPL <= dim && dim % CPL == 0;        // the lane's channels as one vector access
  const int taps = KT > 0 ? KT : a.taps;

  struct alignas(CPL * sizeof(T)) Vec { T e[CPL]; };
  auto load = [&](const T* p, float (&x)[CPL]) {
    // element-wise where a vector access could be misaligned; CPL is chosen so that the common shapes are not
    if (full && (reinterpret_cast<uintptr_t>(p) & (sizeof(Vec) - 1)) == 0) {
      const Vec v = *reinterpret_cast<const Vec*>(p);
#pragma unroll
      for (int i = 0; i < CPL; ++i) x[i] = to_f32(v.e[i]);
    } else {
#pragma unroll
      for (int i = 0; i < CPL; ++i) x[i] = c0 + i < dim ? to_f32(p[i]) : 0.f;
    }
  };
  // raw input of the row's sequence `back` tokens before `row`
  auto fetch = [&](int row, int back, int first_row, int start, int64_t slot, float (&x)[CPL]) {
    const int src = row - back;
    if (src >= first_row) { load(Z + (int64_t)src * a.z_rs + zoff + c0, x); return; }
    const int pos = start + (src - first_row);
    if (pos >= 0 && slot >= 0) { load(table + slot * a.conv_ss + (int64_t)(pos % taps) * ctot + zoff + c0, x); return; }
#pragma unroll
    for (int i = 0; i < CPL; ++i) x[i] = 0.f;
  };
  constexpr int KW = KT > 0 ? KT : 1;
  float w[KW][CPL], win[KW][CPL];
  if constexpr (KT > 0) {
#pragma unroll
    for (int j = 0; j < KT; ++j)
#pragma unroll
      for (int i = 0; i < CPL; ++i) w[j][i] = c0 + i < dim ? to_f32(W[(int64_t)(c0 + i) * KT + j]) : 0.f;
  }
  // U output rows from their convolution sums
  auto finish = [&](int row, auto& acc) {
    constexpr int U = sizeof(acc) / sizeof(acc[0]);
    float ss[U];
#pragma unroll
    for (int r = 0; r < U; ++r) {
      T* op = dst + ((int64_t)(row + r) * heads + head) * dim + c0;
      Vec o;
      ss[r] = 0.f;
#pragma unroll
      for (int i = 0; i < CPL; ++i) {
        o.e[i] = from_f32<T>(silu_for<T>(acc[r][i]));
        const float f = c0 + i < dim ? to_f32(o.e[i]) : 0.f;
        ss[r] = fmaf(f, f, ss[r]);
      }
      if (full && (reinterpret_cast<uintptr_t>(op) & (sizeof(Vec) - 1)) == 0) {
        *reinterpret_cast<Vec*>(op) = o;
      } else {
#pragma unroll
        for (int i = 0; i < CPL; ++i)
          if (c0 + i < dim) op[i] = o.e[i];
      }
    }
    if (part < 2) {
#pragma unroll
      for (int sft = 16; sft > 0; sft >>= 1)
#pragma unroll
        for (int r = 0; r < U; ++r) ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], sft);
      float mine = ss[0];
#pragma unroll
      for (int r = 1; r < U; ++r) mine = lane == r ? ss[r] : mine;
      if (lane < U) {
        const float inv = 1.0f / sqrtf(mine + a.unit_eps);
        if (part == 0) q_inv[(int64_t)(row + lane) * a.G + head] = inv * a.q_scale;
        else k_inv[(int64_t)(row + lane) * a.G + head] = inv;
      }
    }
  };
  for (int row = (int)row0; row < row1;) {
    const int seq = a.row_seq[row];
    const int first_row = a.cu_rows[seq], start = a.start_pos[seq], end = min(row1, a.cu_rows[seq + 1]);
    const int64_t slot = a.slots[seq];
    if constexpr (KT > 0) {
#pragma unroll
      for (int j = 0; j + 1 < KT; ++j) fetch(row, KT - 1 - j, first_row, start, slot, win[j]);
      constexpr int U = 4;                                      // rows requested together, one group ahead
      float nxt[U][CPL];
      auto request = [&](int r0) {
#pragma unroll
        for (int r = 0; r < U; ++r) load(Z + (int64_t)min(r0 + r, end - 1) * a.z_rs + zoff + c0, nxt[r]);
      };
      if (row + U <= end) request(row);
      for (; row + U <= end; row += U) {
        float x[KT - 1 + U][CPL], acc[U][CPL];
#pragma unroll
        for (int j = 0; j + 1 < KT; ++j)
#pragma unroll
          for (int i = 0; i < CPL; ++i) x[j][i] = win[j][i];
#pragma unroll
        for (int r = 0; r < U; ++r)
#pragma unroll
          for (int i = 0; i < CPL; ++i) x[KT - 1 + r][i] = nxt[r][i];
        if (row + 2 * U <= end) request(row + U);
#pragma unroll
        for (int r = 0; r < U; ++r)
#pragma unroll
          for (int i = 0; i < CPL; ++i) {
            acc[r][i] = 0.f;
#pragma unroll
            for (int j = 0; j < KT; ++j) acc[r][i] = fmaf(x[r + j][i], w[j][i], acc[r][i]);
          }
        finish(row, acc);
#pragma unroll
        for (int j = 0; j + 1 < KT; ++j)
#pragma unroll
          for (int i = 0; i < CPL; ++i) win[j][i] = x[U + j][i];
      }
      for (; row < end; ++row) {
        float acc[1][CPL] = {};
        load(Z + (int64_t)row * a.z_rs + zoff + c0, win[KT - 1]);
#pragma unroll
        for (int j = 0; j < KT; ++j)
#pragma unroll
          for (int i = 0; i < CPL; ++i) acc[0][i] = fmaf(win[j][i], w[j][i], acc[0][i]);
#pragma unroll
        for (int j = 0; j + 1 < KT; ++j)
#pragma unroll
          for (int i = 0; i < CPL; ++i) win[j][i] = win[j + 1][i];
        finish(row, acc);
      }
    } else {
      for (; row < end; ++row) {
        float acc[1][CPL] = {};
        for (int j = 0; j < taps; ++j) {
          float x[CPL];
          fetch(row, taps - 1 - j, first_row, start, slot, x);
#pragma unroll
          for (int i = 0; i < CPL; ++i)
            if (c0 + i < dim) acc[0][i] = fmaf(x[i], to_f32(W[(int64_t)(c0 + i) * taps + j]), acc[0][i]);
        }
        finish(row, acc);
      }
    }
  }
}

// The same where every access is one aligned vector of CPL channels: rows travel in raw form a group of eight ahead, sums
// are formed on channel pairs (two fp32 lanes per instruction), pointers advance by row.
template <typename T, int CPL, int KT>
__global__ void __launch_bounds__(128)
delta_prepare_vec_kernel(const atma_delta_args a, T* __restrict__ qo, T* __restrict__ ko, T* __restrict__ vo, float* __restrict__ q_inv,
                         float* __restrict__ k_inv, int run) {
  struct alignas(CPL * sizeof(T)) Vec { T e[CPL]; };
  constexpr int P = CPL / 2, U = 4, N = 2 * U;
  const int lane = threadIdx.x & 31;
  const int units = 2 * a.G + a.H;
  const int64_t wid = (int64_t)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int u = (int)(wid % units);
  const int64_t row0 = wid / units * run;
  if (row0 >= a.total_rows) return;
  const int row1 = (int)min((int64_t)a.total_rows, row0 + run);
  const int nq = a.G * a.dim;
  const int part = u < a.G ? 0 : (u < 2 * a.G ? 1 : 2);
  const int head = part == 0 ? u : (part == 1 ? u - a.G : u - 2 * a.G);
  const int dim = part == 2 ? a.vdim : a.dim, heads = part == 2 ? a.H : a.G;
  const bool on = lane * CPL < dim;                             // the lanes past the head's channels work on its first ones
  const int c0 = on ? lane * CPL : 0;
  const int zc = part * nq + head * dim + c0;
  const int ctot = 2 * nq + a.H * a.vdim;
  const T* zcol = static_cast<const T*>(a.z) + zc;
  const T* table = static_cast<const T*>(a.conv_table) + zc;
  T* dst = (part == 0 ? qo : (part == 1 ? ko : vo)) + head * dim + c0;
  float* inv_out = part == 0 ? q_inv : k_inv;
  const float inv_scale = part == 0 ? a.q_scale : 1.0f;
  const int orow = heads * dim;
  float2 w[KT][P];
  {
    const T* W = static_cast<const T*>(part == 0 ? a.conv_q : (part == 1 ? a.conv_k : a.conv_v)) + ((int64_t)head * dim + c0) * KT;
#pragma unroll
    for (int j = 0; j < KT; ++j)
#pragma unroll
      for (int i = 0; i < P; ++i) w[j][i] = make_float2(to_f32(W[(2 * i) * KT + j]), to_f32(W[(2 * i + 1) * KT + j]));
  }
  auto unpack = [&](const Vec& x, float2 (&f)[P]) {
#pragma unroll
    for (int i = 0; i < P; ++i) f[i] = make_float2(to_f32(x.e[2 * i]), to_f32(x.e[2 * i + 1]));
  };
  for (int row = (int)row0; row < row1;) {
    const int seq = a.row_seq[row];
    const int first_row = a.cu_rows[seq], start = a.start_pos[seq], end = min(row1, a.cu_rows[seq + 1]);
    const int64_t slot = a.slots[seq];
    float2 win[KT - 1][P];
#pragma unroll
    for (int j = 0; j + 1 < KT; ++j) {
      const int src = row - (KT - 1 - j), pos = start + (src - first_row);
#pragma unroll
      for (int i = 0; i < P; ++i) win[j][i] = make_float2(0.f, 0.f);
      if (src >= first_row) unpack(*reinterpret_cast<const Vec*>(zcol + (int64_t)src * a.z_rs), win[j]);
      else if (pos >= 0 && slot >= 0) unpack(*reinterpret_cast<const Vec*>(table + slot * a.conv_ss + (int64_t)(pos % KT) * ctot), win[j]);
    }
    const T* zp = zcol + (int64_t)row * a.z_rs;                 // the next row to request
    T* op = dst + (int64_t)row * orow;
    const int n = end - row;
    Vec raw[N], nxt[N];
#pragma unroll
    for (int r = 0; r < N; ++r)
      if (r < n) nxt[r] = *reinterpret_cast<const Vec*>(zp + (int64_t)r * a.z_rs);
    for (int at = 0; at < n; at += N) {
#pragma unroll
      for (int r = 0; r < N; ++r) raw[r] = nxt[r];
      zp += (int64_t)N * a.z_rs;
#pragma unroll
      for (int r = 0; r < N; ++r)
        if (at + N + r < n) nxt[r] = *reinterpret_cast<const Vec*>(zp + (int64_t)r * a.z_rs);
#pragma unroll
      for (int g = 0; g < 2; ++g) {
        float ss[U];
#pragma unroll
        for (int r = 0; r < U; ++r) {
          float2 cur[P];
          unpack(raw[g * U + r], cur);
          Vec o;
          ss[r] = 0.f;
#pragma unroll
          for (int i = 0; i < P; ++i) {
            float2 acc = make_float2(0.f, 0.f);
#pragma unroll
            for (int j = 0; j + 1 < KT; ++j) acc = __ffma2_rn(win[j][i], w[j][i], acc);
            acc = __ffma2_rn(cur[i], w[KT - 1][i], acc);
            o.e[2 * i] = from_f32<T>(silu_for<T>(acc.x));
            o.e[2 * i + 1] = from_f32<T>(silu_for<T>(acc.y));
            const float x = to_f32(o.e[2 * i]), y = to_f32(o.e[2 * i + 1]);
            ss[r] = fmaf(x, x, fmaf(y, y, ss[r]));
#pragma unroll
            for (int j = 0; j + 2 < KT; ++j) win[j][i] = win[j + 1][i];
            win[KT - 2][i] = cur[i];
          }
          if (on && at + g * U + r < n) *reinterpret_cast<Vec*>(op) = o;
          op += orow;
          if (!on) ss[r] = 0.f;
        }
        if (part < 2) {
#pragma unroll
          for (int sft = 16; sft > 0; sft >>= 1)
#pragma unroll
            for (int r = 0; r < U; ++r) ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], sft);
          float mine = ss[0];
#pragma unroll
          for (int r = 1; r < U; ++r) mine = lane == r ? ss[r] : mine;
          const int rr = at + g * U + lane;
          if (lane < U && rr < n) inv_out[(int64_t)(row + rr) * a.G + head] = inv_scale / sqrtf(mine + a.unit_eps);
        }
      }
    }
    row = end;
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
delta_gates_kernel(const atma_delta_args a, float* __restrict__ log_decay, float* __restrict__ beta) {
  const int64_t i = (int64_t)blockIdx.x * 256 + threadIdx.x;
  if (i >= (int64_t)a.total_rows * a.H) return;
  const int64_t row = i / a.H;
  const int h = (int)(i - row * a.H);
  const T* zr = static_cast<const T*>(a.z) + row * a.z_rs + 2 * a.G * a.dim + 2 * a.H * a.vdim;
  log_decay[i] = -expf(a.A_log[h]) * softplus(to_f32(zr[h]) + a.dt_bias[h]);
  beta[i] = sigmoid(to_f32(zr[a.H + h]));
}

// The last `taps` inputs of every sequence into the table (its own launch: the rows above still read the old ones).
template <typename T>
__global__ void __launch_bounds__(256)
delta_conv_state_kernel(const atma_delta_args a, int ctot) {
  const int s = blockIdx.y;
  const int c = blockIdx.x * 256 + threadIdx.x;
  const int64_t slot = a.slots[s];
  if (c >= ctot || slot < 0) return;
  const int r0 = a.cu_rows[s], n = a.cu_rows[s + 1] - r0, start = a.start_pos[s];
  if (start < 0) return;
  T* table = static_cast<T*>(a.conv_table) + slot * a.conv_ss;
  for (int i = max(0, n - a.taps); i < n; ++i)
    table[(int64_t)((start + i) % a.taps) * ctot + c] = static_cast<const T*>(a.z)[(int64_t)(r0 + i) * a.z_rs + c];
}

// ---- scan: a warp owns four value columns of one head's state, its lanes the key rows -------------------------------
constexpr int kScanWarps = 8, kScanCols = 4;

template <typename T, int RPL>
__global__ void __launch_bounds__(kScanWarps * 32)
delta_scan_kernel(const atma_delta_args a, const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v,
                  const float* __restrict__ q_inv, const float* __restrict__ k_inv, const float* __restrict__ log_decay,
                  const float* __restrict__ beta, T* __restrict__ o) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int h = blockIdx.y, s = blockIdx.z;
  const int col = (blockIdx.x * kScanWarps + warp) * kScanCols;
  if (col >= a.vdim) return;
  const int g = h / (a.H / a.G);
  const int r0 = a.cu_rows[s], r1 = a.cu_rows[s + 1], start = a.start_pos[s];
  const int64_t slot = a.slots[s];
  if (start < 0 || slot < 0) {
    for (int r = r0; r < r1; ++r)
      if (lane < kScanCols && col + lane < a.vdim) o[((int64_t)r * a.H + h) * a.vdim + col + lane] = from_f32<T>(0.f);
    return;
  }
  float* sp = a.state_table + slot * a.state_ss + (int64_t)h * a.dim * a.vdim + col;
  float S[RPL][kScanCols];
#pragma unroll
  for (int i = 0; i < RPL; ++i)
#pragma unroll
    for (int j = 0; j < kScanCols; ++j) {
      const int row = lane + 32 * i;
      S[i][j] = (start > 0 && row < a.dim && col + j < a.vdim) ? sp[(int64_t)row * a.vdim + j] : 0.f;
    }
  float kn[RPL], qn[RPL], vn[kScanCols], ki = 0.f, qi = 0.f, ld = 0.f, bt = 0.f;      // the next row, one ahead
  auto fetch = [&](int r) {
    const T* kr = k + ((int64_t)r * a.G + g) * a.dim;
    const T* qr = q + ((int64_t)r * a.G + g) * a.dim;
    const T* vr = v + ((int64_t)r * a.H + h) * a.vdim + col;
#pragma unroll
    for (int i = 0; i < RPL; ++i) {
      const int c = lane + 32 * i;
      kn[i] = c < a.dim ? to_f32(kr[c]) : 0.f;
      qn[i] = c < a.dim ? to_f32(qr[c]) : 0.f;
    }
#pragma unroll
    for (int j = 0; j < kScanCols; ++j) vn[j] = col + j < a.vdim ? to_f32(vr[j]) : 0.f;
    ki = k_inv[(int64_t)r * a.G + g]; qi = q_inv[(int64_t)r * a.G + g];
    ld = log_decay[(int64_t)r * a.H + h]; bt = beta[(int64_t)r * a.H + h];
  };
  if (r0 < r1) fetch(r0);
  for (int r = r0; r < r1; ++r) {
    float kk[RPL], qq[RPL], vv[kScanCols];
#pragma unroll
    for (int i = 0; i < RPL; ++i) { kk[i] = kn[i] * ki; qq[i] = qn[i] * qi; }
#pragma unroll
    for (int j = 0; j < kScanCols; ++j) vv[j] = vn[j];
    const float gm = expf(ld), b = bt;
    if (r + 1 < r1) fetch(r + 1);
    float pred[kScanCols] = {}, out[kScanCols] = {};
#pragma unroll
    for (int i = 0; i < RPL; ++i)
#pragma unroll
      for (int j = 0; j < kScanCols; ++j) { S[i][j] *= gm; pred[j] = fmaf(S[i][j], kk[i], pred[j]); }
#pragma unroll
    for (int j = 0; j < kScanCols; ++j) pred[j] = b * (vv[j] - warp_sum(pred[j]));
#pragma unroll
    for (int i = 0; i < RPL; ++i)
#pragma unroll
      for (int j = 0; j < kScanCols; ++j) { S[i][j] = fmaf(kk[i], pred[j], S[i][j]); out[j] = fmaf(S[i][j], qq[i], out[j]); }
#pragma unroll
    for (int j = 0; j < kScanCols; ++j) out[j] = warp_sum(out[j]);
    float mine = out[0];
#pragma unroll
    for (int j = 1; j < kScanCols; ++j) mine = lane == j ? out[j] : mine;
    if (lane < kScanCols && col + lane < a.vdim) o[((int64_t)r * a.H + h) * a.vdim + col + lane] = from_f32<T>(mine);
  }
#pragma unroll
  for (int i = 0; i < RPL; ++i)
#pragma unroll
    for (int j = 0; j < kScanCols; ++j) {
      const int row = lane + 32 * i;
      if (row < a.dim && col + j < a.vdim) sp[(int64_t)row * a.vdim + j] = S[i][j];
    }
}

// ---- step: one CTA per (sequence, head) -----------------------------------------------------------------------------
// Warp w holds rows w, w + 8, ... of the state plane, lane l the VEC columns VEC * l of a block of 32 * VEC columns; the
// first block's loads are in flight while the convolutions run.
constexpr int kStepWarps = 8;

template <typename T, int VEC, int RPW, int TAPS>             // TAPS 0: any number
__global__ void __launch_bounds__(kStepWarps * 32)
delta_step_kernel(const atma_delta_args a, const T* __restrict__ norm_w, T* __restrict__ out, int64_t out_rs, float eps) {
  extern __shared__ float sm[];
  const int K = a.dim, V = a.vdim;
  float* s_q = sm;                              // [K]
  float* s_k = s_q + K;                         // [K]
  float* s_v = s_k + K;                         // [V]
  float* s_o = s_v + V;                         // [V]
  __shared__ __align__(16) float s_red[kStepWarps][32 * VEC];
  __shared__ float s_sum[3][kStepWarps];
  const int b = blockIdx.y, h = blockIdx.x;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int rep = a.H / a.G, g = h / rep;
  const int64_t slot = a.slots[b];
  const int pos = a.start_pos[b];
  T* orow = out + b * out_rs + (int64_t)h * V;
  if (slot < 0 || pos < 0) {
    for (int c = tid; c < V; c += kStepWarps * 32) orow[c] = from_f32<T>(0.f);
    return;
  }
  float* sp = a.state_table + slot * a.state_ss + (int64_t)h * K * V;
  struct alignas(VEC * 4) FV { float e[VEC]; };
  FV S[RPW];
  const int cblocks = (V + 32 * VEC - 1) / (32 * VEC);
  auto load_state = [&](int cb) {
    const int c = cb * 32 * VEC + lane * VEC;
#pragma unroll
    for (int i = 0; i < RPW; ++i) {
      const int r = warp + kStepWarps * i;
      if (pos > 0 && r < K && c < V) S[i] = *reinterpret_cast<const FV*>(sp + (int64_t)r * V + c);
      else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) S[i].e[e] = 0.f;
      }
    }
  };
  load_state(0);

  // convolutions of this head's q, k and v channels
  const int nq = a.G * K, ctot = 2 * nq + a.H * V, taps = TAPS > 0 ? TAPS : a.taps;
  const T* zr = static_cast<const T*>(a.z) + b * a.z_rs;
  T* table = static_cast<T*>(a.conv_table) + slot * a.conv_ss;
  const int ring = pos % taps;
  const int goff = 2 * nq + 2 * a.H * V;
  const float za = to_f32(zr[goff + h]), zb = to_f32(zr[goff + a.H + h]), alog = a.A_log[h], dtb = a.dt_bias[h];
  float gate_c = 0.f, norm_c = 0.f;              // V <= 256: one output channel per thread
  if (tid < V) { gate_c = to_f32(zr[2 * nq + a.H * V + h * V + tid]); norm_c = to_f32(norm_w[tid]); }
  constexpr int kRounds = 3, TA = TAPS > 0 ? TAPS : 1;           // 2 K + V <= 768 channels
  float qs = 0.f, ks = 0.f;
  float hist[kRounds][TA], wt[kRounds][TA];
  auto locate = [&](int i, int& part, int& c, int& pc, int& zc) {
    part = i < K ? 0 : (i < 2 * K ? 1 : 2);
    c = i - part * K;
    pc = part < 2 ? g * K + c : h * V + c;                        // channel inside the part
    zc = part * nq + pc;
  };
  if constexpr (TAPS > 0) {                                        // everything requested before the first use
#pragma unroll
    for (int r = 0; r < kRounds; ++r) {
      const int i = tid + r * kStepWarps * 32;
      if (i >= 2 * K + V) continue;
      int part, c, pc, zc;
      locate(i, part, c, pc, zc);
      const T* w = static_cast<const T*>(part == 0 ? a.conv_q : (part == 1 ? a.conv_k : a.conv_v)) + (int64_t)pc * TAPS;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        wt[r][j] = to_f32(w[TAPS - 1 - j]);
        const int at = ring - j + (ring < j ? TAPS : 0);
        hist[r][j] = j == 0 ? to_f32(zr[zc]) : (pos >= j ? to_f32(table[(int64_t)at * ctot + zc]) : 0.f);
      }
    }
  }
#pragma unroll
  for (int r = 0; r < kRounds; ++r) {
    const int i = tid + r * kStepWarps * 32;
    if (i >= 2 * K + V) continue;
    int part, c, pc, zc;
    locate(i, part, c, pc, zc);
    float acc = 0.f;
    if constexpr (TAPS > 0) {
#pragma unroll
      for (int j = 0; j < TAPS; ++j) acc = fmaf(hist[r][j], wt[r][j], acc);
    } else {
      const T* w = static_cast<const T*>(part == 0 ? a.conv_q : (part == 1 ? a.conv_k : a.conv_v)) + (int64_t)pc * taps;
      acc = to_f32(zr[zc]) * to_f32(w[taps - 1]);
      for (int j = 1; j < taps; ++j)
        if (pos >= j) acc = fmaf(to_f32(table[(int64_t)(ring - j + (ring < j ? taps : 0)) * ctot + zc]), to_f32(w[taps - 1 - j]), acc);
    }
    if (part == 2 || h % rep == 0) table[(int64_t)ring * ctot + zc] = zr[zc];
    const float y = round_through<T>(silu_for<T>(acc));
    if (part == 0) { s_q[c] = y; qs = fmaf(y, y, qs); }
    else if (part == 1) { s_k[c] = y; ks = fmaf(y, y, ks); }
    else s_v[c] = y;
  }
  qs = warp_sum(qs); ks = warp_sum(ks);
  if (lane == 0) { s_sum[0][warp] = qs; s_sum[1][warp] = ks; }
  const float gm = expf(-expf(alog) * softplus(za + dtb));
  const float bt = sigmoid(zb);
  __syncthreads();
  qs = 0.f; ks = 0.f;
#pragma unroll
  for (int i = 0; i < kStepWarps; ++i) { qs += s_sum[0][i]; ks += s_sum[1][i]; }
  const float qi = a.q_scale / sqrtf(qs + a.unit_eps), ki = 1.0f / sqrtf(ks + a.unit_eps);

  float osq = 0.f;
  for (int cb = 0; cb < cblocks; ++cb) {
    if (cb > 0) load_state(cb);
    const int c = cb * 32 * VEC + lane * VEC;
    alignas(16) float p[VEC] = {};
#pragma unroll
    for (int i = 0; i < RPW; ++i) {
      const int r = warp + kStepWarps * i;
      const float kn = r < K ? s_k[r] * ki : 0.f;
#pragma unroll
      for (int e = 0; e < VEC; ++e) { S[i].e[e] *= gm; p[e] = fmaf(kn, S[i].e[e], p[e]); }
    }
    __syncthreads();                            // s_red is free again
    *reinterpret_cast<FV*>(&s_red[warp][lane * VEC]) = *reinterpret_cast<const FV*>(p);
    __syncthreads();
    alignas(16) float rd[VEC] = {};
    float u[VEC] = {};
#pragma unroll
    for (int w = 0; w < kStepWarps; ++w) {
      const FV t = *reinterpret_cast<const FV*>(&s_red[w][lane * VEC]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) u[e] += t.e[e];
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) u[e] = c + e < V ? bt * (s_v[c + e] - u[e]) : 0.f;
#pragma unroll
    for (int i = 0; i < RPW; ++i) {
      const int r = warp + kStepWarps * i;
      if (r < K && c < V) {
        const float kn = s_k[r] * ki, qn = s_q[r] * qi;
#pragma unroll
        for (int e = 0; e < VEC; ++e) { S[i].e[e] = fmaf(kn, u[e], S[i].e[e]); rd[e] = fmaf(qn, S[i].e[e], rd[e]); }
        *reinterpret_cast<FV*>(sp + (int64_t)r * V + c) = S[i];
      }
    }
    __syncthreads();
    *reinterpret_cast<FV*>(&s_red[warp][lane * VEC]) = *reinterpret_cast<const FV*>(rd);
    __syncthreads();
    if (tid < 32 * VEC) {
      const int cc = cb * 32 * VEC + tid;
      float t = 0.f;
#pragma unroll
      for (int w = 0; w < kStepWarps; ++w) t += s_red[w][tid];
      if (cc < V) { s_o[cc] = t; osq = fmaf(t, t, osq); }
    }
  }
  osq = warp_sum(osq);
  if (lane == 0) s_sum[2][warp] = osq;
  __syncthreads();
  osq = 0.f;
#pragma unroll
  for (int i = 0; i < kStepWarps; ++i) osq += s_sum[2][i];
  const float rs = 1.0f / sqrtf(osq / (float)V + eps);
  if (tid < V) orow[tid] = from_f32<T>(s_o[tid] * rs * norm_c * silu_for<T>(gate_c));
}

int check(const atma_delta_args* a, const char* what) {
  ATMA_REQUIRE(a != nullptr, "%s: null args", what);
  ATMA_REQUIRE(a->dtype == ATMA_F32 || a->dtype == ATMA_BF16, "%s: unsupported dtype %d", what, a->dtype);
  ATMA_REQUIRE(a->H > 0 && a->G > 0 && a->H % a->G == 0, "%s: %d heads over %d q/k heads", what, a->H, a->G);
  ATMA_REQUIRE(a->dim > 0 && a->dim <= 256, "%s: key size %d outside 1..256", what, a->dim);
  ATMA_REQUIRE(a->vdim > 0 && a->vdim <= 256, "%s: value size %d outside 1..256", what, a->vdim);
  ATMA_REQUIRE(a->taps >= 1, "%s: %d convolution taps", what, a->taps);
  ATMA_REQUIRE(a->H <= 65535 && a->n_seqs <= 65535, "%s: grid limits", what);
  return ATMA_OK;
}

template <typename T, int CPL>
int launch_prepare(const atma_delta_args& a, void* q, void* k, void* v, float* qi, float* ki, float* ld, float* bt, cudaStream_t st) {
  const int run = a.total_rows >= kLongRows ? kRunLong : kRunShort;
  const int64_t warps = (int64_t)((a.total_rows + run - 1) / run) * (2 * a.G + a.H + 1);
  const unsigned grid = (unsigned)((warps + 3) / 4);
  auto al = [](const void* ptr) { return (reinterpret_cast<uintptr_t>(ptr) & 15) == 0; };
  if constexpr (CPL > 1) {
    if (a.taps >= 2 && a.taps <= 4 && a.dim % CPL == 0 && a.vdim % CPL == 0 && a.z_rs % CPL == 0 && a.conv_ss % CPL == 0 && al(a.z) &&
        al(a.conv_table) && al(q) && al(k) && al(v)) {
      const unsigned vgrid = (unsigned)(((int64_t)((a.total_rows + run - 1) / run) * (2 * a.G + a.H) + 3) / 4);
#define ATMA_PREPV(KT) delta_prepare_vec_kernel<T, CPL, KT><<<vgrid, 128, 0, st>>>(a, (T*)q, (T*)k, (T*)v, qi, ki, run)
      if (a.taps == 2) ATMA_PREPV(2); else if (a.taps == 3) ATMA_PREPV(3); else ATMA_PREPV(4);
#undef ATMA_PREPV
      delta_gates_kernel<T><<<(unsigned)(((int64_t)a.total_rows * a.H + 255) / 256), 256, 0, st>>>(a, ld, bt);
      const int ct = 2 * a.G * a.dim + a.H * a.vdim;
      delta_conv_state_kernel<T><<<dim3((ct + 255) / 256, a.n_seqs), 256, 0, st>>>(a, ct);
      return launch_status("delta_prepare");
    }
  }
#define ATMA_PREP(KT) delta_prepare_kernel<T, CPL, KT><<<grid, 128, 0, st>>>(a, (T*)q, (T*)k, (T*)v, qi, ki, ld, bt, run)
  switch (a.taps) {
    case 2: ATMA_PREP(2); break;
    case 3: ATMA_PREP(3); break;
    case 4: ATMA_PREP(4); break;
    default: ATMA_PREP(0); break;
  }
#undef ATMA_PREP
  const int ctot = 2 * a.G * a.dim + a.H * a.vdim;
  delta_conv_state_kernel<T><<<dim3((ctot + 255) / 256, a.n_seqs), 256, 0, st>>>(a, ctot);
  return launch_status("delta_prepare");
}

template <typename T>
int prepare_t(const atma_delta_args& a, void* q, void* k, void* v, float* qi, float* ki, float* ld, float* bt, cudaStream_t st) {
  const int d = a.dim > a.vdim ? a.dim : a.vdim;
  if (d <= 32) return launch_prepare<T, 1>(a, q, k, v, qi, ki, ld, bt, st);
  if (d <= 64) return launch_prepare<T, 2>(a, q, k, v, qi, ki, ld, bt, st);
  if (d <= 128) return launch_prepare<T, 4>(a, q, k, v, qi, ki, ld, bt, st);
  return launch_prepare<T, 8>(a, q, k, v, qi, ki, ld, bt, st);
}

template <typename T>
int scan_t(const atma_delta_args& a, const void* q, const void* k, const void* v, const float* qi, const float* ki, const float* ld,
           const float* bt, void* o, cudaStream_t st) {
  const dim3 grid((a.vdim + kScanWarps * kScanCols - 1) / (kScanWarps * kScanCols), a.H, a.n_seqs);
#define ATMA_SCAN(R) delta_scan_kernel<T, R><<<grid, kScanWarps * 32, 0, st>>>(a, (const T*)q, (const T*)k, (const T*)v, qi, ki, ld, bt, (T*)o)
  if (a.dim <= 32) ATMA_SCAN(1);
  else if (a.dim <= 64) ATMA_SCAN(2);
  else if (a.dim <= 128) ATMA_SCAN(4);
  else ATMA_SCAN(8);
#undef ATMA_SCAN
  return launch_status("delta_scan (fp32 arithmetic)");
}

template <typename T>
int step_t(const atma_delta_args& a, const void* w, void* out, int64_t out_rs, float eps, cudaStream_t st) {
  const dim3 grid(a.H, a.n_seqs);
  const int smem = (2 * a.dim + 2 * a.vdim) * 4;
  const bool vec = a.vdim % 4 == 0 && a.state_ss % 4 == 0 && (reinterpret_cast<uintptr_t>(a.state_table) & 15) == 0;
#define ATMA_STEPT(V, R, K) delta_step_kernel<T, V, R, K><<<grid, kStepWarps * 32, smem, st>>>(a, (const T*)w, (T*)out, out_rs, eps)
#define ATMA_STEP(V, R) do { if (a.taps == 4) ATMA_STEPT(V, R, 4); else ATMA_STEPT(V, R, 0); } while (0)
  if (vec) { if (a.dim <= 64) ATMA_STEP(4, 8); else if (a.dim <= 128) ATMA_STEP(4, 16); else ATMA_STEP(4, 32); }
  else { if (a.dim <= 64) ATMA_STEP(1, 8); else if (a.dim <= 128) ATMA_STEP(1, 16); else ATMA_STEP(1, 32); }
#undef ATMA_STEPT
#undef ATMA_STEP
  return launch_status("delta_step");
}

}  // namespace
}  // namespace atma

using namespace atma;

extern "C" int atma_delta_prepare(const atma_delta_args* a, void* q, void* k, void* v, float* q_inv, float* k_inv, float* log_decay,
                                  float* beta, void* stream) {
  int rc = check(a, "delta_prepare");
  if (rc != ATMA_OK) return rc;
  if (a->total_rows <= 0 || a->n_seqs <= 0) return ATMA_OK;
  cudaStream_t st = (cudaStream_t)stream;
  if (a->dtype == ATMA_F32) return prepare_t<float>(*a, q, k, v, q_inv, k_inv, log_decay, beta, st);
  return prepare_t<__nv_bfloat16>(*a, q, k, v, q_inv, k_inv, log_decay, beta, st);
}

extern "C" int atma_delta_scan_path(const atma_delta_args* a) { return a != nullptr && delta_scan_sm100_supported(*a) ? 1 : 0; }
extern "C" int64_t atma_delta_scan_scratch_bytes(const atma_delta_args* a) {
  return a != nullptr && delta_scan_sm100_supported(*a) ? delta_scan_sm100_scratch_bytes(*a) : 0;
}

extern "C" int atma_delta_scan(const atma_delta_args* a, const void* q, const void* k, const void* v, const float* q_inv,
                               const float* k_inv, const float* log_decay, const float* beta, void* o, void* scratch, void* stream) {
  int rc = check(a, "delta_scan");
  if (rc != ATMA_OK) return rc;
  if (a->total_rows <= 0 || a->n_seqs <= 0) return ATMA_OK;
  cudaStream_t st = (cudaStream_t)stream;
  if (delta_scan_sm100_supported(*a)) return delta_scan_sm100(*a, q, k, v, q_inv, k_inv, log_decay, beta, o, scratch, st);
  if (a->dtype == ATMA_F32) return scan_t<float>(*a, q, k, v, q_inv, k_inv, log_decay, beta, o, st);
  return scan_t<__nv_bfloat16>(*a, q, k, v, q_inv, k_inv, log_decay, beta, o, st);
}

extern "C" int atma_delta_step(const atma_delta_args* a, const void* norm_w, void* out, int64_t out_rs, float eps, void* stream) {
  int rc = check(a, "delta_step");
  if (rc != ATMA_OK) return rc;
  if (a->n_seqs <= 0) return ATMA_OK;
  if (a->dtype == ATMA_F32) return step_t<float>(*a, norm_w, out, out_rs, eps, (cudaStream_t)stream);
  return step_t<__nv_bfloat16>(*a, norm_w, out, out_rs, eps, (cudaStream_t)stream);
}
