// Short causal convolutions over time, channel by channel, that are linear (no activation):
//
//   tlc_rmsnorm_conv   h = x / sqrt(mean(x^2) + eps) * g;   out_t = h_t + sum_j w[:, j] h_(t - K + 1 + j)
//   tlc_channel_conv   y_t = sum_j w[:, j] u_(t - K + 1 + j) on a range of the columns of a 32-bit projection, the columns
//                      from mix_from on blended with another matrix: y <- (1 - lam) y + lam * first
//
// with zeros before a sequence's first row.  The last K - 1 rows that were convolved (normed rows, projected rows) are kept
// per sequence, 32-bit, in `state` [n_slots, K - 1, C]; a sequence at position 0 starts from zeros whatever its slot holds.
// Everything is 32-bit but the stored result.  Weights are laid out tap by tap, [K, C].
//
// Prompts: a block takes CONV_R consecutive packed rows; a thread walks them in order for its columns with the last
// K - 1 rows in registers (a rolling window), which it loads anew where a sequence begins.  After a sequence's last row the
// window IS the sequence's new state; the walking thread stores it, unless some sequence of the step goes on from an
// earlier step: another block may then still have to read the old state, and a kernel of its own stores the new one when
// every reader has finished.  One-token steps: a thread owns one column group of one sequence, reads its window before it
// waits for the previous kernel (an earlier step wrote it) and writes the shifted one back.
#include "common.cuh"

#define CONV_R 8             // rows a block of the prompt kernels takes
#define CONV_MAX_K 17        // taps at most

template <int V> struct Vec;
template <> struct Vec<1> {
  float v[1];
  static __device__ __forceinline__ Vec ld(const float* p) { Vec r; r.v[0] = *p; return r; }
  __device__ __forceinline__ void st(float* p) const { *p = v[0]; }
  __device__ __forceinline__ void st(__nv_bfloat16* p) const { *p = __float2bfloat16_rn(v[0]); }
};
template <> struct Vec<4> {
  float v[4];
  static __device__ __forceinline__ Vec ld(const float* p) {
    const float4 q = *reinterpret_cast<const float4*>(p);
    Vec r;
    r.v[0] = q.x; r.v[1] = q.y; r.v[2] = q.z; r.v[3] = q.w;
    return r;
  }
  __device__ __forceinline__ void st(float* p) const { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
  __device__ __forceinline__ void st(__nv_bfloat16* p) const {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    uint2 u;
    u.x = *reinterpret_cast<const unsigned*>(&lo);
    u.y = *reinterpret_cast<const unsigned*>(&hi);
    *reinterpret_cast<uint2*>(p) = u;
  }
};
template <int V> __device__ __forceinline__ Vec<V> vzero() {
  Vec<V> r;
#pragma unroll
  for (int e = 0; e < V; e++) r.v[e] = 0.f;
  return r;
}
template <int V> __device__ __forceinline__ void vfma(Vec<V>& acc, const Vec<V>& a, const Vec<V>& b) {
#pragma unroll
  for (int e = 0; e < V; e++) acc.v[e] = fmaf(a.v[e], b.v[e], acc.v[e]);
}

// What the rows of a block of the prompt kernels are: index inside the sequence's rows of this step, slot, whether the
// sequence has a stored window, whether the row is the sequence's last one.
struct ConvRows { int i[CONV_R], slot[CONV_R], has[CONV_R], last[CONV_R]; };
__device__ __forceinline__ void conv_rows_describe(ConvRows& s, int t0, int n_rows, const int* row_seq, const int* cu_seqlens,
                                                   const int* slots, const int* start_pos) {
  if (threadIdx.x < CONV_R) {
    const int t = t0 + threadIdx.x;
    int i = 0, slot = 0, has = 0, last = 0;
    if (t < n_rows) {
      const int b = row_seq[t];
      i = t - cu_seqlens[b];
      slot = slots[b];
      has = start_pos[b] > 0;
      last = t == cu_seqlens[b + 1] - 1;
    }
    s.i[threadIdx.x] = i;
    s.slot[threadIdx.x] = slot;
    s.has[threadIdx.x] = has;
    s.last[threadIdx.x] = last;
  }
}

// The rolling window of one column group: win[j] is the row j - (K - 1) steps back (win[K - 2] the previous row).  KT > 0:
// the number of taps, else K is read at run time and the window takes the limit's registers.
template <int KT, int V> struct Window {
  static constexpr int N = KT > 0 ? (KT > 1 ? KT - 1 : 1) : CONV_MAX_K - 1;
  Vec<V> win[N];
  __device__ __forceinline__ void clear() {
#pragma unroll
    for (int j = 0; j < N; j++) win[j] = vzero<V>();
  }
  // sum over the taps with `cur` under the last one; then the window moves on by `cur`
  __device__ __forceinline__ Vec<V> step(const Vec<V>& cur, const float* w, size_t C, int K, Vec<V> acc) {
#pragma unroll
    for (int j = 0; j < N; j++)
      if (j < K - 1) vfma<V>(acc, win[j], Vec<V>::ld(w + (size_t)j * C));
    vfma<V>(acc, cur, Vec<V>::ld(w + (size_t)(K - 1) * C));
    push(cur, K);
    return acc;
  }
  __device__ __forceinline__ void push(const Vec<V>& cur, int K) {
#pragma unroll
    for (int j = 0; j < N; j++) {
      if (j < K - 2) win[j] = win[j + 1 < N ? j + 1 : j];
      else if (j == K - 2) win[j] = cur;
    }
  }
  __device__ __forceinline__ void load(const float* st, size_t C, int K) {
#pragma unroll
    for (int j = 0; j < N; j++) win[j] = j < K - 1 ? Vec<V>::ld(st + (size_t)j * C) : vzero<V>();
  }
  __device__ __forceinline__ void store(float* st, size_t C, int K) const {
#pragma unroll
    for (int j = 0; j < N; j++)
      if (j < K - 1) win[j].st(st + (size_t)j * C);
  }
};

// Weights of a column group in registers where the number of taps is known at compile time.
template <int KT, int V> struct Taps {
  Vec<V> w[KT > 0 ? KT : 1];
  __device__ __forceinline__ void load(const float* p, size_t C) {
    if constexpr (KT > 0) {
#pragma unroll
      for (int j = 0; j < KT; j++) w[j] = Vec<V>::ld(p + (size_t)j * C);
    }
  }
};
template <int KT, int V>
__device__ __forceinline__ Vec<V> conv_step(Window<KT, V>& win, const Taps<KT, V>& taps, const Vec<V>& cur, const float* w, size_t C,
                                            int K, Vec<V> acc) {
  if constexpr (KT == 0) {
    return win.step(cur, w, C, K, acc);
  } else {
#pragma unroll
    for (int j = 0; j < KT - 1; j++) vfma<V>(acc, win.win[j], taps.w[j]);
    vfma<V>(acc, cur, taps.w[KT - 1]);
    win.push(cur, K);
    return acc;
  }
}

// ---- norm, then the row plus its convolution ------------------------------------------------------------------------------
template <typename TO, int KT, int V>
__global__ void __launch_bounds__(256)
rmsnorm_conv_rows_kernel(const float* __restrict__ x, const float* __restrict__ g, float eps, const float* __restrict__ w,
                         const int* __restrict__ row_seq, const int* __restrict__ cu_seqlens, const int* __restrict__ slots,
                         const int* __restrict__ start_pos, float* state, TO* __restrict__ out, int n_rows, int D, int K,
                         int write_state) {
  tlc_pdl(x, state, out);
  if (KT > 0) K = KT;
  __shared__ ConvRows s;
  __shared__ float s_inv[CONV_R + CONV_MAX_K - 1];       // of packed row t0 - (K - 1) + q
  const int t0 = blockIdx.x * CONV_R, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  conv_rows_describe(s, t0, n_rows, row_seq, cu_seqlens, slots, start_pos);
  for (int q = warp; q < CONV_R + K - 1; q += 8) {
    const int t = t0 - (K - 1) + q;
    float ss = 0.f;
    if (t >= 0 && t < n_rows) {
      const float* xr = x + (size_t)t * D;
      constexpr int U = 8;                              // (loads issued together)
      int d = lane * V;
      for (; d + (U - 1) * 32 * V < D; d += U * 32 * V) {
        Vec<V> v[U];
#pragma unroll
        for (int u = 0; u < U; u++) v[u] = Vec<V>::ld(xr + d + u * 32 * V);
#pragma unroll
        for (int u = 0; u < U; u++)
#pragma unroll
          for (int e = 0; e < V; e++) ss = fmaf(v[u].v[e], v[u].v[e], ss);
      }
      for (; d < D; d += 32 * V) {
        const Vec<V> v = Vec<V>::ld(xr + d);
#pragma unroll
        for (int e = 0; e < V; e++) ss = fmaf(v.v[e], v.v[e], ss);
      }
    }
    ss = warp_sum(ss);
    if (lane == 0) s_inv[q] = 1.0f / sqrtf(ss / (float)D + eps);
  }
  __syncthreads();
  for (int d = threadIdx.x * V; d < D; d += 256 * V) {
    const Vec<V> gv = Vec<V>::ld(g + d);
    Vec<V> rows[CONV_R];                                // (loads issued together)
#pragma unroll
    for (int r = 0; r < CONV_R; r++) rows[r] = t0 + r < n_rows ? Vec<V>::ld(x + (size_t)(t0 + r) * D + d) : vzero<V>();
    auto scaled = [&](Vec<V> v, float inv) {
#pragma unroll
      for (int e = 0; e < V; e++) v.v[e] = v.v[e] * inv * gv.v[e];
      return v;
    };
    Taps<KT, V> taps;
    taps.load(w + d, D);
    Window<KT, V> win;
    win.clear();
    // rows in front of the block's first: of this step, else of the stored window, else zeros
#pragma unroll
    for (int j = 0; j < Window<KT, V>::N; j++) {
      if (j < K - 1) {
        const int back = K - 1 - j, i = s.i[0] - back;
        if (i >= 0) win.win[j] = scaled(Vec<V>::ld(x + (size_t)(t0 - back) * D + d), s_inv[j]);
        else if (s.has[0]) win.win[j] = Vec<V>::ld(state + ((size_t)s.slot[0] * (K - 1) + (K - 1 + i)) * D + d);
      }
    }
#pragma unroll
    for (int r = 0; r < CONV_R; r++) {
      const int t = t0 + r;
      if (t >= n_rows) break;
      if (r > 0 && s.i[r] == 0) {
        if (s.has[r]) win.load(state + (size_t)s.slot[r] * (K - 1) * D + d, D, K);
        else win.clear();
      }
      const Vec<V> cur = scaled(rows[r], s_inv[K - 1 + r]);
      conv_step<KT, V>(win, taps, cur, w + d, D, K, cur).st(out + (size_t)t * D + d);
      if (write_state && s.last[r]) win.store(state + (size_t)s.slot[r] * (K - 1) * D + d, D, K);
    }
  }
}

// The new windows of sequences that brought several rows (some of which went on from an earlier step): grid (B), a block
// norms the sequence's last K - 1 rows; a thread reads what it needs of the old window before it writes.
template <int V>
__global__ void __launch_bounds__(256)
rmsnorm_conv_state_kernel(const float* __restrict__ x, const float* __restrict__ g, float eps, const int* __restrict__ cu_seqlens,
                          const int* __restrict__ slots, const int* __restrict__ start_pos, float* state, int D, int K) {
  tlc_pdl(x, state);
  __shared__ float s_inv[CONV_MAX_K - 1];
  const int b = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t0 = cu_seqlens[b], n = cu_seqlens[b + 1] - t0;
  if (n == 0) return;
  for (int j = warp; j < K - 1; j += 8) {
    const int i = n - (K - 1) + j;
    float ss = 0.f;
    if (i >= 0)
      for (int d = lane * V; d < D; d += 32 * V) {
        const Vec<V> v = Vec<V>::ld(x + (size_t)(t0 + i) * D + d);
#pragma unroll
        for (int e = 0; e < V; e++) ss = fmaf(v.v[e], v.v[e], ss);
      }
    ss = warp_sum(ss);
    if (lane == 0) s_inv[j] = 1.0f / sqrtf(ss / (float)D + eps);
  }
  __syncthreads();
  const bool has = start_pos[b] > 0;
  float* st = state + (size_t)slots[b] * (K - 1) * D;
  for (int d = threadIdx.x * V; d < D; d += 256 * V) {
    const Vec<V> gv = Vec<V>::ld(g + d);
    for (int j = 0; j < K - 1; j++) {               // (window row j comes from row j + n of the old one or from a new row: upwards)
      const int i = n - (K - 1) + j;
      Vec<V> v = vzero<V>();
      if (i >= 0) {
        v = Vec<V>::ld(x + (size_t)(t0 + i) * D + d);
#pragma unroll
        for (int e = 0; e < V; e++) v.v[e] = v.v[e] * s_inv[j] * gv.v[e];
      } else if (has) {
        v = Vec<V>::ld(st + (size_t)(K - 1 + i) * D + d);
      }
      v.st(st + (size_t)j * D + d);
    }
  }
}

// One-token steps: a block per sequence.  ONE: every thread has at most one column group, and what does not depend on the
// previous kernel (window, weights) is fetched before the wait on it.
template <typename TO, int KT, int V, bool ONE>
__global__ void __launch_bounds__(1024)
rmsnorm_conv_decode_kernel(const float* __restrict__ x, const float* __restrict__ g, float eps, const float* __restrict__ w,
                           const int* __restrict__ slots, const int* __restrict__ start_pos, float* state, TO* __restrict__ out,
                           int D, int K) {
  asm volatile("griddepcontrol.launch_dependents;");
  if (KT > 0) K = KT;
  __shared__ float red[33];
  const int b = blockIdx.x, step = blockDim.x * V;
  const bool has = start_pos[b] > 0;
  float* st = state + (size_t)slots[b] * (K - 1) * D;
  const int d0 = threadIdx.x * V;
  Window<KT, V> win;
  Taps<KT, V> taps;
  Vec<V> gv = vzero<V>();
  if (ONE && d0 < D) {
    if (has) win.load(st + d0, D, K); else win.clear();
    taps.load(w + d0, D);
    gv = Vec<V>::ld(g + d0);
  }
  tlc_wait(x, out);
  const float* xr = x + (size_t)b * D;
  float ss = 0.f;
  Vec<V> cur = vzero<V>();
  for (int d = d0; d < D; d += step) {
    const Vec<V> v = Vec<V>::ld(xr + d);
#pragma unroll
    for (int e = 0; e < V; e++) ss = fmaf(v.v[e], v.v[e], ss);
    if (ONE) cur = v;
  }
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)D + eps);
  for (int d = d0; d < D; d += step) {
    if (!ONE) {
      if (has) win.load(st + d, D, K); else win.clear();
      taps.load(w + d, D);
      gv = Vec<V>::ld(g + d);
      cur = Vec<V>::ld(xr + d);
    }
#pragma unroll
    for (int e = 0; e < V; e++) cur.v[e] = cur.v[e] * inv * gv.v[e];
    conv_step<KT, V>(win, taps, cur, w + d, D, K, cur).st(out + (size_t)b * D + d);
    win.store(st + d, D, K);
  }
}

template <typename TO, int KT, int V>
static void rmsnorm_conv_launch(const float* x, const float* g, float eps, const float* w, float* state, const int* cu_seqlens,
                                const int* row_seq, const int* slots, const int* start_pos, void* out, int T, int B, int D, int K,
                                int single_rows, int all_fresh, cudaStream_t stream) {
  if (single_rows && T == B) {
    const int groups = (D + V - 1) / V;
    const int nt = groups >= 1024 ? 1024 : (groups + 31) / 32 * 32;
    if (groups <= 1024)
      tlc_launch(rmsnorm_conv_decode_kernel<TO, KT, V, true>, dim3(B), dim3(nt), 0, stream, x, g, eps, w, slots, start_pos, state,
                 (TO*)out, D, K);
    else
      tlc_launch(rmsnorm_conv_decode_kernel<TO, KT, V, false>, dim3(B), dim3(nt), 0, stream, x, g, eps, w, slots, start_pos, state,
                 (TO*)out, D, K);
    return;
  }
  tlc_launch(rmsnorm_conv_rows_kernel<TO, KT, V>, dim3((T + CONV_R - 1) / CONV_R), dim3(256), 0, stream, x, g, eps, w, row_seq,
             cu_seqlens, slots, start_pos, state, (TO*)out, T, D, K, all_fresh);
  if (!all_fresh && K > 1)
    tlc_launch(rmsnorm_conv_state_kernel<V>, dim3(B), dim3(256), 0, stream, x, g, eps, cu_seqlens, slots, start_pos, state, D, K);
}

#define CONV_DISPATCH_K(K, KT, ...)                              \
  switch (K) {                                                   \
    case 2: { constexpr int KT = 2; __VA_ARGS__; } break;        \
    case 3: { constexpr int KT = 3; __VA_ARGS__; } break;        \
    case 4: { constexpr int KT = 4; __VA_ARGS__; } break;        \
    default: { constexpr int KT = 0; __VA_ARGS__; } break;       \
  }

// x float [T, D]; g [D]; w [K, D]; state [n_slots, K - 1, D]; out [T, D] of out_dtype.  single_rows: every sequence brings
// exactly one row (row b belongs to sequence b); all_fresh: every sequence starts at position 0.
extern "C" int tlc_rmsnorm_conv(const float* x, const float* g, float eps, const float* w, float* state, const int* cu_seqlens,
                                const int* row_seq, const int* slots, const int* start_pos, void* out, int out_dtype, int T, int B,
                                int D, int K, int single_rows, int all_fresh, cudaStream_t stream) {
  if (T == 0) return 0;
  TLC_REQUIRE(K >= 1 && K <= CONV_MAX_K, "rmsnorm_conv: %d taps are outside the kernel's range 1..%d", K, CONV_MAX_K);
  const bool vec = D % 4 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)g % 16 == 0 && (uintptr_t)w % 16 == 0 &&
                   (uintptr_t)state % 16 == 0 && (uintptr_t)out % 16 == 0;
  TLC_DISPATCH_DTYPE(out_dtype, TO, CONV_DISPATCH_K(K, KT, {
    if (vec)
      rmsnorm_conv_launch<TO, KT, 4>(x, g, eps, w, state, cu_seqlens, row_seq, slots, start_pos, out, T, B, D, K, single_rows, all_fresh, stream);
    else
      rmsnorm_conv_launch<TO, KT, 1>(x, g, eps, w, state, cu_seqlens, row_seq, slots, start_pos, out, T, B, D, K, single_rows, all_fresh, stream);
  }));
  TLC_CHECK_LAUNCH("rmsnorm_conv");
  return 0;
}

// ---- columns of a projection --------------------------------------------------------------------------------------------------
// What the columns from `from` on are blended with: rows of `first`, whose heads hold vd_f values in hd_f columns each where
// this matrix's hold vd in hd (the columns past a head's values are padding and stay as they are).
struct Blend {
  const float* first;
  int ld, from, hd, vd, hd_f, vd_f;
  float lam;
};
template <int V>
__device__ __forceinline__ Vec<V> blend(Vec<V> y, const Blend& bl, const float* first, int t, int d) {
  const int c = d - bl.from;
  if (first == nullptr || c < 0) return y;
  const float* row = first + (size_t)t * bl.ld;
  if (V == 1) {
    const int h = c / bl.hd, e = c - h * bl.hd;
    if (e >= bl.vd) return y;
    const int flat = h * bl.vd + e, hf = flat / bl.vd_f;
    y.v[0] = fmaf(bl.lam, row[(size_t)hf * bl.hd_f + flat - hf * bl.vd_f], (1.0f - bl.lam) * y.v[0]);
    return y;
  }
  const Vec<V> f = Vec<V>::ld(row + c);              // (one layout: padding is zero in both)
#pragma unroll
  for (int e = 0; e < V; e++) y.v[e] = fmaf(bl.lam, f.v[e], (1.0f - bl.lam) * y.v[e]);
  return y;
}

template <int KT, int V>
__global__ void __launch_bounds__(256)
channel_conv_rows_kernel(const float* __restrict__ proj, int ld, int off, const float* __restrict__ w, const int* __restrict__ row_seq,
                         const int* __restrict__ cu_seqlens, const int* __restrict__ slots, const int* __restrict__ start_pos,
                         float* state, float* __restrict__ out, Blend bl, int n_rows, int C, int K, int write_state) {
  const float* first = bl.first;
  tlc_pdl(proj, state, out, first);
  if (KT > 0) K = KT;
  __shared__ ConvRows s;
  const int t0 = blockIdx.x * CONV_R;
  conv_rows_describe(s, t0, n_rows, row_seq, cu_seqlens, slots, start_pos);
  __syncthreads();
  const int d = (blockIdx.y * 256 + threadIdx.x) * V;
  if (d >= C) return;
  const float* src = proj + off + d;
  Taps<KT, V> taps;
  taps.load(w + d, C);
  Window<KT, V> win;
  win.clear();
#pragma unroll
  for (int j = 0; j < Window<KT, V>::N; j++) {
    if (j < K - 1) {
      const int back = K - 1 - j, i = s.i[0] - back;
      if (i >= 0) win.win[j] = Vec<V>::ld(src + (size_t)(t0 - back) * ld);
      else if (s.has[0]) win.win[j] = Vec<V>::ld(state + ((size_t)s.slot[0] * (K - 1) + (K - 1 + i)) * C + d);
    }
  }
  Vec<V> rows[CONV_R];                                  // (all loads issued together)
#pragma unroll
  for (int r = 0; r < CONV_R; r++) rows[r] = t0 + r < n_rows ? Vec<V>::ld(src + (size_t)(t0 + r) * ld) : vzero<V>();
#pragma unroll
  for (int r = 0; r < CONV_R; r++) {
    const int t = t0 + r;
    if (t >= n_rows) break;
    if (r > 0 && s.i[r] == 0) {
      if (s.has[r]) win.load(state + (size_t)s.slot[r] * (K - 1) * C + d, C, K);
      else win.clear();
    }
    Vec<V> y = conv_step<KT, V>(win, taps, rows[r], w + d, C, K, vzero<V>());
    blend<V>(y, bl, first, t, d).st(out + (size_t)t * C + d);
    if (write_state && s.last[r]) win.store(state + (size_t)s.slot[r] * (K - 1) * C + d, C, K);
  }
}

template <int V>
__global__ void __launch_bounds__(256)
channel_conv_state_kernel(const float* __restrict__ proj, int ld, int off, const int* __restrict__ cu_seqlens, const int* __restrict__ slots,
                          const int* __restrict__ start_pos, float* state, int C, int K) {
  tlc_pdl(proj, state);
  const int b = blockIdx.x, d = (blockIdx.y * 256 + threadIdx.x) * V;
  if (d >= C) return;
  const int t0 = cu_seqlens[b], n = cu_seqlens[b + 1] - t0;
  if (n == 0) return;
  const bool has = start_pos[b] > 0;
  float* st = state + (size_t)slots[b] * (K - 1) * C + d;
  for (int j = 0; j < K - 1; j++) {
    const int i = n - (K - 1) + j;
    Vec<V> v = vzero<V>();
    if (i >= 0) v = Vec<V>::ld(proj + (size_t)(t0 + i) * ld + off + d);
    else if (has) v = Vec<V>::ld(st + (size_t)(K - 1 + i) * C);
    v.st(st + (size_t)j * C);
  }
}

template <int KT, int V>
__global__ void __launch_bounds__(128)
channel_conv_decode_kernel(const float* __restrict__ proj, int ld, int off, const float* __restrict__ w, const int* __restrict__ slots,
                           const int* __restrict__ start_pos, float* state, float* __restrict__ out, Blend bl, int C, int K) {
  asm volatile("griddepcontrol.launch_dependents;");
  const float* first = bl.first;
  if (KT > 0) K = KT;
  const int b = blockIdx.x, d = (blockIdx.y * 128 + threadIdx.x) * V;
  if (d >= C) return;
  float* st = state + (size_t)slots[b] * (K - 1) * C + d;
  Window<KT, V> win;
  if (start_pos[b] > 0) win.load(st, C, K); else win.clear();
  Taps<KT, V> taps;
  taps.load(w + d, C);
  tlc_wait(proj, out, first);
  const Vec<V> cur = Vec<V>::ld(proj + (size_t)b * ld + off + d);
  Vec<V> y = conv_step<KT, V>(win, taps, cur, w + d, C, K, vzero<V>());
  blend<V>(y, bl, first, b, d).st(out + (size_t)b * C + d);
  win.store(st, C, K);
}

template <int KT, int V>
static void channel_conv_launch(const float* proj, int ld, int off, const float* w, float* state, const int* cu_seqlens,
                                const int* row_seq, const int* slots, const int* start_pos, float* out, const Blend& bl, int T, int B, int C,
                                int K, int single_rows, int all_fresh, cudaStream_t stream) {
  const int groups = (C + V - 1) / V;
  if (single_rows && T == B) {
    tlc_launch(channel_conv_decode_kernel<KT, V>, dim3(B, (groups + 127) / 128), dim3(128), 0, stream, proj, ld, off, w, slots, start_pos,
               state, out, bl, C, K);
    return;
  }
  const unsigned gy = (unsigned)((groups + 255) / 256);
  tlc_launch(channel_conv_rows_kernel<KT, V>, dim3((T + CONV_R - 1) / CONV_R, gy), dim3(256), 0, stream, proj, ld, off, w, row_seq,
             cu_seqlens, slots, start_pos, state, out, bl, T, C, K, all_fresh);
  if (!all_fresh && K > 1)
    tlc_launch(channel_conv_state_kernel<V>, dim3(B, gy), dim3(256), 0, stream, proj, ld, off, cu_seqlens, slots, start_pos, state, C, K);
}

// proj float [T, ld], the C columns from `off`; w [K, C]; state [n_slots, K - 1, C]; out float [T, C].  first (or NULL) float
// [T, ld_first]: the columns from mix_from on, heads of hd columns that hold vd values, become (1 - lam) y + lam * first[t, .],
// value by value; the rows of `first` hold the same number of values in heads of vd_first in hd_first columns.
extern "C" int tlc_channel_conv(const float* proj, int ld, int off, const float* w, float* state, const int* cu_seqlens,
                                const int* row_seq, const int* slots, const int* start_pos, float* out, const float* first,
                                int ld_first, int mix_from, int hd, int vd, int hd_first, int vd_first, float lam, int T, int B, int C,
                                int K, int single_rows, int all_fresh, cudaStream_t stream) {
  if (T == 0 || C == 0) return 0;
  TLC_REQUIRE(K >= 1 && K <= CONV_MAX_K, "channel_conv: %d taps are outside the kernel's range 1..%d", K, CONV_MAX_K);
  if (first != nullptr) {
    TLC_REQUIRE(mix_from >= 0 && mix_from <= C && vd >= 1 && hd >= vd && vd_first >= 1 && hd_first >= vd_first && (C - mix_from) % hd == 0,
                "channel_conv: %d mixed columns in heads of %d of %d", C - mix_from, vd, hd);
    const int values = (C - mix_from) / hd * vd;
    TLC_REQUIRE(values % vd_first == 0 && ld_first >= values / vd_first * hd_first, "channel_conv: %d mixed values in rows of %d, heads of %d of %d",
                values, ld_first, vd_first, hd_first);
  }
  const Blend bl = {first, ld_first, mix_from, hd, vd, hd_first, vd_first, lam};
  const bool vec = C % 4 == 0 && ld % 4 == 0 && off % 4 == 0 && (uintptr_t)proj % 16 == 0 && (uintptr_t)w % 16 == 0 &&
                   (uintptr_t)state % 16 == 0 && (uintptr_t)out % 16 == 0 &&
                   (first == nullptr || ((uintptr_t)first % 16 == 0 && ld_first % 4 == 0 && mix_from % 4 == 0 && hd == hd_first && vd == vd_first));
  CONV_DISPATCH_K(K, KT, {
    if (vec)
      channel_conv_launch<KT, 4>(proj, ld, off, w, state, cu_seqlens, row_seq, slots, start_pos, out, bl, T, B, C, K,
                                 single_rows, all_fresh, stream);
    else
      channel_conv_launch<KT, 1>(proj, ld, off, w, state, cu_seqlens, row_seq, slots, start_pos, out, bl, T, B, C, K,
                                 single_rows, all_fresh, stream);
  });
  TLC_CHECK_LAUNCH("channel_conv");
  return 0;
}
