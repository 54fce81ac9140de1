// What lies between the projection of queries, keys and values and attention, in one kernel on 32-bit rows:
//
//   a short causal convolution over time on every column,  y_t = sum_j w[:, j] u_(t - K + 1 + j)     (K taps; K = 1 with no weights: none)
//   an RMS norm over ALL query columns and one over all key columns, each with a weight                (optional)
//   a rotation of neighbouring pairs (2i, 2i+1) of the first `rot` dimensions of every query and key head by
//     position * inv_freq[i], cosines and sines times `amplitude`                                      (rot 0: none)
//   the stores: queries to q_out, keys and values into the pages of their sequences; or, for a kernel that stores by
//     itself, the whole row to out (32-bit).
//
// Single-token steps: one kernel, a block per row; a thread owns groups of four neighbouring columns (a pair never crosses a
// group), so the convolved values stay in registers while the block adds up their squares.  Kept rows and weights are fetched
// before the wait on the projection (an earlier step wrote them), and the thread that read a kept row writes its successor.
// Prompts: a block takes QP_R packed rows of 1,024 columns.  Where the projections are normed, a first kernel convolves and
// leaves the rows' sums of squares, block by block of columns (added up in one order, whatever else is in the batch); the
// second convolves again, with its inputs in the L2 by then, and finishes.  (One kernel whose blocks hold whole rows takes
// twice as long: few blocks fit an SM, and each is a chain of loads, a block's sum and stores.)
// kept rows: state [n_slots, K - 1, C], oldest first; a sequence at position 0 has zeros.
#include "common.cuh"

namespace {

constexpr int QP_R = 8;              // packed rows of a block of a prompt's kernels
constexpr int QP_NT = 256;           // and its threads, a group of four columns each

struct QpArgs {
  const float* proj;                 // [T, ld], the C columns from `off`: queries | keys | values
  int ld, off, C, K;
  const float* w;                    // taps [K, C] (NULL: no convolution)
  float* state;                      // kept rows
  int H, KV, hd;
  const float* q_w;                  // norm weights, [H * hd] and [KV * hd] (NULL: no norm)
  const float* k_w;
  float q_inv_n, k_inv_n, eps;       // one over how many columns each mean is over
  const float* inv_freq;
  int rot;
  float amplitude;
  const int* positions;
  const int* row_seq;
  const int* cu_seqlens;
  const int* slots;
  const int* start_pos;
  const int* block_table;
  int max_pages, n_rows;
  int write_state;                   // the block that holds a sequence's last row writes its kept rows
  float* sums;                       // [T, n_sums, 2]: the squares' sums of a row's query and key columns, a block of columns each
  int n_sums;
  float* out;                        // [T, C], or NULL: the three below
  void* q_out;
  void* k_pages;
  void* v_pages;
};

__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put4(float* p, float4 v) { st4(p, v); }
__device__ __forceinline__ void put4(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<const unsigned*>(&lo);
  u.y = *reinterpret_cast<const unsigned*>(&hi);
  *reinterpret_cast<uint2*>(p) = u;
}
__device__ __forceinline__ void fma4(float4& a, float4 x, float4 y) {
  a.x = fmaf(x.x, y.x, a.x); a.y = fmaf(x.y, y.y, a.y); a.z = fmaf(x.z, y.z, a.z); a.w = fmaf(x.w, y.w, a.w);
}
__device__ __forceinline__ float dot4(float4 a) { return a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w; }

// A block's sums of the queries' and the keys' squares of its row: tot[0], tot[1], one over the root mean squares.
__device__ __forceinline__ void norm_scales(const QpArgs& a, float sq, float sk, float* red, float* tot) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if (lane == 0) { red[2 * warp] = sq; red[2 * warp + 1] = sk; }
  __syncthreads();
  for (int k = warp; k < 2; k += nw) {                  // (a block may be a single warp)
    const float v = warp_sum(lane < nw ? red[2 * lane + k] : 0.f);
    if (lane == 0) tot[k] = 1.0f / sqrtf(v * (k ? a.k_inv_n : a.q_inv_n) + a.eps);
  }
  __syncthreads();
}

// Rotates the two pairs of a group that starts at dimension d of its head; cs: the row's [rot/2] cosines, then sines.
__device__ __forceinline__ float4 turn4(float4 y, int d, int rot, const float* cs) {
  const int half = rot >> 1, p = d >> 1;
  if (d < rot) {
    const float c = cs[p], s = cs[half + p], u = y.x, v = y.y;
    y.x = u * c - v * s;
    y.y = v * c + u * s;
  }
  if (d + 2 < rot) {
    const float c = cs[p + 1], s = cs[half + p + 1], u = y.z, v = y.w;
    y.z = u * c - v * s;
    y.w = v * c + u * s;
  }
  return y;
}

// Where one group of columns goes: 0 a query, 1 a key, 2 a value; its head, and its first dimension there.
struct Group {
  int c, kind, at, h, d;
  __device__ __forceinline__ Group(const QpArgs& a, int col) : c(col) {
    const int nq = a.H * a.hd, nk = a.KV * a.hd;
    kind = c < nq ? 0 : (c < nq + nk ? 1 : 2);
    at = kind == 0 ? c : (kind == 1 ? c - nq : c - nq - nk);
    h = at / a.hd;
    d = at - h * a.hd;
  }
};

// Norm (scale: the row's, for this kind of columns; nw: the weight), rotation and store of one group of a row.
template <typename T>
__device__ __forceinline__ void finish(const QpArgs& a, const Group& g, float4 y, float4 nw, float scale, const float* cs, int t, int page,
                                       int prow) {
  if (g.kind < 2) {
    if (a.q_w) { y.x *= scale * nw.x; y.y *= scale * nw.y; y.z *= scale * nw.z; y.w *= scale * nw.w; }
    if (a.rot) y = turn4(y, g.d, a.rot, cs);
  }
  if (a.out) {
    st4(a.out + (size_t)t * a.C + g.c, y);
  } else if (g.kind == 0) {
    put4((T*)a.q_out + (size_t)t * a.H * a.hd + g.at, y);
  } else if (page >= 0) {
    put4((T*)(g.kind == 1 ? a.k_pages : a.v_pages) + (((size_t)page * a.KV + g.h) * TLC_PAGE + prow) * a.hd + g.d, y);
  }
}

// What a block of a prompt's kernels knows about its rows.
struct QpRows {
  int i[QP_R], has[QP_R], slot[QP_R], last[QP_R];       // row of its sequence's rows in this step; kept rows exist; slot; last row
};
__device__ __forceinline__ void describe(const QpArgs& a, QpRows& s, int t0, int rows) {
  if (threadIdx.x < QP_R) {
    const int r = threadIdx.x, t = t0 + r;
    if (r < rows) {
      const int b = a.row_seq[t];
      s.i[r] = t - a.cu_seqlens[b];
      s.last[r] = t + 1 == a.cu_seqlens[b + 1];
      s.has[r] = a.start_pos[b] > 0;
      s.slot[r] = a.slots[b];
    } else {
      s.i[r] = 1 << 20;
      s.has[r] = s.slot[r] = s.last[r] = 0;
    }
  }
}
// The rows t0 - (KT - 1) .. t0 + QP_R - 1 of a group of columns; all loads are issued together.
template <int KT>
__device__ __forceinline__ void load_rows(const QpArgs& a, float4 (&x)[KT - 1 + QP_R], int t0, int c) {
  const float* src = a.proj + a.off + c;
#pragma unroll
  for (int i = 0; i < KT - 1 + QP_R; i++) {
    const int t = t0 - (KT - 1) + i;
    x[i] = (t >= 0 && t < a.n_rows) ? ld4(src + (size_t)t * a.ld) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
}
// The convolved group of row r.
template <int KT>
__device__ __forceinline__ float4 convolve(const QpArgs& a, const QpRows& s, const float4 (&x)[KT - 1 + QP_R], const float4 (&w)[KT], int r,
                                           int c) {
  float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
  if (s.i[r] >= KT - 1) {
#pragma unroll
    for (int j = 0; j < KT; j++) fma4(y, w[j], x[r + j]);
    return y;
  }
#pragma unroll
  for (int j = 0; j < KT; j++) {
    float4 u = x[r + j];
    if (KT - 1 - j > s.i[r])                            // in front of the sequence's rows of this step
      u = s.has[r] ? ld4(a.state + ((size_t)s.slot[r] * (KT - 1) + s.i[r] + j) * a.C + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    fma4(y, w[j], u);
  }
  return y;
}
template <int KT>
__device__ __forceinline__ void load_taps(const QpArgs& a, float4 (&w)[KT], int c) {
#pragma unroll
  for (int j = 0; j < KT; j++) w[j] = a.w ? __ldg(reinterpret_cast<const float4*>(a.w + (size_t)j * a.C + c)) : make_float4(1.f, 1.f, 1.f, 1.f);
}

// grid (row blocks, blocks of query and key columns)
template <int KT>
__global__ void __launch_bounds__(QP_NT)
qkv_sums_kernel(const __grid_constant__ QpArgs args) {
  asm volatile("griddepcontrol.launch_dependents;");
  QpArgs a = args;
  __shared__ QpRows s;
  __shared__ float red[QP_NT / 32][2 * QP_R];
  const int t0 = blockIdx.x * QP_R, rows = min(QP_R, a.n_rows - t0), lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int c = 4 * (blockIdx.y * QP_NT + threadIdx.x), nq = a.H * a.hd, n = nq + a.KV * a.hd;
  describe(a, s, t0, rows);
  float4 w[KT];
  if (c < n) load_taps<KT>(a, w, c);
  tlc_wait(a.proj);
  float4 x[KT - 1 + QP_R];
  if (c < n) load_rows<KT>(a, x, t0, c);
  __syncthreads();
  float sum[QP_R];
#pragma unroll
  for (int r = 0; r < QP_R; r++) sum[r] = c < n ? dot4(convolve<KT>(a, s, x, w, r, c)) : 0.f;
  // (a group is all queries or all keys; a warp that holds both adds up both)
  const bool any_q = __any_sync(0xffffffffu, c < nq), any_k = __any_sync(0xffffffffu, c >= nq && c < n);
#pragma unroll
  for (int r = 0; r < QP_R; r++) {
    const float q = any_q ? warp_sum(c < nq ? sum[r] : 0.f) : 0.f, k = any_k ? warp_sum(c >= nq ? sum[r] : 0.f) : 0.f;
    if (lane == 0) { red[warp][2 * r] = q; red[warp][2 * r + 1] = k; }
  }
  __syncthreads();
  if (threadIdx.x < 2 * QP_R && (threadIdx.x >> 1) < rows) {
    float v = 0.f;
#pragma unroll
    for (int i = 0; i < QP_NT / 32; i++) v += red[i][threadIdx.x];
    a.sums[((size_t)(t0 + (threadIdx.x >> 1)) * a.n_sums + blockIdx.y) * 2 + (threadIdx.x & 1)] = v;
  }
}

// grid (row blocks, blocks of columns)
template <typename T, int KT>
__global__ void __launch_bounds__(QP_NT)
qkv_prepare_rows_kernel(const __grid_constant__ QpArgs args) {
  asm volatile("griddepcontrol.launch_dependents;");
  QpArgs a = args;
  __shared__ QpRows s;
  __shared__ int s_page[QP_R], s_prow[QP_R];
  __shared__ float scale[2 * QP_R];
  extern __shared__ float cs[];                         // [QP_R][rot]
  const int t0 = blockIdx.x * QP_R, rows = min(QP_R, a.n_rows - t0), half = a.rot >> 1;
  const int c = 4 * (blockIdx.y * QP_NT + threadIdx.x), nq = a.H * a.hd, nk = a.KV * a.hd;
  const bool mine = c < a.C;
  describe(a, s, t0, rows);
  if (threadIdx.x < rows) {
    const int t = t0 + threadIdx.x, pos = a.positions[t];
    s_page[threadIdx.x] = a.out ? -1 : a.block_table[(size_t)a.slots[a.row_seq[t]] * a.max_pages + pos / TLC_PAGE];
    s_prow[threadIdx.x] = pos % TLC_PAGE;
  }
  if (4 * (int)blockIdx.y * QP_NT < nq + nk) {          // (a block of values only turns nothing)
    for (int i = threadIdx.x; i < rows * half; i += QP_NT) {
      const int r = i / half, j = i - r * half;
      float sn, co;
      sincosf((float)a.positions[t0 + r] * a.inv_freq[j], &sn, &co);
      cs[r * a.rot + j] = co * a.amplitude;
      cs[r * a.rot + half + j] = sn * a.amplitude;
    }
  }
  const Group g(a, c);
  float4 w[KT], nw = make_float4(1.f, 1.f, 1.f, 1.f);
  if (mine) {
    load_taps<KT>(a, w, c);
    if (a.q_w && g.kind < 2) nw = __ldg(reinterpret_cast<const float4*>((g.kind == 0 ? a.q_w : a.k_w) + g.at));
  }
  tlc_wait(a.proj, a.sums);
  float4 x[KT - 1 + QP_R];
  if (mine) load_rows<KT>(a, x, t0, c);
  if (a.q_w && threadIdx.x < 2 * rows) {
    const int r = threadIdx.x >> 1, k = threadIdx.x & 1;
    float v = 0.f;
    for (int i = 0; i < a.n_sums; i++) v += a.sums[((size_t)(t0 + r) * a.n_sums + i) * 2 + k];
    scale[threadIdx.x] = 1.0f / sqrtf(v * (k ? a.k_inv_n : a.q_inv_n) + a.eps);
  }
  __syncthreads();
  if (!mine) return;
#pragma unroll
  for (int r = 0; r < QP_R; r++) {
    if (r >= rows) break;
    finish<T>(a, g, convolve<KT>(a, s, x, w, r, c), nw, a.q_w && g.kind < 2 ? scale[2 * r + g.kind] : 1.f, cs + r * a.rot, t0 + r, s_page[r],
              s_prow[r]);
    if (KT > 1 && a.write_state && s.last[r]) {         // (no sequence of the step reads kept rows: see the launcher)
#pragma unroll
      for (int j = 0; j < KT - 1; j++)
        st4(a.state + ((size_t)s.slot[r] * (KT - 1) + j) * a.C + c, KT - 2 - j <= s.i[r] ? x[r + j + 1] : make_float4(0.f, 0.f, 0.f, 0.f));
    }
  }
}

// After a step in which sequences went on from kept rows: the last K - 1 rows of every sequence.
__global__ void __launch_bounds__(256)
qkv_keep_rows_kernel(QpArgs a) {
  tlc_pdl(a.proj, a.state);
  const int b = blockIdx.x, c = 4 * (blockIdx.y * 256 + threadIdx.x), N = a.K - 1;
  if (c >= a.C) return;
  const int t0 = a.cu_seqlens[b], n = a.cu_seqlens[b + 1] - t0;
  if (n == 0) return;
  const bool has = a.start_pos[b] > 0;
  float* st = a.state + (size_t)a.slots[b] * N * a.C + c;
  for (int j = 0; j < N; j++) {
    const int i = n - N + j;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i >= 0) v = ld4(a.proj + (size_t)(t0 + i) * a.ld + a.off + c);
    else if (has) v = ld4(st + (size_t)(N + i) * a.C);             // (N + i > j: not overwritten yet)
    st4(st + (size_t)j * a.C, v);
  }
}

template <typename T, int KT, int NV>
__global__ void __launch_bounds__(1024)
qkv_prepare_decode_kernel(QpArgs a) {
  asm volatile("griddepcontrol.launch_dependents;");
  __shared__ float red[32 * 2], tot[2];
  extern __shared__ float cs[];                         // [rot]
  const int t = blockIdx.x, half = a.rot >> 1, pos = a.positions[t], slot = a.slots[t];
  const int n4 = a.C >> 2, nq = a.H * a.hd, nk = a.KV * a.hd;
  const bool has = a.start_pos[t] > 0;
  const int page = a.out ? -1 : a.block_table[(size_t)slot * a.max_pages + pos / TLC_PAGE];
  float4 s[NV], nw[NV], w_new[NV];
  float* st = a.state + (size_t)slot * (KT - 1) * a.C;
#pragma unroll
  for (int v = 0; v < NV; v++) {
    const int c = 4 * (threadIdx.x + v * blockDim.x);
    s[v] = make_float4(0.f, 0.f, 0.f, 0.f);
    nw[v] = w_new[v] = make_float4(1.f, 1.f, 1.f, 1.f);
    if (c >= 4 * n4) continue;
    if (KT > 1) {
      float4 kept[KT];
#pragma unroll
      for (int j = 0; j < KT - 1; j++) kept[j] = has ? ld4(st + (size_t)j * a.C + c) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int j = 0; j < KT - 1; j++) fma4(s[v], __ldg(reinterpret_cast<const float4*>(a.w + (size_t)j * a.C + c)), kept[j]);
#pragma unroll
      for (int j = 0; j + 1 < KT - 1; j++) st4(st + (size_t)j * a.C + c, kept[j + 1]);
    }
    if (a.w) w_new[v] = __ldg(reinterpret_cast<const float4*>(a.w + (size_t)(KT - 1) * a.C + c));
    if (a.q_w && c < nq + nk) nw[v] = __ldg(reinterpret_cast<const float4*>(c < nq ? a.q_w + c : a.k_w + (c - nq)));
  }
  for (int j = threadIdx.x; j < half; j += blockDim.x) {
    float sn, c;
    sincosf((float)pos * a.inv_freq[j], &sn, &c);
    cs[j] = c * a.amplitude;
    cs[half + j] = sn * a.amplitude;
  }
  tlc_wait(a.proj);
  float sq = 0.f, sk = 0.f;
#pragma unroll
  for (int v = 0; v < NV; v++) {
    const int c = 4 * (threadIdx.x + v * blockDim.x);
    if (c >= 4 * n4) continue;
    const float4 u = ld4(a.proj + (size_t)t * a.ld + a.off + c);
    fma4(s[v], w_new[v], u);
    if (KT > 1) st4(st + (size_t)(KT - 2) * a.C + c, u);
    if (c < nq) sq += dot4(s[v]);
    else if (c < nq + nk) sk += dot4(s[v]);
  }
  if (a.q_w) norm_scales(a, sq, sk, red, tot);
  else __syncthreads();                                 // (the cosines)
#pragma unroll
  for (int v = 0; v < NV; v++) {
    const int c = 4 * (threadIdx.x + v * blockDim.x);
    if (c >= 4 * n4) continue;
    const Group g(a, c);
    finish<T>(a, g, s[v], nw[v], a.q_w && g.kind < 2 ? tot[g.kind] : 1.f, cs, t, page, pos % TLC_PAGE);
  }
}

template <typename T, int KT>
void launch(const QpArgs& a, int B, int single, cudaStream_t stream) {
  const int n4 = a.C >> 2;
  if (single) {
    const int nv = (n4 + 1023) / 1024, need = (n4 + nv - 1) / nv, nt = (need + 31) / 32 * 32;      // groups a thread, threads
#define QP_SINGLE(NV) tlc_launch(qkv_prepare_decode_kernel<T, KT, NV>, dim3(B), dim3(nt), (size_t)a.rot * sizeof(float), stream, a)
    if (nv == 1) QP_SINGLE(1); else if (nv == 2) QP_SINGLE(2); else if (nv == 3) QP_SINGLE(3); else QP_SINGLE(4);
#undef QP_SINGLE
    return;
  }
  const unsigned gx = (a.n_rows + QP_R - 1) / QP_R;
  if (a.q_w) tlc_launch(qkv_sums_kernel<KT>, dim3(gx, a.n_sums), dim3(QP_NT), 0, stream, a);
  tlc_launch(qkv_prepare_rows_kernel<T, KT>, dim3(gx, (n4 + QP_NT - 1) / QP_NT), dim3(QP_NT), (size_t)QP_R * a.rot * sizeof(float), stream, a);
  if (KT > 1 && !a.write_state) tlc_launch(qkv_keep_rows_kernel, dim3(B, (n4 + 255) / 256), dim3(256), 0, stream, a);
}

}  // namespace

extern "C" int tlc_qkv_prepare_ok(int H, int KV, int hd, int K, int ld, int off) {
  const long long C = (long long)(H + 2 * KV) * hd;
  return H >= 1 && KV >= 1 && K >= 1 && K <= 4 && hd % 4 == 0 && ld % 4 == 0 && off % 4 == 0 && C <= 4 * 1024 * 4 && hd <= 1024;
}

// Blocks of query and key columns: a step of T rows takes scratch of T * 2 * that many floats (single-token steps take none).
extern "C" int tlc_qkv_prepare_sums(int H, int KV, int hd) { return ((H + KV) * hd + 4 * QP_NT - 1) / (4 * QP_NT); }

extern "C" int tlc_qkv_prepare(const float* proj, int ld, int off, const float* w, int K, float* state, const float* q_w, const float* k_w,
                               int q_count, int k_count, float eps, const float* inv_freq, int rot, float amplitude, const int* positions,
                               const int* row_seq, const int* cu_seqlens, const int* slots, const int* start_pos, const int* block_table,
                               int max_pages, float* out, void* q_out, void* k_pages, void* v_pages, int dtype, int T, int B, int H, int KV,
                               int hd, int single_rows, int all_fresh, float* sums, cudaStream_t stream) {
  if (T == 0) return 0;
  TLC_REQUIRE(tlc_qkv_prepare_ok(H, KV, hd, K, ld, off), "qkv_prepare: %d and %d heads of %d behind %d taps (row stride %d, offset %d) are not built",
              H, KV, hd, K, ld, off);
  TLC_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= hd, "qkv_prepare: %d rotated of %d dimensions", rot, hd);
  TLC_REQUIRE((q_w == nullptr) == (k_w == nullptr) && (K == 1 || (w != nullptr && state != nullptr)), "qkv_prepare: the norms' weights come together, taps with kept rows");
  TLC_REQUIRE(out != nullptr || (q_out != nullptr && k_pages != nullptr && v_pages != nullptr && block_table != nullptr), "qkv_prepare: nowhere to store");
  TLC_REQUIRE(((uintptr_t)proj | (uintptr_t)w | (uintptr_t)state | (uintptr_t)q_w | (uintptr_t)k_w | (uintptr_t)out | (uintptr_t)q_out |
               (uintptr_t)k_pages | (uintptr_t)v_pages) % 16 == 0, "qkv_prepare: buffers must start on 16-byte boundaries");
  TLC_REQUIRE(q_w == nullptr || (q_count >= 1 && k_count >= 1), "qkv_prepare: norms over %d and %d columns", q_count, k_count);
  const int single = single_rows && T == B;
  TLC_REQUIRE(single || q_w == nullptr || sums != nullptr, "qkv_prepare: the norms of a prompt's rows need scratch");
  const QpArgs a = {proj, ld, off, (H + 2 * KV) * hd, K, w, state, H, KV, hd, q_w, k_w, 1.0f / (float)(q_count > 0 ? q_count : 1),
                    1.0f / (float)(k_count > 0 ? k_count : 1), eps, inv_freq, rot, amplitude, positions, row_seq, cu_seqlens, slots, start_pos,
                    block_table, max_pages, T, all_fresh, sums, tlc_qkv_prepare_sums(H, KV, hd), out, q_out, k_pages, v_pages};
  TLC_DISPATCH_DTYPE(dtype, TT, {
    if (K == 1) launch<TT, 1>(a, B, single, stream);
    else if (K == 2) launch<TT, 2>(a, B, single, stream);
    else if (K == 3) launch<TT, 3>(a, B, single, stream);
    else launch<TT, 4>(a, B, single, stream);
  });
  TLC_CHECK_LAUNCH("qkv_prepare");
  return 0;
}
