// What lies between the projection of queries, keys and values and attention, in one kernel on 32-bit rows:
//
//   a short causal convolution over time on every column,  y_t = sum_j w[:, j] u_(t - K + 1 + j)     (K taps; K = 1 with no weights: none)
//   an RMS norm over ALL query columns and one over all key columns, each with a weight                (optional)
//   a rotation of neighbouring pairs (2i, 2i+1) of the first `rot` dimensions of every query and key head by
//     position * inv_freq[i], cosines and sines times `amplitude`                                      (rot 0: none)
//   the stores: queries to q_out, keys and values into the pages of their sequences; or, for a kernel that stores by
//     itself, the whole row to out (32-bit).
//
// A thread owns the same groups of four neighbouring columns in every row of its block (a pair never crosses a group), so
// the convolved values stay in registers while the block adds up the sums of squares.  Prompts: a block takes QP_R packed
// rows; the K - 1 rows in front of them are read again (they are in the L2), or come from the sequences' kept rows.
// Single-token steps: a block per row; kept rows and weights are fetched before the wait on the projection (an earlier step
// wrote them), and the thread that read a kept row writes its successor.
// kept rows: state [n_slots, K - 1, C], oldest first; a sequence at position 0 has zeros.
#include "common.cuh"

namespace {

constexpr int QP_R = 4;              // packed rows of a block of a prompt's kernel

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

// R sums of the queries' squares and R of the keys', over the block; every thread gets all of them in tot[2 * R].
template <int R>
__device__ __forceinline__ void sums_of_squares(const float (&sq)[R], const float (&sk)[R], float* red, float* tot) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
#pragma unroll
  for (int r = 0; r < R; r++) {
    const float a = warp_sum(sq[r]), b = warp_sum(sk[r]);
    if (lane == 0) { red[warp * 2 * R + 2 * r] = a; red[warp * 2 * R + 2 * r + 1] = b; }
  }
  __syncthreads();
  for (int v = warp; v < 2 * R; v += nw) {
    const float s = warp_sum(lane < nw ? red[lane * 2 * R + v] : 0.f);
    if (lane == 0) tot[v] = s;
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

// Norm, rotation and store of one group of a row.
template <typename T>
__device__ __forceinline__ void finish(const QpArgs& a, float4 y, int c, float4 nw, float rq, float rk, const float* cs, int t, int page,
                                       int prow) {
  const int nq = a.H * a.hd, nk = a.KV * a.hd;
  const int kind = c < nq ? 0 : (c < nq + nk ? 1 : 2), at = kind == 0 ? c : (kind == 1 ? c - nq : c - nq - nk);
  const int h = at / a.hd, d = at - h * a.hd;
  if (kind < 2) {
    if (a.q_w) {
      const float s = kind == 0 ? rq : rk;
      y.x *= s * nw.x; y.y *= s * nw.y; y.z *= s * nw.z; y.w *= s * nw.w;
    }
    if (a.rot) y = turn4(y, d, a.rot, cs);
  }
  if (a.out) {
    st4(a.out + (size_t)t * a.C + c, y);
  } else if (kind == 0) {
    put4((T*)a.q_out + (size_t)t * nq + at, y);
  } else if (page >= 0) {
    put4((T*)(kind == 1 ? a.k_pages : a.v_pages) + (((size_t)page * a.KV + h) * TLC_PAGE + prow) * a.hd + d, y);
  }
}

template <typename T, int KT, int NV>
__global__ void __launch_bounds__(512)
qkv_prepare_rows_kernel(QpArgs a) {
  tlc_pdl(a.proj, a.state, a.out, a.q_out, a.k_pages, a.v_pages);
  __shared__ float red[16 * 2 * QP_R], tot[2 * QP_R];
  __shared__ int s_i[QP_R], s_has[QP_R], s_slot[QP_R], s_last[QP_R], s_page[QP_R], s_prow[QP_R];
  extern __shared__ float cs[];                         // [QP_R][rot]
  const int t0 = blockIdx.x * QP_R, rows = min(QP_R, a.n_rows - t0), half = a.rot >> 1;
  if (threadIdx.x < rows) {
    const int r = threadIdx.x, t = t0 + r, b = a.row_seq[t], pos = a.positions[t];
    s_i[r] = t - a.cu_seqlens[b];
    s_last[r] = t + 1 == a.cu_seqlens[b + 1];
    s_has[r] = a.start_pos[b] > 0;
    s_slot[r] = a.slots[b];
    s_page[r] = a.out ? -1 : a.block_table[(size_t)a.slots[b] * a.max_pages + pos / TLC_PAGE];
    s_prow[r] = pos % TLC_PAGE;
  }
  for (int i = threadIdx.x; i < rows * half; i += blockDim.x) {
    const int r = i / half, j = i - r * half;
    float sn, c;
    sincosf((float)a.positions[t0 + r] * a.inv_freq[j], &sn, &c);
    cs[r * a.rot + j] = c * a.amplitude;
    cs[r * a.rot + half + j] = sn * a.amplitude;
  }
  __syncthreads();
  const int n4 = a.C >> 2, nq = a.H * a.hd, nk = a.KV * a.hd;
  float4 y[NV][QP_R];
  float sq[QP_R], sk[QP_R];
#pragma unroll
  for (int r = 0; r < QP_R; r++) { sq[r] = 0.f; sk[r] = 0.f; }
#pragma unroll
  for (int v = 0; v < NV; v++) {
    const int c = 4 * (threadIdx.x + v * blockDim.x);
    if (c >= 4 * n4) continue;
    const float* src = a.proj + a.off + c;
    float4 x[KT - 1 + QP_R];                            // packed rows t0 - (KT - 1) .. t0 + QP_R - 1
#pragma unroll
    for (int i = 0; i < KT - 1 + QP_R; i++) {
      const int t = t0 - (KT - 1) + i;
      x[i] = (t >= 0 && t < a.n_rows) ? ld4(src + (size_t)t * a.ld) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    float4 w[KT];
    if (KT > 1) {
#pragma unroll
      for (int j = 0; j < KT; j++) w[j] = ld4(a.w + (size_t)j * a.C + c);
    } else {
      w[0] = a.w ? ld4(a.w + c) : make_float4(1.f, 1.f, 1.f, 1.f);
    }
#pragma unroll
    for (int r = 0; r < QP_R; r++) {
      float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
      if (r < rows) {
        const float* st = a.state + (size_t)s_slot[r] * (KT - 1) * a.C + c;
#pragma unroll
        for (int j = 0; j < KT; j++) {
          const int back = KT - 1 - j;
          float4 u = x[r + j];
          if (back > s_i[r])                            // in front of the sequence's rows of this step
            u = s_has[r] ? ld4(st + (size_t)(s_i[r] + j) * a.C) : make_float4(0.f, 0.f, 0.f, 0.f);
          fma4(s, w[j], u);
        }
        if (KT > 1 && a.write_state && s_last[r]) {     // (no sequence of the step reads kept rows: see the launcher)
#pragma unroll
          for (int j = 0; j < KT - 1; j++)
            st4(a.state + ((size_t)s_slot[r] * (KT - 1) + j) * a.C + c, KT - 2 - j <= s_i[r] ? x[r + j + 1] : make_float4(0.f, 0.f, 0.f, 0.f));
        }
      }
      y[v][r] = s;
      if (c < nq) sq[r] += dot4(s);
      else if (c < nq + nk) sk[r] += dot4(s);
    }
  }
  if (a.q_w) sums_of_squares<QP_R>(sq, sk, red, tot);
#pragma unroll
  for (int v = 0; v < NV; v++) {
    const int c = 4 * (threadIdx.x + v * blockDim.x);
    if (c >= 4 * n4) continue;
    float4 nw = make_float4(1.f, 1.f, 1.f, 1.f);
    if (a.q_w && c < nq + nk) nw = c < nq ? ld4(a.q_w + c) : ld4(a.k_w + (c - nq));
#pragma unroll
    for (int r = 0; r < QP_R; r++) {
      if (r >= rows) break;
      const float rq = a.q_w ? 1.0f / sqrtf(tot[2 * r] * a.q_inv_n + a.eps) : 1.f, rk = a.q_w ? 1.0f / sqrtf(tot[2 * r + 1] * a.k_inv_n + a.eps) : 1.f;
      finish<T>(a, y[v][r], c, nw, rq, rk, cs + r * a.rot, t0 + r, s_page[r], s_prow[r]);
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
  tlc_wait(a.proj, a.out, a.q_out, a.k_pages, a.v_pages);
  float sq[1] = {0.f}, sk[1] = {0.f};
#pragma unroll
  for (int v = 0; v < NV; v++) {
    const int c = 4 * (threadIdx.x + v * blockDim.x);
    if (c >= 4 * n4) continue;
    const float4 u = ld4(a.proj + (size_t)t * a.ld + a.off + c);
    fma4(s[v], w_new[v], u);
    if (KT > 1) st4(st + (size_t)(KT - 2) * a.C + c, u);
    if (c < nq) sq[0] += dot4(s[v]);
    else if (c < nq + nk) sk[0] += dot4(s[v]);
  }
  float rq = 1.f, rk = 1.f;
  if (a.q_w) {
    sums_of_squares<1>(sq, sk, red, tot);
    rq = 1.0f / sqrtf(tot[0] * a.q_inv_n + a.eps);
    rk = 1.0f / sqrtf(tot[1] * a.k_inv_n + a.eps);
  } else {
    __syncthreads();                                    // (the cosines)
  }
#pragma unroll
  for (int v = 0; v < NV; v++) {
    const int c = 4 * (threadIdx.x + v * blockDim.x);
    if (c < 4 * n4) finish<T>(a, s[v], c, nw[v], rq, rk, cs, t, page, pos % TLC_PAGE);
  }
}

template <typename T, int KT>
void launch(const QpArgs& a, int B, int single, cudaStream_t stream) {
  const int n4 = a.C >> 2;
  // groups a thread: as few as a block of 1,024 threads (512 for prompts, whose rows take registers) allows
  const int most = single ? 1024 : 512;
  const int nv = (n4 + most - 1) / most, need = (n4 + nv - 1) / nv, nt = (need + 31) / 32 * 32;
#define QP_LAUNCH(NV)                                                                                                               \
  if (single) tlc_launch(qkv_prepare_decode_kernel<T, KT, NV>, dim3(B), dim3(nt), (size_t)a.rot * sizeof(float), stream, a);           \
  else tlc_launch(qkv_prepare_rows_kernel<T, KT, NV>, dim3((a.n_rows + QP_R - 1) / QP_R), dim3(nt),                                    \
                  (size_t)QP_R * a.rot * sizeof(float), stream, a)
  if (nv == 1) { QP_LAUNCH(1); }
  else if (nv == 2) { QP_LAUNCH(2); }
  else if (nv == 3) { QP_LAUNCH(3); }
  else { QP_LAUNCH(4); }
#undef QP_LAUNCH
  if (!single && KT > 1 && !a.write_state)
    tlc_launch(qkv_keep_rows_kernel, dim3(B, (n4 + 255) / 256), dim3(256), 0, stream, a);
}

}  // namespace

extern "C" int tlc_qkv_prepare_ok(int H, int KV, int hd, int K, int ld, int off) {
  const long long C = (long long)(H + 2 * KV) * hd;
  return H >= 1 && KV >= 1 && K >= 1 && K <= 4 && hd % 4 == 0 && ld % 4 == 0 && off % 4 == 0 && C <= 8192 && hd <= 1024;
}

extern "C" int tlc_qkv_prepare(const float* proj, int ld, int off, const float* w, int K, float* state, const float* q_w, const float* k_w,
                               int q_count, int k_count, float eps, const float* inv_freq, int rot, float amplitude, const int* positions,
                               const int* row_seq, const int* cu_seqlens, const int* slots, const int* start_pos, const int* block_table,
                               int max_pages, float* out, void* q_out, void* k_pages, void* v_pages, int dtype, int T, int B, int H, int KV,
                               int hd, int single_rows, int all_fresh, cudaStream_t stream) {
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
  const QpArgs a = {proj, ld, off, (H + 2 * KV) * hd, K, w, state, H, KV, hd, q_w, k_w, 1.0f / (float)(q_count > 0 ? q_count : 1),
                    1.0f / (float)(k_count > 0 ? k_count : 1), eps, inv_freq, rot, amplitude, positions, row_seq, cu_seqlens, slots, start_pos,
                    block_table, max_pages, T, all_fresh, out, q_out, k_pages, v_pages};
  TLC_DISPATCH_DTYPE(dtype, TT, {
    if (K == 1) launch<TT, 1>(a, B, single, stream);
    else if (K == 2) launch<TT, 2>(a, B, single, stream);
    else if (K == 3) launch<TT, 3>(a, B, single, stream);
    else launch<TT, 4>(a, B, single, stream);
  });
  TLC_CHECK_LAUNCH("qkv_prepare");
  return 0;
}
