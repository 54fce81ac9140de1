// Retention: linear attention with one fixed decay per head and no softmax or denominator.
//
// Per head, with the token's rotated query q and rotated key k (dk values, the key times dk^-1/2), value v (dv values) and
// the head's decay a:
//   S <- a S + k v^T;   o = S^T q;   out = o / sqrt(mean(o^2) + eps) * silu(gate)
// S is 32-bit, zero at position 0 and kept per sequence between steps; it is stored value by value, [H, dv, dk], the
// layout of the selective scan's state (mamba.cu): with the decay as a step's factor, k, q as its B, C and a step size of
// one the two recurrences are the same, so the row-by-row and the chunked 32-bit scans there serve this one.
//
//   tlc_retention_prepare   rotates and scales q and k of prompt rows and lays v | k | q out as those scans read them
//   tlc_retention_decode    one-token steps, everything between the projections and the output projection in one kernel
//   tlc_retention_chunked   prompts of a bfloat16 run in chunks, as products of 32-bit values on the tensor cores
#include "common.cuh"

// Split-half rotation of dimension d of a head at `pos`: dimensions i and i + half of the first 2 * half are a pair.
__device__ __forceinline__ float rotated(const float* __restrict__ x, int d, int half, const float* __restrict__ inv_freq, float pos) {
  if (d >= 2 * half) return x[d];
  const int i = d < half ? d : d - half;
  float sn, cs;
  sincosf(pos * inv_freq[i], &sn, &cs);
  const float u = x[i], w = x[i + half];
  return d < half ? u * cs - w * sn : w * cs + u * sn;
}

// grid (T): vkq [T, H * dv | H * dk | H * dk], ones [T, H], decays [T, H] (the scans' step sizes and factors).
__global__ void __launch_bounds__(256)
retention_prepare_kernel(const float* __restrict__ proj, int ld, int q_off, int k_off, int v_off, const float* __restrict__ inv_freq,
                         int half, const int* __restrict__ positions, const float* __restrict__ decay, float k_scale, int H, int dk,
                         int dv, float* __restrict__ vkq, float* __restrict__ ones, float* __restrict__ decays) {
  tlc_pdl(proj, vkq, ones, decays);
  extern __shared__ float cs_sn[];                       // [half] cos | [half] sin
  const int t = blockIdx.x;
  const float pos = (float)positions[t];
  for (int i = threadIdx.x; i < half; i += 256) sincosf(pos * inv_freq[i], &cs_sn[half + i], &cs_sn[i]);
  __syncthreads();
  const float* row = proj + (size_t)t * ld;
  const int nv = H * dv, nk = H * dk;
  float* o = vkq + (size_t)t * (nv + 2 * nk);
  for (int c = threadIdx.x; c < nv; c += 256) o[c] = row[v_off + c];
  for (int c = threadIdx.x; c < 2 * nk; c += 256) {
    const bool is_k = c < nk;
    const int cc = is_k ? c : c - nk, h = cc / dk, d = cc - h * dk;
    const float* x = row + (is_k ? k_off : q_off) + (size_t)h * dk;
    float y = x[d];
    if (d < 2 * half) {
      const int i = d < half ? d : d - half;
      const float cs = cs_sn[i], sn = cs_sn[half + i], u = x[i], w = x[i + half];
      y = d < half ? u * cs - w * sn : w * cs + u * sn;
    }
    o[nv + c] = is_k ? y * k_scale : y;
  }
  for (int h = threadIdx.x; h < H; h += 256) {
    ones[(size_t)t * H + h] = 1.0f;
    decays[(size_t)t * H + h] = decay[h];
  }
}

extern "C" int tlc_retention_prepare(const float* proj, int ld, int q_off, int k_off, int v_off, const float* inv_freq, int rope_dim,
                                     const int* positions, const float* decay, float k_scale, int T, int H, int dk, int dv, float* vkq,
                                     float* ones, float* decays, cudaStream_t stream) {
  if (T == 0) return 0;
  TLC_REQUIRE(rope_dim % 2 == 0 && rope_dim <= dk && rope_dim <= 4096, "retention: rotated width %d must be even and at most %d", rope_dim, dk);
  tlc_launch(retention_prepare_kernel, dim3(T), dim3(256), (size_t)rope_dim * sizeof(float), stream, proj, ld, q_off, k_off, v_off, inv_freq,
             rope_dim / 2, positions, decay, k_scale, H, dk, dv, vkq, ones, decays);
  TLC_CHECK_LAUNCH("retention_prepare");
  return 0;
}

// One token per sequence.  grid (H, B), 8 warps: a warp takes the value rows warp, warp + 8, ... of the head's state, RP at a
// time; a lane holds the key columns 4 lane + 128 j (VEC) or lane + 32 j of each.  The first RP rows a warp takes are
// fetched before the wait on the previous kernel: an earlier step wrote them.
template <typename TO, int NC, bool VEC, int RP>
__global__ void __launch_bounds__(256)
retention_decode_kernel(const float* __restrict__ proj, int ld, int q_off, int k_off, int v_off, int g_off,
                        const float* __restrict__ inv_freq, int half, const int* __restrict__ positions, const int* __restrict__ slots,
                        const float* __restrict__ decay, float k_scale, float eps, float* state, int H, int dk, int dv,
                        TO* __restrict__ out, int out_ld) {
  asm volatile("griddepcontrol.launch_dependents;");
  constexpr int W = VEC ? 4 : 1, DP = NC * 32 * W;
  extern __shared__ float sh[];                          // q [DP] | k [DP] | v [dv] | o [dv]
  __shared__ float red[33];
  float *qs = sh, *ks = sh + DP, *vs = ks + DP, *os = vs + dv;
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int pos = positions[b];
  const float a = decay[h];
  float* st = state + ((size_t)slots[b] * H + h) * dv * dk;
  float S[RP][NC * W];
  auto fetch = [&](int v0) {
#pragma unroll
    for (int r = 0; r < RP; r++) {
      const int v = v0 + warp + 8 * r;
#pragma unroll
      for (int j = 0; j < NC; j++) {
        const int d = (lane + 32 * j) * W;
        const bool there = pos > 0 && v < dv && d < dk;
        if (VEC) {
          const float4 q = there ? *reinterpret_cast<const float4*>(st + (size_t)v * dk + d) : make_float4(0.f, 0.f, 0.f, 0.f);
          S[r][j * W] = q.x; S[r][j * W + (VEC ? 1 : 0)] = q.y; S[r][j * W + (VEC ? 2 : 0)] = q.z; S[r][j * W + (VEC ? 3 : 0)] = q.w;
        } else {
          S[r][j] = there ? st[(size_t)v * dk + d] : 0.f;
        }
      }
    }
  };
  fetch(0);
  tlc_wait(proj, out);
  const float* row = proj + (size_t)b * ld;
  for (int d = tid; d < DP; d += 256) {
    qs[d] = d < dk ? rotated(row + q_off + (size_t)h * dk, d, half, inv_freq, (float)pos) : 0.f;
    ks[d] = d < dk ? rotated(row + k_off + (size_t)h * dk, d, half, inv_freq, (float)pos) * k_scale : 0.f;
  }
  for (int d = tid; d < dv; d += 256) vs[d] = row[v_off + (size_t)h * dv + d];
  __syncthreads();
  for (int v0 = 0; v0 < dv; v0 += 8 * RP) {
    if (v0 > 0) fetch(v0);
    float o[RP];
#pragma unroll
    for (int r = 0; r < RP; r++) o[r] = 0.f;
#pragma unroll
    for (int j = 0; j < NC; j++) {
      const int d = (lane + 32 * j) * W;
      float kk[W], qq[W];
#pragma unroll
      for (int e = 0; e < W; e++) { kk[e] = ks[d + e]; qq[e] = qs[d + e]; }
#pragma unroll
      for (int r = 0; r < RP; r++) {
        const int v = v0 + warp + 8 * r;
        const float vv = v < dv ? vs[v] : 0.f;
#pragma unroll
        for (int e = 0; e < W; e++) {
          const float s = fmaf(a, S[r][j * W + e], kk[e] * vv);
          S[r][j * W + e] = s;
          o[r] = fmaf(s, qq[e], o[r]);
        }
        if (v < dv && d < dk) {
          if (VEC) *reinterpret_cast<float4*>(st + (size_t)v * dk + d) =
              make_float4(S[r][j * W], S[r][j * W + (VEC ? 1 : 0)], S[r][j * W + (VEC ? 2 : 0)], S[r][j * W + (VEC ? 3 : 0)]);
          else st[(size_t)v * dk + d] = S[r][j];
        }
      }
    }
#pragma unroll
    for (int r = 0; r < RP; r++) {
      o[r] = warp_sum(o[r]);
      const int v = v0 + warp + 8 * r;
      if (lane == 0 && v < dv) os[v] = o[r];
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int d = tid; d < dv; d += 256) ss = fmaf(os[d], os[d], ss);
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)dv + eps);
  for (int d = tid; d < dv; d += 256)
    out[(size_t)b * out_ld + (size_t)h * dv + d] = from_f32<TO>(os[d] * inv * silu_f(row[g_off + (size_t)h * dv + d]));
}

// proj float [B, ld]: q, k (H heads of dk), v and the gate (H heads of dv) from their column offsets; state float
// [n_slots, H, dv, dk]; out [B, out_ld] of out_dtype.  Row b belongs to sequence b.
extern "C" int tlc_retention_decode(const float* proj, int ld, int q_off, int k_off, int v_off, int g_off, const float* inv_freq,
                                    int rope_dim, const int* positions, const int* slots, const float* decay, float k_scale, float eps,
                                    float* state, int B, int H, int dk, int dv, void* out, int out_dtype, int out_ld,
                                    cudaStream_t stream) {
  if (B == 0) return 0;
  TLC_REQUIRE(dk >= 1 && dk <= 256 && dv >= 1 && dv <= 4096, "retention: heads of %d x %d are outside what the kernel is built for (256 x 4096)", dk, dv);
  TLC_REQUIRE(rope_dim % 2 == 0 && rope_dim <= dk, "retention: rotated width %d must be even and at most %d", rope_dim, dk);
  TLC_REQUIRE(H <= 65535 && B <= 65535, "retention: too many heads (%d) or sequences (%d)", H, B);
  const bool vec = dk % 4 == 0 && (uintptr_t)state % 16 == 0;
#define TLC_RETENTION(NC, VEC, RP)                                                                                                    \
  TLC_DISPATCH_DTYPE(out_dtype, TO, tlc_launch(retention_decode_kernel<TO, NC, VEC, RP>, dim3(H, B), dim3(256),                         \
      (size_t)(2 * NC * 32 * (VEC ? 4 : 1) + 2 * dv) * sizeof(float), stream, proj, ld, q_off, k_off, v_off, g_off, inv_freq,            \
      rope_dim / 2, positions, slots, decay, k_scale, eps, state, H, dk, dv, (TO*)out, out_ld))
  if (vec) {
    if (dk <= 128) { TLC_RETENTION(1, true, 16); } else { TLC_RETENTION(2, true, 8); }
  } else {
    if (dk <= 32) { TLC_RETENTION(1, false, 16); } else if (dk <= 64) { TLC_RETENTION(2, false, 16); } else if (dk <= 128) { TLC_RETENTION(4, false, 8); }
    else { TLC_RETENTION(8, false, 4); }
  }
#undef TLC_RETENTION
  TLC_CHECK_LAUNCH("retention_decode");
  return 0;
}

// ---- prompts, in chunks on the tensor cores -------------------------------------------------------------------------------------
// With the state S_0 in front of a chunk and its rows counted from 0, the recurrence is
//   o_i = a^(i+1) S_0^T q_i + sum_{j <= i} a^(i-j) (q_i . k_j) v_j,        S_n = a^n S_0 + sum_j a^(n-1-j) k_j v_j^T
// so three kernels serve a prompt cut into chunks of up to RET_C rows:
//   1. per (chunk, head): q and k are rotated in place in the projection (k times k_scale) and the chunk's own contribution
//      to the state, sum_j a^(n-1-j) v_j k_j^T, is formed;
//   2. the states are carried through every sequence's chunks (the selective scan's pass, mamba.cu);
//   3. per (chunk, head): the scores q_i . k_j with their decays, their product with the values and the share of the state
//      in front of the chunk; the head's norm and gate follow in the same kernel.
// The products are of 32-bit values: each operand is split into two TF32 numbers, x = hi + lo (11 bits each), and hi hi' +
// hi lo' + lo hi' is summed in 32 bits by mma.sync (what is left out is below 2^-21 of a term).
#define RET_C 64

struct Split { uint32_t hi, lo; };
__device__ __forceinline__ Split tf32_split(float x) {
  Split s;
  s.hi = (__float_as_uint(x) + 0x1000u) & 0xffffe000u;           // nearest number of 11 significant bits
  s.lo = __float_as_uint(x - __uint_as_float(s.hi)) & 0xffffe000u;
  return s;
}
__device__ __forceinline__ void mma_tf32(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// One 16 x 8 operand tile, split.
struct TileA {
  uint32_t hi[4], lo[4];
  __device__ __forceinline__ void set(float x0, float x1, float x2, float x3) {
    const Split s0 = tf32_split(x0), s1 = tf32_split(x1), s2 = tf32_split(x2), s3 = tf32_split(x3);
    hi[0] = s0.hi; hi[1] = s1.hi; hi[2] = s2.hi; hi[3] = s3.hi;
    lo[0] = s0.lo; lo[1] = s1.lo; lo[2] = s2.lo; lo[3] = s3.lo;
  }
};
// The three products of M x Q tiles, one kind after the other, so that products into one accumulator do not follow one another.
template <int M, int Q, int N>
__device__ __forceinline__ void mma_split(float (&c)[M][N][4], int q0, const TileA (&a)[M], const Split (&b)[Q][2]) {
#pragma unroll
  for (int q = 0; q < Q; q++)
#pragma unroll
    for (int m = 0; m < M; m++)
      if (q0 + q < N) mma_tf32(c[m][q0 + q < N ? q0 + q : 0], a[m].lo, b[q][0].hi, b[q][1].hi);
#pragma unroll
  for (int q = 0; q < Q; q++)
#pragma unroll
    for (int m = 0; m < M; m++)
      if (q0 + q < N) mma_tf32(c[m][q0 + q < N ? q0 + q : 0], a[m].hi, b[q][0].lo, b[q][1].lo);
#pragma unroll
  for (int q = 0; q < Q; q++)
#pragma unroll
    for (int m = 0; m < M; m++)
      if (q0 + q < N) mma_tf32(c[m][q0 + q < N ? q0 + q : 0], a[m].hi, b[q][0].hi, b[q][1].hi);
}

__device__ __forceinline__ void ret_cp16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void ret_cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void ret_cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// Kernel 1.  grid (chunks, H), 8 warps: warp (wm, wn) = (warp / 4, warp % 4) forms the value rows wm * 16 MT .. of the chunk's
// contribution [dv, dk] and its key columns wn * 8 NT ...  Shared memory: k scaled by its decay [RET_C][LDK], v [RET_C][LDV],
// cosines and sines [RET_C][2 half]; LDK and LDV are 8 above a multiple of 32, so that the fragments' reads (four rows of
// eight neighbouring values) meet all banks.
template <int MT, int NT>
__global__ void __launch_bounds__(256)
retention_chunk_state_kernel(float* proj, int ld, int q_off, int k_off, int v_off, const float* __restrict__ inv_freq, int half,
                             const int* __restrict__ positions, const float* __restrict__ decay, float k_scale,
                             const int* __restrict__ seg_start, int H, int dk, int dv, float* __restrict__ chunk_state,
                             float* __restrict__ chunk_decay) {
  tlc_pdl(proj, chunk_state, chunk_decay);
  constexpr int DVP = 32 * MT, DKP = 32 * NT, LDK = DKP + 8, LDV = DVP + 8;
  extern __shared__ __align__(16) float sh[];
  __shared__ float pw[RET_C + 1];
  float *ks = sh, *vs = ks + RET_C * LDK, *cs = vs + RET_C * LDV;
  const int seg = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int t0 = seg_start[seg], n = min(seg_start[seg + 1] - t0, RET_C);
  const float a = decay[h];
  if (tid <= RET_C) pw[tid] = powf(a, (float)tid);
  if (n < RET_C || dk < DKP || dv < DVP)                  // rows and columns that no copy fills
    for (int i = tid; i < RET_C * (LDK + LDV); i += 256) sh[i] = 0.f;
  // pairs of four dimensions each (the rotated ones), then four dimensions that are only scaled; a thread takes BATCH items
  // at a time and fetches the first ones before the cosines are computed
  constexpr int BATCH = 4;
  const int p4 = half >> 2, per = p4 + ((dk - 2 * half) >> 2), items = n * per;
  float4 qa[BATCH], qb[BATCH], ka[BATCH], kb[BATCH];
  auto fetch = [&](int i0) {
#pragma unroll
    for (int u = 0; u < BATCH; u++) {
      const int i = i0 + 256 * u;
      if (i >= items) break;
      const int r = i / per, it = i - r * per;
      const float* row = proj + (size_t)(t0 + r) * ld + (size_t)h * dk;
      if (it < p4) {
        qa[u] = *reinterpret_cast<const float4*>(row + q_off + 4 * it);
        qb[u] = *reinterpret_cast<const float4*>(row + q_off + half + 4 * it);
        ka[u] = *reinterpret_cast<const float4*>(row + k_off + 4 * it);
        kb[u] = *reinterpret_cast<const float4*>(row + k_off + half + 4 * it);
      } else {
        ka[u] = *reinterpret_cast<const float4*>(row + k_off + 2 * half + 4 * (it - p4));
      }
    }
  };
  fetch(tid);
  for (int i = tid; i < n * half; i += 256) {
    const int r = i / half, j = i - r * half;
    sincosf((float)positions[t0 + r] * inv_freq[j], &cs[r * 2 * half + half + j], &cs[r * 2 * half + j]);
  }
  __syncthreads();
  const int dv4 = dv >> 2;
  for (int i = tid; i < n * dv4; i += 256) {
    const int r = i / dv4, c = (i - r * dv4) << 2;
    ret_cp16(vs + r * LDV + c, proj + (size_t)(t0 + r) * ld + v_off + (size_t)h * dv + c);
  }
  ret_cp_commit();
  for (int i0 = tid; i0 < items; i0 += 256 * BATCH) {
    if (i0 != tid) fetch(i0);
#pragma unroll
    for (int u = 0; u < BATCH; u++) {
      const int i = i0 + 256 * u;
      if (i >= items) break;
      const int r = i / per, it = i - r * per;
      float* row = proj + (size_t)(t0 + r) * ld + (size_t)h * dk;
      const float w = pw[n - 1 - r];
      float* kd = ks + r * LDK;
      if (it < p4) {
        const int d = 4 * it;
        const float4 c = *reinterpret_cast<const float4*>(cs + r * 2 * half + d), s = *reinterpret_cast<const float4*>(cs + r * 2 * half + half + d);
        float4 y = qa[u], x = qb[u];
        *reinterpret_cast<float4*>(row + q_off + d) = make_float4(y.x * c.x - x.x * s.x, y.y * c.y - x.y * s.y, y.z * c.z - x.z * s.z, y.w * c.w - x.w * s.w);
        *reinterpret_cast<float4*>(row + q_off + half + d) = make_float4(x.x * c.x + y.x * s.x, x.y * c.y + y.y * s.y, x.z * c.z + y.z * s.z, x.w * c.w + y.w * s.w);
        y = ka[u];
        x = kb[u];
        const float4 lo = make_float4((y.x * c.x - x.x * s.x) * k_scale, (y.y * c.y - x.y * s.y) * k_scale, (y.z * c.z - x.z * s.z) * k_scale,
                                      (y.w * c.w - x.w * s.w) * k_scale);
        const float4 hi = make_float4((x.x * c.x + y.x * s.x) * k_scale, (x.y * c.y + y.y * s.y) * k_scale, (x.z * c.z + y.z * s.z) * k_scale,
                                      (x.w * c.w + y.w * s.w) * k_scale);
        *reinterpret_cast<float4*>(row + k_off + d) = lo;
        *reinterpret_cast<float4*>(row + k_off + half + d) = hi;
        *reinterpret_cast<float4*>(kd + d) = make_float4(lo.x * w, lo.y * w, lo.z * w, lo.w * w);
        *reinterpret_cast<float4*>(kd + half + d) = make_float4(hi.x * w, hi.y * w, hi.z * w, hi.w * w);
      } else {
        const int d = 2 * half + 4 * (it - p4);
        const float4 y = make_float4(ka[u].x * k_scale, ka[u].y * k_scale, ka[u].z * k_scale, ka[u].w * k_scale);
        *reinterpret_cast<float4*>(row + k_off + d) = y;
        *reinterpret_cast<float4*>(kd + d) = make_float4(y.x * w, y.y * w, y.z * w, y.w * w);
      }
    }
  }
  ret_cp_wait<0>();
  __syncthreads();
  const int g = lane >> 2, t = lane & 3, m0 = (warp >> 2) * 16 * MT, n0 = (warp & 3) * 8 * NT;
  float acc[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; m++)
#pragma unroll
    for (int q = 0; q < NT; q++)
#pragma unroll
      for (int e = 0; e < 4; e++) acc[m][q][e] = 0.f;
  const int steps = (n + 7) >> 3;
  for (int s = 0; s < steps; s++) {
    const float *v0 = vs + (8 * s + t) * LDV + g, *v4 = v0 + 4 * LDV, *k0 = ks + (8 * s + t) * LDK + g, *k4 = k0 + 4 * LDK;
    TileA A[MT];
#pragma unroll
    for (int m = 0; m < MT; m++) A[m].set(v0[m0 + 16 * m], v0[m0 + 16 * m + 8], v4[m0 + 16 * m], v4[m0 + 16 * m + 8]);
    constexpr int QS = NT % 2 == 0 ? 2 : 1;               // (column tiles at a time)
#pragma unroll
    for (int q = 0; q < NT; q += QS) {
      Split b[QS][2];
#pragma unroll
      for (int j = 0; j < QS; j++) { b[j][0] = tf32_split(k0[n0 + 8 * (q + j)]); b[j][1] = tf32_split(k4[n0 + 8 * (q + j)]); }
      mma_split<MT, QS, NT>(acc, q, A, b);
    }
  }
  float* u = chunk_state + ((size_t)seg * H + h) * dv * dk;
#pragma unroll
  for (int m = 0; m < MT; m++)
#pragma unroll
    for (int q = 0; q < NT; q++) {
      const int v = m0 + 16 * m + g, k = n0 + 8 * q + 2 * t;
      if (k < dk) {                                       // (dk is even: a pair is inside or outside)
        if (v < dv) *reinterpret_cast<float2*>(u + (size_t)v * dk + k) = make_float2(acc[m][q][0], acc[m][q][1]);
        if (v + 8 < dv) *reinterpret_cast<float2*>(u + (size_t)(v + 8) * dk + k) = make_float2(acc[m][q][2], acc[m][q][3]);
      }
    }
  if (tid == 0) chunk_decay[(size_t)seg * H + h] = pw[n];
}

// Kernel 3.  grid (chunks, H), 8 warps: warp (wr, wc) = (warp / 4, warp % 4) takes rows 32 wr .. + 31 and, of every 32 value
// columns, the eight from 8 wc.  Shared memory, small enough for two blocks on an SM: q and k in rows of LDK (the scores take
// k's place), and one more buffer that holds in turn up to 64 columns of the state in front of the chunk (rows of LDK), the
// next 64, and the values (rows of LDV).  LDK and LDV are 4 above a multiple of 32: a fragment's reads meet all banks.  The
// scores' fragments pair their columns 2 t and 2 t + 1 with the value rows of the same numbers.
template <typename TO, int NT>
__global__ void __launch_bounds__(256, 2)
retention_chunk_out_kernel(const float* __restrict__ proj, int ld, int q_off, int k_off, int v_off, int g_off,
                           const float* __restrict__ decay, float eps, const float* __restrict__ chunk_state,
                           const int* __restrict__ seg_start, const int* __restrict__ seg_seq, const int* __restrict__ seq_seg_start,
                           const int* __restrict__ start_pos, int H, int dk, int dv, int LDK, TO* __restrict__ out, int out_ld) {
  tlc_pdl(proj, chunk_state, out);
  constexpr int DVP = 32 * NT, LDV = DVP + 4, LDP = RET_C + 4, PIECE = NT < 2 ? NT : 2;     // n-tiles of a piece of the state
  extern __shared__ __align__(16) float sh[];
  __shared__ float pw[RET_C + 1], red[RET_C][4];
  float *qs = sh, *ks = qs + RET_C * LDK, *buf = ks + RET_C * max(LDK, LDP);
  const int seg = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int t0 = seg_start[seg], n = min(seg_start[seg + 1] - t0, RET_C);
  const int b = seg_seq[seg];
  const bool empty = seg == seq_seg_start[b] && start_pos[b] == 0;         // nothing in front of the chunk
  const float a = decay[h];
  const int dkp = (dk + 7) & ~7, dk4 = dk >> 2, dv4 = dv >> 2;
  const bool padded = n < RET_C || dk < dkp || dv < DVP;
  if (tid <= RET_C) pw[tid] = powf(a, (float)tid);
  const int buf_floats = max(PIECE * 32 * LDK, RET_C * LDV);
  if (padded) {                                           // rows and columns that no copy fills
    const int total = RET_C * (LDK + max(LDK, LDP)) + buf_floats;
    for (int i = tid; i < total; i += 256) sh[i] = 0.f;
    __syncthreads();
  }
  for (int i = tid; i < n * dk4; i += 256) {
    const int r = i / dk4, c = (i - r * dk4) << 2;
    const float* row = proj + (size_t)(t0 + r) * ld + (size_t)h * dk + c;
    ret_cp16(qs + r * LDK + c, row + q_off);
    ret_cp16(ks + r * LDK + c, row + k_off);
  }
  ret_cp_commit();
  // value columns 32 p .. of the state (row v of it is a row of dk), PIECE * 32 of them; rows past dv stay as they are (they
  // meet columns of the result that nobody stores)
  auto load_state = [&](int p) {
    const int first = 32 * p, rows = min(dv - first, 32 * PIECE);
    for (int i = tid; i < rows * dk4; i += 256) {
      const int r = i / dk4, c = (i - r * dk4) << 2;
      ret_cp16(buf + r * LDK + c, chunk_state + (((size_t)seg * H + h) * dv + first + r) * dk + c);
    }
    ret_cp_commit();
  };
  auto load_values = [&]() {
    for (int i = tid; i < n * dv4; i += 256) {
      const int r = i / dv4, c = (i - r * dv4) << 2;
      ret_cp16(buf + r * LDV + c, proj + (size_t)(t0 + r) * ld + v_off + (size_t)h * dv + c);
    }
    ret_cp_commit();
  };
  if (empty) load_values(); else load_state(0);
  ret_cp_wait<1>();
  __syncthreads();
  const int g = lane >> 2, t = lane & 3, r0 = (warp >> 2) * 32, wc = warp & 3;
  // the scores of rows r0 .. + 31 and columns 16 wc .. + 15 (above the diagonal there is nothing)
  float p[2][2][4];
#pragma unroll
  for (int m = 0; m < 2; m++)
#pragma unroll
    for (int q = 0; q < 2; q++)
#pragma unroll
      for (int e = 0; e < 4; e++) p[m][q][e] = 0.f;
  if (16 * wc < r0 + 32)
#pragma unroll 2
    for (int d = 0; d < dkp; d += 8) {
      TileA A[2];
#pragma unroll
      for (int m = 0; m < 2; m++) {
        const float* x = qs + (r0 + 16 * m + g) * LDK + d + t;
        A[m].set(x[0], x[8 * LDK], x[4], x[8 * LDK + 4]);
      }
      Split kb[2][2];
#pragma unroll
      for (int q = 0; q < 2; q++) {
        const float* y = ks + (16 * wc + 8 * q + g) * LDK + d + t;
        kb[q][0] = tf32_split(y[0]);
        kb[q][1] = tf32_split(y[4]);
      }
      mma_split<2, 2, 2>(p, 0, A, kb);
    }
  __syncthreads();                                        // k has been read
  float* ps = ks;
#pragma unroll
  for (int m = 0; m < 2; m++)
#pragma unroll
    for (int q = 0; q < 2; q++)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int i = r0 + 16 * m + g + (e >> 1) * 8, j = 16 * wc + 8 * q + 2 * t;
        *reinterpret_cast<float2*>(ps + i * LDP + j) = make_float2(j <= i ? p[m][q][e] * pw[i - j] : 0.f, j + 1 <= i ? p[m][q][e + 1] * pw[i - j - 1] : 0.f);
      }
  float acc[2][NT][4];
#pragma unroll
  for (int m = 0; m < 2; m++)
#pragma unroll
    for (int q = 0; q < NT; q++)
#pragma unroll
      for (int e = 0; e < 4; e++) acc[m][q][e] = 0.f;
  if (!empty) {
#pragma unroll
    for (int q0 = 0; q0 < NT; q0 += PIECE) {
      ret_cp_wait<0>();
      __syncthreads();                                    // this piece of the state has landed
#pragma unroll 2
      for (int d = 0; d < dkp; d += 8) {
        TileA A[2];
#pragma unroll
        for (int m = 0; m < 2; m++) {
          const float* x = qs + (r0 + 16 * m + g) * LDK + d + t;
          A[m].set(x[0], x[8 * LDK], x[4], x[8 * LDK + 4]);
        }
        Split sb[PIECE][2];
#pragma unroll
        for (int q = 0; q < PIECE; q++) {
          const float* y = buf + (32 * q + 8 * wc + g) * LDK + d + t;
          sb[q][0] = tf32_split(y[0]);
          sb[q][1] = tf32_split(y[4]);
        }
        mma_split<2, PIECE, NT>(acc, q0, A, sb);
      }
      __syncthreads();                                    // the buffer has been read
      if (q0 + PIECE < NT) {
        load_state(q0 + PIECE);
      } else {
        if (padded) {
          for (int i = tid; i < buf_floats; i += 256) buf[i] = 0.f;
          __syncthreads();
        }
        load_values();
      }
    }
#pragma unroll
    for (int m = 0; m < 2; m++) {
      const float w0 = pw[r0 + 16 * m + g + 1], w1 = pw[r0 + 16 * m + g + 9];
#pragma unroll
      for (int q = 0; q < NT; q++) {
        acc[m][q][0] *= w0; acc[m][q][1] *= w0;
        acc[m][q][2] *= w1; acc[m][q][3] *= w1;
      }
    }
  }
  ret_cp_wait<0>();
  __syncthreads();                                        // the values and every warp's scores are there
  const int last = min(r0 + 32, (n + 7) & ~7);            // later columns meet no row of this warp
  for (int j = 0; j < last; j += 8) {
    TileA A[2];
#pragma unroll
    for (int m = 0; m < 2; m++) {
      const float2 x = *reinterpret_cast<const float2*>(ps + (r0 + 16 * m + g) * LDP + j + 2 * t);
      const float2 y = *reinterpret_cast<const float2*>(ps + (r0 + 16 * m + g + 8) * LDP + j + 2 * t);
      A[m].set(x.x, y.x, x.y, y.y);
    }
    Split vb[NT][2];
#pragma unroll
    for (int q = 0; q < NT; q++) {
      const float* y = buf + (j + 2 * t) * LDV + 32 * q + 8 * wc + g;
      vb[q][0] = tf32_split(y[0]);
      vb[q][1] = tf32_split(y[LDV]);
    }
    mma_split<2, NT, NT>(acc, 0, A, vb);
  }
  // the head's norm over all value columns (four warps share a row), then the gate
#pragma unroll
  for (int m = 0; m < 2; m++) {
    float s0 = 0.f, s1 = 0.f;
#pragma unroll
    for (int q = 0; q < NT; q++) {
      if (32 * q + 8 * wc + 2 * t >= dv) continue;        // (what stands in columns past the head's is of no account)
      s0 += acc[m][q][0] * acc[m][q][0] + acc[m][q][1] * acc[m][q][1];
      s1 += acc[m][q][2] * acc[m][q][2] + acc[m][q][3] * acc[m][q][3];
    }
    s0 += __shfl_xor_sync(0xffffffffu, s0, 1); s0 += __shfl_xor_sync(0xffffffffu, s0, 2);
    s1 += __shfl_xor_sync(0xffffffffu, s1, 1); s1 += __shfl_xor_sync(0xffffffffu, s1, 2);
    if (t == 0) { red[r0 + 16 * m + g][wc] = s0; red[r0 + 16 * m + g + 8][wc] = s1; }
  }
  __syncthreads();
  const bool pairs = out_ld % 2 == 0 && (uintptr_t)out % 4 == 0;
#pragma unroll
  for (int m = 0; m < 2; m++)
#pragma unroll
    for (int e = 0; e < 2; e++) {
      const int r = r0 + 16 * m + g + 8 * e;
      if (r >= n) continue;
      const float inv = 1.0f / sqrtf((red[r][0] + red[r][1] + red[r][2] + red[r][3]) / (float)dv + eps);
      const float* gate = proj + (size_t)(t0 + r) * ld + g_off + (size_t)h * dv;
      TO* o = out + (size_t)(t0 + r) * out_ld + (size_t)h * dv;
#pragma unroll
      for (int q = 0; q < NT; q++) {
        const int v = 32 * q + 8 * wc + 2 * t;
        if (v < dv) {                                     // (dv is a multiple of 4)
          const float2 z = *reinterpret_cast<const float2*>(gate + v);
          const float y0 = acc[m][q][2 * e] * inv * silu_of<sizeof(TO) == 2>(z.x), y1 = acc[m][q][2 * e + 1] * inv * silu_of<sizeof(TO) == 2>(z.y);
          if (sizeof(TO) == 2 && pairs) {
            *reinterpret_cast<__nv_bfloat162*>(o + v) = __floats2bfloat162_rn(y0, y1);
          } else {
            o[v] = from_f32<TO>(y0);
            o[v + 1] = from_f32<TO>(y1);
          }
        }
      }
    }
}

static int ret_ldk(int dk) { return (dk + 31) / 32 * 32 + 4; }
static size_t ret_out_smem(int dk, int dvp) {
  const int ldk = ret_ldk(dk);
  const int piece = (dvp < 64 ? dvp : 64) * ldk, values = RET_C * (dvp + 4);
  return (size_t)(RET_C * (ldk + (ldk > RET_C + 4 ? ldk : RET_C + 4)) + (piece > values ? piece : values)) * sizeof(float);
}
static size_t ret_state_smem(int dk, int dv, int rope_dim) {
  return (size_t)RET_C * ((dk + 31) / 32 * 32 + 8 + (dv + 31) / 32 * 32 + 8 + rope_dim) * sizeof(float);
}

// Whether prompts of these heads run in chunks on the tensor cores (rope_dim: dimensions of a head that are rotated).
extern "C" int tlc_retention_chunks_ok(int dk, int dv, int rope_dim) {
  return dk >= 4 && dk <= 128 && dv >= 4 && dv <= 128 && dk % 4 == 0 && dv % 4 == 0 && rope_dim % 8 == 0 && rope_dim <= dk;
}

extern "C" int tlc_retention_init() {
  cudaError_t e = cudaSuccess;
  const size_t out_most = ret_out_smem(128, 128), state_most = ret_state_smem(128, 128, 128);
#define RET_ATTR(F, BYTES) if (e == cudaSuccess) e = cudaFuncSetAttribute(F, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(BYTES))
#define RET_OUT_ATTR(NT) RET_ATTR((retention_chunk_out_kernel<float, NT>), out_most); RET_ATTR((retention_chunk_out_kernel<__nv_bfloat16, NT>), out_most)
#define RET_STATE_ATTR(MT) RET_ATTR((retention_chunk_state_kernel<MT, 1>), state_most); RET_ATTR((retention_chunk_state_kernel<MT, 2>), state_most); \
                           RET_ATTR((retention_chunk_state_kernel<MT, 3>), state_most); RET_ATTR((retention_chunk_state_kernel<MT, 4>), state_most)
  RET_OUT_ATTR(1); RET_OUT_ATTR(2); RET_OUT_ATTR(3); RET_OUT_ATTR(4);
  RET_STATE_ATTR(1); RET_STATE_ATTR(2); RET_STATE_ATTR(3); RET_STATE_ATTR(4);
#undef RET_OUT_ATTR
#undef RET_STATE_ATTR
#undef RET_ATTR
  if (e != cudaSuccess) return tlc_fail(-2, "retention: shared memory of the chunk kernels: %s", cudaGetErrorString(e));
  return 0;
}

int tlc_ssm_state_pass_launch(const float* chunk_decay, float* state, float* chunk_state, const int* seq_seg_start, const int* slots,
                              const int* start_pos, int B, int Hs, int PN, int write_final, cudaStream_t stream);

// proj float [T, ld] as for tlc_retention_decode, its q and k columns are rotated in place; chunk tables as for the chunked
// selective scan, no chunk longer than RET_C rows; scratch: n_seg * H * (dk * dv + 1) floats, 16-byte aligned.
extern "C" int tlc_retention_chunked(float* proj, int ld, int q_off, int k_off, int v_off, int g_off, const float* inv_freq, int rope_dim,
                                     const int* positions, const float* decay, float k_scale, float eps, float* state, float* scratch,
                                     const int* seg_start, const int* seg_seq, const int* seq_seg_start, const int* slots,
                                     const int* start_pos, int B, int n_seg, int chunk_rows, int H, int dk, int dv, void* out,
                                     int out_dtype, int out_ld, cudaStream_t stream) {
  if (B == 0 || n_seg == 0) return 0;
  TLC_REQUIRE(tlc_retention_chunks_ok(dk, dv, rope_dim) && chunk_rows <= RET_C && H <= 65535,
              "retention: heads of %d x %d, %d rotated, in chunks of %d rows are outside what the chunk kernels are built for", dk, dv, rope_dim,
              chunk_rows);
  TLC_REQUIRE(ld % 4 == 0 && q_off % 4 == 0 && k_off % 4 == 0 && v_off % 4 == 0 && g_off % 4 == 0 && (uintptr_t)proj % 16 == 0 &&
                  (uintptr_t)scratch % 16 == 0, "retention: the projection's pieces must start on 16-byte boundaries");
  float* chunk_decay = scratch + (size_t)n_seg * H * dk * dv;
  const dim3 grid(n_seg, H);
  const int mt = (dv + 31) / 32, nt = (dk + 31) / 32;
  const size_t smem1 = ret_state_smem(dk, dv, rope_dim), smem3 = ret_out_smem(dk, 32 * mt);
#define RET_STATE(MT, NT)                                                                                                          \
  if (mt == MT && nt == NT)                                                                                                        \
    tlc_launch(retention_chunk_state_kernel<MT, NT>, grid, dim3(256), smem1, stream, proj, ld, q_off, k_off, v_off, inv_freq, rope_dim / 2, \
               positions, decay, k_scale, seg_start, H, dk, dv, scratch, chunk_decay)
#define RET_STATES(MT) RET_STATE(MT, 1); RET_STATE(MT, 2); RET_STATE(MT, 3); RET_STATE(MT, 4)
  RET_STATES(1); RET_STATES(2); RET_STATES(3); RET_STATES(4);
#undef RET_STATES
#undef RET_STATE
  TLC_CHECK_LAUNCH("retention_chunk_state");
  if (int rc = tlc_ssm_state_pass_launch(chunk_decay, state, scratch, seq_seg_start, slots, start_pos, B, H, dk * dv, 1, stream)) return rc;
#define RET_OUT(NT)                                                                                                                 \
  if (mt == NT)                                                                                                                     \
    TLC_DISPATCH_DTYPE(out_dtype, TO, tlc_launch(retention_chunk_out_kernel<TO, NT>, grid, dim3(256), smem3, stream, (const float*)proj, ld, \
        q_off, k_off, v_off, g_off, decay, eps, (const float*)scratch, seg_start, seg_seq, seq_seg_start, start_pos, H, dk, dv,       \
        ret_ldk(dk), (TO*)out, out_ld))
  RET_OUT(1); RET_OUT(2); RET_OUT(3); RET_OUT(4);
#undef RET_OUT
  TLC_CHECK_LAUNCH("retention_chunk_out");
  return 0;
}
