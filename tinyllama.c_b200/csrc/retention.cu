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
