// Polynomial activation over normed powers of a row:
//
//   out = a N(z) + b N(z^2) + c N(z^3) + e,      N(u) = u / sqrt(mean(u^2) + eps) over the row, powers element by element
//
// so a row needs three sums, of z^2, z^4 and z^6.  One block per row; the row stays in registers between the sums and the
// result where it fits (PN_PER_THREAD values a thread), else it is read twice.  Everything is 32-bit but the stored result.
#include "common.cuh"

#define PN_PER_THREAD 16

template <int NT> __device__ __forceinline__ float3 block_sum3(float3 s, float (*red)[3]) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  s.x = warp_sum(s.x); s.y = warp_sum(s.y); s.z = warp_sum(s.z);
  if (NT == 32) return s;
  if (lane == 0) { red[warp][0] = s.x; red[warp][1] = s.y; red[warp][2] = s.z; }
  __syncthreads();
  float3 t = make_float3(0.f, 0.f, 0.f);
#pragma unroll
  for (int w = 0; w < NT / 32; w++) { t.x += red[w][0]; t.y += red[w][1]; t.z += red[w][2]; }
  return t;
}

template <typename TO, int NT, bool VEC>
__global__ void __launch_bounds__(NT)
polynorm_kernel(const float* __restrict__ z, int ldz, int F, float a, float b, float c, float e, float eps, TO* __restrict__ out) {
  tlc_pdl(z, out);
  __shared__ float red[NT / 32][3];
  const float* zr = z + (size_t)blockIdx.x * ldz;
  TO* o = out + (size_t)blockIdx.x * F;
  const bool fits = F <= NT * PN_PER_THREAD;
  float v[PN_PER_THREAD];
  float3 s = make_float3(0.f, 0.f, 0.f);
  auto add = [&](float u) { const float u2 = u * u, u4 = u2 * u2; s.x += u2; s.y += u4; s.z = fmaf(u2, u4, s.z); };
  if (fits) {
#pragma unroll
    for (int j = 0; j < PN_PER_THREAD; j += VEC ? 4 : 1) {
      if (VEC) {
        const int d = (j / 4 * NT + threadIdx.x) * 4;
        const float4 q = d < F ? *reinterpret_cast<const float4*>(zr + d) : make_float4(0.f, 0.f, 0.f, 0.f);
        v[j] = q.x; v[j + (VEC ? 1 : 0)] = q.y; v[j + (VEC ? 2 : 0)] = q.z; v[j + (VEC ? 3 : 0)] = q.w;
      } else {
        const int d = j * NT + threadIdx.x;
        v[j] = d < F ? zr[d] : 0.f;
      }
    }
#pragma unroll
    for (int j = 0; j < PN_PER_THREAD; j++) add(v[j]);
  } else {
    for (int d = threadIdx.x; d < F; d += NT) add(zr[d]);
  }
  s = block_sum3<NT>(s, red);
  const float n = 1.0f / (float)F;
  const float ca = a / sqrtf(s.x * n + eps), cb = b / sqrtf(s.y * n + eps), cc = c / sqrtf(s.z * n + eps);
  auto value = [&](float u) { return fmaf(u, fmaf(u, fmaf(u, cc, cb), ca), e); };
  if (fits) {
#pragma unroll
    for (int j = 0; j < PN_PER_THREAD; j += VEC ? 4 : 1) {
      if (VEC) {
        const int d = (j / 4 * NT + threadIdx.x) * 4;
        if (d < F) {
          const float y0 = value(v[j]), y1 = value(v[j + (VEC ? 1 : 0)]), y2 = value(v[j + (VEC ? 2 : 0)]), y3 = value(v[j + (VEC ? 3 : 0)]);
          if (sizeof(TO) == 4) {
            *reinterpret_cast<float4*>(o + d) = make_float4(y0, y1, y2, y3);
          } else {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(y0, y1), hi = __floats2bfloat162_rn(y2, y3);
            uint2 u;
            u.x = *reinterpret_cast<const unsigned*>(&lo);
            u.y = *reinterpret_cast<const unsigned*>(&hi);
            *reinterpret_cast<uint2*>(o + d) = u;
          }
        }
      } else {
        const int d = j * NT + threadIdx.x;
        if (d < F) o[d] = from_f32<TO>(value(v[j]));
      }
    }
  } else {
    for (int d = threadIdx.x; d < F; d += NT) o[d] = from_f32<TO>(value(zr[d]));
  }
}

// z float [T, F] with row stride ldz; out [T, F] of `dtype`.
extern "C" int tlc_polynorm(const float* z, int ldz, int T, int F, float a, float b, float c, float e, float eps, void* out, int dtype,
                            cudaStream_t stream) {
  if (T == 0 || F == 0) return 0;
  const bool vec = F % 4 == 0 && ldz % 4 == 0 && (uintptr_t)z % 16 == 0 && (uintptr_t)out % 16 == 0;
#define TLC_POLYNORM(NT)                                                                                                          \
  TLC_DISPATCH_DTYPE(dtype, TO, {                                                                                                 \
    if (vec) tlc_launch(polynorm_kernel<TO, NT, true>, dim3(T), dim3(NT), 0, stream, z, ldz, F, a, b, c, e, eps, (TO*)out);         \
    else tlc_launch(polynorm_kernel<TO, NT, false>, dim3(T), dim3(NT), 0, stream, z, ldz, F, a, b, c, e, eps, (TO*)out);            \
  })
  if (F <= 512) { TLC_POLYNORM(32); }
  else if (F <= 2048) { TLC_POLYNORM(128); }
  else if (F <= 4096) { TLC_POLYNORM(256); }
  else if (F <= 8192) { TLC_POLYNORM(512); }
  else { TLC_POLYNORM(1024); }
#undef TLC_POLYNORM
  TLC_CHECK_LAUNCH("polynorm");
  return 0;
}
