// Mixture of experts: routing, and the experts' gated feed-forwards as grouped products.
//
// Routing (tlc_moe_route): a token's scores are s = sigmoid(router logits), 32-bit; its `top` experts are those with
// the largest scores (the lowest index wins a tie); its weights are the chosen scores as they are.  The kernel also
// sorts the (token, choice) pairs by expert -- counts, offsets, and for every expert the list of its pairs -- so that
// each expert's rows form one contiguous range of a permutation; nothing goes through the host, so the same launches
// serve any routing (and a captured graph).  tlc_moe_route_tables needs no logits: a table gives every token id its
// experts, all of one weight; it depends on the step's tokens alone, so one launch serves every layer of a model.
//
// Experts (tlc_moe_gate_up, tlc_moe_down): an expert is fed the token scaled by its weight, expert(w h); gate and up are
// linear, so W (w h) = w (W h) and the epilogue of the first product applies w in 32 bits: act(w g) * (w u).  The
// second product writes every pair's result into its own row of [T, top, D]; the norm that follows adds a token's rows
// in the order of its choices, so the sum does not depend on where other tokens went.
//
// Both products work on tiles of 32 sorted rows of ONE expert; the grid is an upper bound (pairs / 32 + experts in
// use) and a block past the last tile returns.
#include "common.cuh"

#define MOE_TM 32

// A warp per token: its `top` experts by descending logit (lowest index first on ties) and their weights.  In every pass a
// lane finds the best of its experts (lane, lane + 32, ...) that come after the last choice in that order, and the
// warp the best of the lanes.
__global__ void __launch_bounds__(128)
moe_topk_kernel(const float* __restrict__ logits, int ld, int T, int E, int top, int mode, const float* __restrict__ choice_bias,
                int* __restrict__ ids, float* __restrict__ wts, float sum_to) {
  tlc_pdl(logits, ids, wts);
  const int t = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (t >= T) return;
  const float* lr = logits + (size_t)t * ld;
  float last = INFINITY, first = 0.f, sum = 0.f;
  int last_e = -1;
  // TLC_ROUTE_SOFTMAX_ALL: scores are the softmax over all E outputs; an expert is chosen by score + choice_bias[e] and
  // weighted by the score alone
  float all_max = 0.f, all_inv = 1.0f;
  if (mode == TLC_ROUTE_SOFTMAX_ALL) {
    float m = -INFINITY;
    for (int e = lane; e < E; e += 32) m = fmaxf(m, lr[e]);
    all_max = warp_max(m);
    float s = 0.f;
    for (int e = lane; e < E; e += 32) s += expf(lr[e] - all_max);
    all_inv = 1.0f / warp_sum(s);
  }
  auto rank_of = [&](int e) {
    if (mode != TLC_ROUTE_SOFTMAX_ALL) return lr[e];
    const float s = __fmul_rn(expf(lr[e] - all_max), all_inv);      // (no contraction with the sum: the weight below is this s)
    return choice_bias ? __fadd_rn(s, choice_bias[e]) : s;
  };
  for (int k = 0; k < top; k++) {
    float best = -INFINITY;
    int be = 0x7fffffff;                     // none yet
    for (int e = lane; e < E; e += 32) {
      const float v = rank_of(e);
      const bool after = v < last || (v == last && e > last_e);
      if (after && (be == 0x7fffffff || v > best)) { best = v; be = e; }   // (a lane's experts come in ascending order)
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      const bool take = oe != 0x7fffffff && (be == 0x7fffffff || ov > best || (ov == best && oe < be));
      if (take) { best = ov; be = oe; }
    }
    if (be == 0x7fffffff) be = 0;            // (NaN logits: no order; keep indices valid)
    if (lane == 0) {
      ids[t * top + k] = be;
      if (mode == TLC_ROUTE_SOFTMAX) {       // the first choice has the largest logit: numerators exp(z_k - z_0)
        if (k == 0) first = lr[be];
        const float e = expf(lr[be] - first);
        sum += e;
        wts[t * top + k] = e;
      } else if (mode == TLC_ROUTE_SOFTMAX_ALL) {
        const float w = __fmul_rn(expf(lr[be] - all_max), all_inv);
        sum += w;
        wts[t * top + k] = w;
      } else {
        wts[t * top + k] = 1.0f / (1.0f + expf(-lr[be]));
      }
    }
    last = best;                             // (the value the comparison saw, not one computed anew: the same bits)
    last_e = be;
  }
  if (mode == TLC_ROUTE_SOFTMAX && lane == 0) {
    const float inv = 1.0f / sum;
    for (int k = 0; k < top; k++) wts[t * top + k] *= inv;
  }
  // the chosen scores divided by their sum (+ 1e-20, which keeps a sum of zero finite) and multiplied by sum_to
  if (mode == TLC_ROUTE_SOFTMAX_ALL && sum_to > 0.f && lane == 0) {
    const float inv = 1.0f / (sum + 1e-20f);
    for (int k = 0; k < top; k++) wts[t * top + k] = wts[t * top + k] * inv * sum_to;
  }
}

// A block sorts the pairs by expert: counts, offsets (and every expert's first tile of `tm` sorted rows), then the list order
// [n_pairs]: pair index (t * top + k) of every sorted position.  shi: 2 * E ints.  ids[i] is read by the thread that owns i
// (i modulo the block) only.
__device__ __forceinline__ void moe_sort_pairs(const int* ids, int n_pairs, int E, int E_tiled, int tm, int* __restrict__ order,
                                               int* __restrict__ offsets, int* __restrict__ tile_off, int* shi) {
  int* count = shi;            // [E]
  int* cursor = shi + E;       // [E]
  for (int e = threadIdx.x; e < E; e += blockDim.x) count[e] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < n_pairs; i += blockDim.x) atomicAdd(&count[ids[i]], 1);
  __syncthreads();
  if (threadIdx.x < 32) {      // running sums of pairs and tiles, 32 experts at a time
    const int lane = threadIdx.x;
    int pairs = 0, tiles = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + lane, c = e < E ? count[e] : 0;
      const int k = e < E_tiled ? (c + tm - 1) / tm : 0;       // (the others have no weights: no product visits them)
      int ci = c, ki = k;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int a = __shfl_up_sync(0xffffffffu, ci, o), b = __shfl_up_sync(0xffffffffu, ki, o);
        if (lane >= o) { ci += a; ki += b; }
      }
      if (e < E) {
        offsets[e] = cursor[e] = pairs + ci - c;
        tile_off[e] = tiles + ki - k;
      }
      pairs += __shfl_sync(0xffffffffu, ci, 31);
      tiles += __shfl_sync(0xffffffffu, ki, 31);
    }
    if (lane == 0) {
      offsets[E] = pairs;
      tile_off[E] = tiles;
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < n_pairs; i += blockDim.x) order[atomicAdd(&cursor[ids[i]], 1)] = i;
}

__global__ void __launch_bounds__(1024)
moe_sort_kernel(const int* __restrict__ ids, int n_pairs, int E, int E_tiled, int tm, int* __restrict__ order,
                int* __restrict__ offsets, int* __restrict__ tile_off) {
  tlc_pdl(ids, order, offsets, tile_off);
  extern __shared__ int shi[];
  moe_sort_pairs(ids, n_pairs, E, E_tiled, tm, order, offsets, tile_off, shi);
}

// Routing without a router, for all layers of a model that route this way: block p takes table p.  desc [n, 4] (64-bit): the
// table's address (int [V, top]), its experts E, top, and whether its products may take tiles of 64 rows (they do when an
// expert gets 64 rows or more on average).  Block p writes ids | order | offsets | tile_off from ints + p * ld_ints and the
// weights, 1 / top each, from wts + p * ld_wts.
__global__ void __launch_bounds__(1024)
moe_route_tables_kernel(const int* __restrict__ tokens, const long long* __restrict__ desc, int T, int V, int* ints, int ld_ints, float* wts,
                        int ld_wts) {
  tlc_pdl(tokens, ints, wts);
  extern __shared__ int shi[];
  const long long* d = desc + 4 * (size_t)blockIdx.x;
  const int* table = reinterpret_cast<const int*>(d[0]);
  const int E = (int)d[1], top = (int)d[2], n_pairs = T * top;
  const int tm = (d[3] && (long long)n_pairs >= 64LL * E) ? 64 : 32;
  int* ids = ints + (size_t)blockIdx.x * ld_ints;
  float* w = wts + (size_t)blockIdx.x * ld_wts;
  const float weight = 1.0f / (float)top;
  for (int i = threadIdx.x; i < n_pairs; i += blockDim.x) {
    const int t = i / top;
    int tok = tokens[t];
    tok = tok < 0 ? 0 : (tok >= V ? V - 1 : tok);
    const int e = table[(size_t)tok * top + (i - t * top)];
    ids[i] = e < 0 ? 0 : (e >= E ? E - 1 : e);          // (tables are checked when they are bound; never index out of bounds)
    w[i] = weight;
  }
  int* order = ids + n_pairs;
  int* offsets = order + n_pairs;
  moe_sort_pairs(ids, n_pairs, E, E, tm, order, offsets, offsets + E + 1, shi);
}

extern "C" int tlc_moe_route(const float* logits, int ld, int T, int E, int top, int mode, const float* choice_bias, int n_identity,
                             int* ids, float* wts, int* order, int* offsets, int* tile_off, int tile_rows, float sum_to,
                             cudaStream_t stream) {
  if (T == 0) return 0;
  TLC_REQUIRE(tile_rows >= 1, "moe_route: tiles of %d rows", tile_rows);
  TLC_REQUIRE(E >= 1 && top >= 1 && top <= E && E <= 4096, "moe_route: %d experts, %d chosen", E, top);
  TLC_REQUIRE(mode == TLC_ROUTE_SIGMOID || mode == TLC_ROUTE_SOFTMAX || mode == TLC_ROUTE_SOFTMAX_ALL, "moe_route: unknown weighting %d", mode);
  TLC_REQUIRE(n_identity >= 0 && n_identity < E, "moe_route: %d of %d router outputs without an expert's weights", n_identity, E);
  tlc_launch(moe_topk_kernel, dim3((T + 3) / 4), dim3(128), 0, stream, logits, ld, T, E, top, mode, choice_bias, ids, wts, sum_to);
  TLC_CHECK_LAUNCH("moe_topk");
  tlc_launch(moe_sort_kernel, dim3(1), dim3(1024), (size_t)2 * E * sizeof(int), stream, (const int*)ids, T * top, E, E - n_identity, tile_rows,
             order, offsets, tile_off);
  TLC_CHECK_LAUNCH("moe_sort");
  return 0;
}

extern "C" int tlc_moe_route_tables(const int* tokens, const long long* desc, int n, int T, int V, int max_experts, int* ints, int ld_ints,
                                    float* wts, int ld_wts, cudaStream_t stream) {
  if (T == 0 || n == 0) return 0;
  TLC_REQUIRE(max_experts >= 1 && max_experts <= 4096 && V >= 1, "moe_route_tables: %d experts, %d token ids", max_experts, V);
  tlc_launch(moe_route_tables_kernel, dim3(n), dim3(1024), (size_t)2 * max_experts * sizeof(int), stream, tokens, desc, T, V, ints, ld_ints,
             wts, ld_wts);
  TLC_CHECK_LAUNCH("moe_route_tables");
  return 0;
}

// Which expert and which of its rows a tile covers: the last expert whose first tile is <= tile.
__device__ __forceinline__ bool moe_tile(int tile, const int* __restrict__ tile_off, const int* __restrict__ offsets, int E,
                                         int* expert, int* row0, int* rows) {
  if (tile >= tile_off[E]) return false;
  int lo = 0, hi = E - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (tile_off[mid] <= tile) lo = mid; else hi = mid - 1;
  }
  *expert = lo;
  *row0 = offsets[lo] + (tile - tile_off[lo]) * MOE_TM;
  *rows = min(MOE_TM, offsets[lo + 1] - *row0);
  return true;
}

// act[i, f] = silu(w_i g) * (w_i u) for sorted position i, with g | u = Wgu[e] x[token(i)]; Wgu [E, 2F, D] (F gate rows,
// then F up rows).  Tile: 32 rows x 32 features, both halves.
#define MOE_TN 32
#define MOE_TK 32
template <typename TA, typename TW, typename TO, bool QUICK>
__global__ void __launch_bounds__(256)
moe_gate_up_kernel(const TA* __restrict__ x, int ldx, const TW* __restrict__ wgu, const int* __restrict__ order,
                   const int* __restrict__ offsets, const int* __restrict__ tile_off, const float* __restrict__ wts, int E, int top,
                   int F, int D, TO* __restrict__ act, int act_code, int w_out, float limit, float alpha, int gated) {
  tlc_pdl(x, order, offsets, tile_off, wts, act);
  __shared__ float As[MOE_TK][MOE_TM + 1], Gs[MOE_TK][MOE_TN + 1], Us[MOE_TK][MOE_TN + 1];
  __shared__ int tok[MOE_TM];
  int e, row0, rows;
  if (!moe_tile(blockIdx.x, tile_off, offsets, E, &e, &row0, &rows)) return;
  const int n0 = blockIdx.y * MOE_TN;
  if (threadIdx.x < MOE_TM) tok[threadIdx.x] = threadIdx.x < rows ? order[row0 + threadIdx.x] / top : -1;
  __syncthreads();
  const TW* wg = wgu + (size_t)e * (gated ? 2 : 1) * F * D;      // (ungated experts: [E, F, D], one product)
  const TW* wu = gated ? wg + (size_t)F * D : wg;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float g00 = 0.f, g01 = 0.f, g10 = 0.f, g11 = 0.f, u00 = 0.f, u01 = 0.f, u10 = 0.f, u11 = 0.f;
  for (int k0 = 0; k0 < D; k0 += MOE_TK) {
    for (int i = threadIdx.x; i < MOE_TM * MOE_TK; i += 256) {
      const int rr = i / MOE_TK, kk = i % MOE_TK, k = k0 + kk;
      const int tk = tok[rr];
      As[kk][rr] = (tk >= 0 && k < D) ? to_f32(x[(size_t)tk * ldx + k]) : 0.f;
      const int n = n0 + rr;
      const bool ok = n < F && k < D;
      Gs[kk][rr] = ok ? to_f32(wg[(size_t)n * D + k]) : 0.f;
      Us[kk][rr] = (ok && gated) ? to_f32(wu[(size_t)n * D + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < MOE_TK; kk++) {
      const float a0 = As[kk][ty], a1 = As[kk][ty + 16];
      const float p0 = Gs[kk][tx], p1 = Gs[kk][tx + 16], q0 = Us[kk][tx], q1 = Us[kk][tx + 16];
      g00 = fmaf(a0, p0, g00); g01 = fmaf(a0, p1, g01); g10 = fmaf(a1, p0, g10); g11 = fmaf(a1, p1, g11);
      u00 = fmaf(a0, q0, u00); u01 = fmaf(a0, q1, u01); u10 = fmaf(a1, q0, u10); u11 = fmaf(a1, q1, u11);
    }
    __syncthreads();
  }
  const int na = n0 + tx, nb = na + 16;
  if (ty < rows) {
    const float w = wts[order[row0 + ty]];
    TO* o = act + (size_t)(row0 + ty) * F;
    if (na < F) o[na] = from_f32<TO>(moe_pair_act<QUICK>(act_code, w_out, limit, alpha, w, g00, u00));
    if (nb < F) o[nb] = from_f32<TO>(moe_pair_act<QUICK>(act_code, w_out, limit, alpha, w, g01, u01));
  }
  if (ty + 16 < rows) {
    const float w = wts[order[row0 + ty + 16]];
    TO* o = act + (size_t)(row0 + ty + 16) * F;
    if (na < F) o[na] = from_f32<TO>(moe_pair_act<QUICK>(act_code, w_out, limit, alpha, w, g10, u10));
    if (nb < F) o[nb] = from_f32<TO>(moe_pair_act<QUICK>(act_code, w_out, limit, alpha, w, g11, u11));
  }
}

// y[pair(i), :] = Wd[e] act[i, :]; Wd [E, D, F]; y float [T*top, D].
template <typename TA, typename TW>
__global__ void __launch_bounds__(256)
moe_down_kernel(const TA* __restrict__ act, const TW* __restrict__ wd, const int* __restrict__ order,
                const int* __restrict__ offsets, const int* __restrict__ tile_off, int E, int F, int D, float* __restrict__ y) {
  tlc_pdl(act, order, offsets, tile_off, y);
  __shared__ float As[MOE_TK][MOE_TM + 1], Ws[MOE_TK][MOE_TN + 1];
  int e, row0, rows;
  if (!moe_tile(blockIdx.x, tile_off, offsets, E, &e, &row0, &rows)) return;
  const int n0 = blockIdx.y * MOE_TN;
  const TW* w = wd + (size_t)e * D * F;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float c00 = 0.f, c01 = 0.f, c10 = 0.f, c11 = 0.f;
  for (int k0 = 0; k0 < F; k0 += MOE_TK) {
    for (int i = threadIdx.x; i < MOE_TM * MOE_TK; i += 256) {
      const int rr = i / MOE_TK, kk = i % MOE_TK, k = k0 + kk;
      As[kk][rr] = (rr < rows && k < F) ? to_f32(act[(size_t)(row0 + rr) * F + k]) : 0.f;
      const int n = n0 + rr;
      Ws[kk][rr] = (n < D && k < F) ? to_f32(w[(size_t)n * F + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < MOE_TK; kk++) {
      const float a0 = As[kk][ty], a1 = As[kk][ty + 16], w0 = Ws[kk][tx], w1 = Ws[kk][tx + 16];
      c00 = fmaf(a0, w0, c00); c01 = fmaf(a0, w1, c01); c10 = fmaf(a1, w0, c10); c11 = fmaf(a1, w1, c11);
    }
    __syncthreads();
  }
  const int na = n0 + tx, nb = na + 16;
  if (ty < rows) {
    float* o = y + (size_t)order[row0 + ty] * D;
    if (na < D) o[na] = c00;
    if (nb < D) o[nb] = c01;
  }
  if (ty + 16 < rows) {
    float* o = y + (size_t)order[row0 + ty + 16] * D;
    if (na < D) o[na] = c10;
    if (nb < D) o[nb] = c11;
  }
}

static inline int moe_max_tiles(int T, int E, int top) {
  const long long pairs = (long long)T * top;
  return (int)(pairs / MOE_TM + (pairs < E ? pairs : E));
}

extern "C" int tlc_moe_gate_up(const void* x, int x_dtype, int ldx, const void* wgu, int w_dtype, const int* order,
                               const int* offsets, const int* tile_off, const float* wts, int T, int E, int top, int F, int D,
                               void* act, int act_dtype, int act_code, int w_out, float limit, float alpha, cudaStream_t stream) {
  if (T == 0) return 0;
  TLC_REQUIRE(act_code >= TLC_ACT_SILU && act_code <= TLC_ACT_RELU_SQUARED, "moe_gate_up: unknown activation %d", act_code);
  const int gated = act_code != TLC_ACT_RELU_SQUARED;
  dim3 grid(moe_max_tiles(T, E, top), (F + MOE_TN - 1) / MOE_TN);
  if (act_dtype == TLC_BF16) {
    TLC_DISPATCH_DTYPE(x_dtype, TA, TLC_DISPATCH_DTYPE(w_dtype, TW, tlc_launch(moe_gate_up_kernel<TA, TW, __nv_bfloat16, true>, grid,
        dim3(256), 0, stream, (const TA*)x, ldx, (const TW*)wgu, order, offsets, tile_off, wts, E, top, F, D, (__nv_bfloat16*)act, act_code, w_out, limit,
        alpha, gated)));
  } else {
    TLC_DISPATCH_DTYPE(x_dtype, TA, TLC_DISPATCH_DTYPE(w_dtype, TW, tlc_launch(moe_gate_up_kernel<TA, TW, float, false>, grid,
        dim3(256), 0, stream, (const TA*)x, ldx, (const TW*)wgu, order, offsets, tile_off, wts, E, top, F, D, (float*)act, act_code, w_out, limit, alpha, gated)));
  }
  TLC_CHECK_LAUNCH("moe_gate_up");
  return 0;
}

extern "C" int tlc_moe_down(const void* act, int act_dtype, const void* wd, int w_dtype, const int* order, const int* offsets,
                            const int* tile_off, int T, int E, int top, int F, int D, float* y, cudaStream_t stream) {
  if (T == 0) return 0;
  dim3 grid(moe_max_tiles(T, E, top), (D + MOE_TN - 1) / MOE_TN);
  TLC_DISPATCH_DTYPE(act_dtype, TA, TLC_DISPATCH_DTYPE(w_dtype, TW, tlc_launch(moe_down_kernel<TA, TW>, grid, dim3(256), 0, stream,
      (const TA*)act, (const TW*)wd, order, offsets, tile_off, E, F, D, y)));
  TLC_CHECK_LAUNCH("moe_down");
  return 0;
}

// Router outputs without an expert's weights stand for experts that return their input: y[pair, :] = weight * x[token, :]
// for every pair routed to an output >= E (no product visits those pairs).  A block per pair.
template <typename TX>
__global__ void __launch_bounds__(256)
moe_identity_kernel(const TX* __restrict__ x, int ldx, const int* __restrict__ ids, const float* __restrict__ wts, int top, int E, int D,
                    float* __restrict__ y) {
  tlc_pdl(x, ids, wts, y);
  const int pair = blockIdx.x;
  if (ids[pair] < E) return;
  const float w = wts[pair];
  const TX* xr = x + (size_t)(pair / top) * ldx;
  for (int d = threadIdx.x; d < D; d += blockDim.x) y[(size_t)pair * D + d] = w * to_f32(xr[d]);
}
extern "C" int tlc_moe_identity(const void* x, int x_dtype, int ldx, const int* ids, const float* wts, int T, int top, int E, int D,
                                float* y, cudaStream_t stream) {
  if (T == 0) return 0;
  TLC_DISPATCH_DTYPE(x_dtype, TX, tlc_launch(moe_identity_kernel<TX>, dim3(T * top), dim3(256), 0, stream, (const TX*)x, ldx, ids, wts, top,
                                             E, D, y));
  TLC_CHECK_LAUNCH("moe_identity");
  return 0;
}
